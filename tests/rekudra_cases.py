"""Small Rekudra configurations and random weights for the tests. Weights are drawn so that the mechanisms matter: attention
scales make the softmax peaked (a single key more or less shows), convolutions, hyper-connections and gates are of order one,
decays spread from almost none to strong."""

import torch

from tests.pudisun_cases import relative_error, tokens, write_folder  # noqa: F401

BANDS = {"factor": 4.0, "high": 4.0, "low": 1.0, "original": 96}


def attention(heads=4, kv_heads=2, dim=40, vdim=24, conv=3, rot_dims=24, scale=0.5, base=10000.0, scaling=BANDS, ff=160, kv_from=None):
    mixer = {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim,
             "rot": {"base": base, "dims": rot_dims}}
    if scaling:
        mixer["rot"]["scaling"] = scaling
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return entry("attention", mixer, ff)


def delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, ff=None):
    return entry("channel_delta", {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim}, ff)


def entry(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def config(layers, width=104, vocab=333, eps=1e-5, streams=2, embed_scale=3.7):
    return {"architecture": "Rekudra", "embedding": {"scale": embed_scale}, "layers": layers, "norm": {"eps": eps},
            "streams": streams, "vocab": vocab, "width": width}


CONFIGS = {
    # ragged sizes everywhere, keys and values read by later layers, layers without feed-forward, recurrent layer last
    "ragged": config([attention(), delta(), attention(heads=6, kv_heads=3, dim=20, vdim=36, rot_dims=10, ff=None), attention(kv_from=0),
                      attention(heads=6, kv_heads=3, dim=20, vdim=36, rot_dims=10, scale=0.8, kv_from=2), delta(heads=3, kv_heads=3, ff=72)],
                     streams=3),
    # single heads and streams, a convolution of one tap, no frequency scaling, recurrent layer first, another layer's keys last
    "ones": config([delta(heads=1, kv_heads=1, dim=16, vdim=16, conv=1), attention(heads=1, kv_heads=1, dim=16, vdim=16, conv=1, rot_dims=2,
                                                                                  scale=1.0, scaling=None, ff=64),
                    attention(heads=1, kv_heads=1, dim=16, vdim=16, conv=1, rot_dims=2, scale=1.0, scaling=None, ff=64, kv_from=1)],
                   width=64, vocab=128, eps=1e-6, streams=1, embed_scale=1.0),
    # aligned sizes: every GEMM of a decode step on the weight-streaming kernels
    "aligned": config([attention(heads=4, kv_heads=1, dim=64, vdim=64, rot_dims=64, ff=512), delta(heads=2, kv_heads=1, dim=64, vdim=128, ff=512),
                       attention(heads=4, kv_heads=1, dim=64, vdim=64, rot_dims=64, ff=512, kv_from=0)], width=256, vocab=512),
    # more query heads per key/value head than one MMA tile, a value wider than the key, wide states, four streams
    "wide": config([attention(heads=36, kv_heads=2, dim=32, vdim=48, conv=2, rot_dims=32, ff=None), delta(heads=3, kv_heads=1, dim=160, vdim=64, conv=2)],
                   width=192, vocab=320, streams=4),
}


def random_state(cfg: dict, seed: int) -> dict:
    """bf16 checkpoint tensors of a configuration, including the low ranks (5 and 7) that only a tensor's shape gives."""
    gen = torch.Generator().manual_seed(seed)

    def w(*shape, std=None, base=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        return (torch.randn(*shape, generator=gen) * std + base).bfloat16()

    C, n, ranks = cfg["width"], cfg["streams"], (5, 7)
    state = {"embed": w(cfg["vocab"], C, std=1.0), "final.norm": w(C, std=0.2), "head": w(cfg["vocab"], C)}
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        H, G, D, V, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        state[p + "norm1"] = w(C, std=0.2)
        recurrent = e["type"] == "channel_delta"
        rows = {"q": (G if recurrent else H) * D, "k": G * D, "v": (H if recurrent else G) * V}
        for name, count in rows.items():
            if name == "q" or "kv_from" not in m:
                state.update({p + "mix." + name: w(count, C), p + f"mix.{name}.conv": w(count, taps, std=0.7)})
        state[p + "mix.o"] = w(C, H * V)
        if recurrent:
            state.update({p + "mix.b": w(H, C), p + "mix.A_log": w(H, std=1.0), p + "mix.norm": w(V, std=0.2, base=1.0),
                          p + "mix.a1": w(ranks[0], C), p + "mix.a2": w(H * D, ranks[0], std=1.0), p + "mix.dt_bias": w(H * D, std=2.0, base=-3.0),
                          p + "mix.g1": w(ranks[1], C), p + "mix.g2": w(H * V, ranks[1], std=1.0)})
        else:
            state[p + "mix.g"] = w(H, C, std=2 * C ** -0.5)
        for q in (1, 2) if e["mlp"] is not None else (1,):
            state.update({p + f"hc{q}.in": w(n, std=0.5, base=0.7), p + f"hc{q}.out": w(n, std=0.5, base=1.0),
                          p + f"hc{q}.mix": (torch.eye(n) * 0.8 + torch.randn(n, n, generator=gen) * 0.2).bfloat16()})
        if e["mlp"] is not None:
            F = e["mlp"]["ff"]
            state[p + "norm2"] = w(C, std=0.2)
            state.update({p + "mlp.gate": w(F, C), p + "mlp.up": w(F, C), p + "mlp.down": w(C, F)})
    return state
