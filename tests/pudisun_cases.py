"""Small Pudisun configurations and random weights for the tests. Weights are drawn so that the mechanisms matter: attention
scales make the softmax peaked (a single key more or less shows), sinks and gates are of order one, decays spread from almost
none to strong."""

import json
import struct

import torch

YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


def latent(heads=3, dim=40, rot_dim=24, vdim=48, kv_rank=72, scale=0.35, base=10000.0, scaling=YARN, ff=160, of=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = scaling
    return entry("latent_attention", {"dim": dim, "heads": heads, "kv_rank": kv_rank, "rot": rot, "rot_dim": rot_dim,
                                      "scale": scale, "vdim": vdim}, ff, of)


def gla(heads=2, dim=24, vdim=40, tau=8.0, ff=160, of=None):
    return entry("gla", {"dim": dim, "heads": heads, "tau": tau, "vdim": vdim}, ff, of)


def entry(kind, mixer, ff, of):
    e = {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}
    if of is not None:
        e["weights_of"] = of
    return e


def config(layers, width=104, vocab=333, eps=1e-5, residual_mult=0.45, logit_scale=0.7):
    return {"architecture": "Pudisun", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps},
            "residual_mult": residual_mult, "vocab": vocab, "width": width}


CONFIGS = {
    # ragged sizes everywhere, shared weights in both kinds, a layer without feed-forward, recurrent layer last
    "ragged": config([latent(), gla(), latent(heads=2, vdim=20, ff=None, scaling=None), latent(of=0), gla(of=1)]),
    # single heads, unit multipliers, one key channel group, no interpolation of the frequencies
    "ones": config([gla(heads=1, dim=16, vdim=16, tau=1.0, ff=None), latent(heads=1, dim=32, rot_dim=2, vdim=16, kv_rank=32, scale=1.0,
                                                                            scaling=None, ff=64)],
                   width=64, vocab=128, eps=1e-6, residual_mult=1.0, logit_scale=1.0),
    # aligned sizes: every GEMM of a decode step on the weight-streaming kernels
    "aligned": config([latent(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, ff=512), gla(heads=2, dim=64, vdim=128, tau=16.0, ff=512)],
                      width=256, vocab=512, logit_scale=0.5),
    # more heads than one MMA tile, latent wider than the small instantiations
    "wide": config([latent(heads=18, dim=32, rot_dim=16, vdim=32, kv_rank=320, ff=None, scale=0.5),
                    gla(heads=3, dim=160, vdim=64, tau=2.0, ff=None)], width=192, vocab=320),
}


def random_state(cfg: dict, seed: int) -> dict:
    """bf16 checkpoint tensors of a configuration, including the decay rank (5) that only a tensor's shape gives."""
    gen = torch.Generator().manual_seed(seed)

    def w(*shape, std=None, base=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        return (torch.randn(*shape, generator=gen) * std + base).bfloat16()

    C, rank_a = cfg["width"], 5
    state = {"embed": w(cfg["vocab"], C, std=1.0), "final.norm": w(C, std=0.2, base=1.0)}
    for i, e in enumerate(cfg["layers"]):
        if "weights_of" in e:
            continue
        m, p = e["mixer"], f"l{i}."
        H, D, V = m["heads"], m["dim"], m["vdim"]
        state[p + "norm1"] = w(C, std=0.2, base=1.0)
        state.update({p + "mix.q": w(H * D if e["type"] == "gla" else H * (D + m["rot_dim"]), C), p + "mix.g": w(H * V, C),
                      p + "mix.o": w(C, H * V)})
        if e["type"] == "gla":
            state.update({p + "mix.k": w(H * D, C), p + "mix.v": w(H * V, C), p + "mix.a1": w(rank_a, C),
                          p + "mix.a2": w(H * D, rank_a, std=1.0), p + "mix.a2.b": w(H * D, std=2.0, base=2.0),
                          p + "mix.norm": w(V, std=0.2, base=1.0)})
        else:
            rank = m["kv_rank"]
            state.update({p + "mix.dkv": w(rank + m["rot_dim"], C), p + "mix.dkv.norm": w(rank, std=0.2, base=1.0),
                          p + "mix.uk": w(H * D, rank), p + "mix.uv": w(H * V, rank), p + "mix.sink": w(H, std=1.0, base=1.0)})
        if e["mlp"] is not None:
            F = e["mlp"]["ff"]
            state[p + "norm2"] = w(C, std=0.2, base=1.0)
            state.update({p + "mlp.gate": w(F, C), p + "mlp.up": w(F, C), p + "mlp.down": w(C, F)})
    return state


def tokens(cfg: dict, n: int, seed: int) -> list[int]:
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def write_folder(folder, cfg: dict, state: dict) -> None:
    """config.json and model.safetensors as a checkpoint folder holds them."""
    names = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}
    header, blobs, at = {}, [], 0
    for name, t in state.items():
        raw = t.contiguous().view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + b"".join(blobs))


def relative_error(got: torch.Tensor, want: torch.Tensor) -> float:
    """Largest rms difference of a row over the rms of all wanted values."""
    d = got.double().cpu() - want.double()
    return float(d.square().mean(-1).sqrt().max() / want.double().square().mean().sqrt())
