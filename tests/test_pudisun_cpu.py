"""Pudisun without a GPU: the oracle's own mechanisms against independent statements of them (and against planted mistakes,
so that the tolerances of the GPU tests are known to catch them), the checkpoint reader, configuration, registry, row plans."""

import json
import math
import re
import struct
from pathlib import Path

import numpy as np
import pytest
import torch

from nanochat_b200 import checkpoint, native, registry
from nanochat_b200.__main__ import DTYPE_REFUSED, main
from nanochat_b200.hybrid import HybridConfig
from nanochat_b200.mixers import RowPlan
from nanochat_b200.rotary import half_tables, yarn_frequencies
from oracle import pudisun as oracle
from tests import pudisun_cases as cases

ROOT = Path(__file__).resolve().parent.parent
BF16_TOLERANCE = 0.05  # of the GPU tests, on relative_error of a bf16 run


# ---- the oracle -------------------------------------------------------------------------------------------------------

def test_gla_recurrence_equals_its_unrolled_sum():
    """o_t = sum over s <= t of (q_t . prod of decays . k_s) v_s, written without a state."""
    gen = torch.Generator().manual_seed(1)
    n, C, H, D, V = 9, 12, 2, 4, 6
    m = {"heads": H, "dim": D, "vdim": V, "tau": 3.0}
    w = {k: torch.randn(*s, generator=gen, dtype=torch.float64) for k, s in
         {"q": (H * D, C), "k": (H * D, C), "v": (H * V, C), "g": (H * V, C), "o": (C, H * V), "a1": (2, C), "a2": (H * D, 2),
          "a2.b": (H * D,), "norm": (V,)}.items()}
    h = torch.randn(n, C, generator=gen, dtype=torch.float64)
    got = oracle.gated_linear_attention(h, w, m, 1e-6)
    q, k, v = (h @ w["q"].T / math.sqrt(D)).view(n, H, D), (h @ w["k"].T).view(n, H, D), (h @ w["v"].T).view(n, H, V)
    la = torch.nn.functional.logsigmoid((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]).view(n, H, D) / 3.0
    out = torch.zeros(n, H, V, dtype=torch.float64)
    for t in range(n):
        for s in range(t + 1):
            a = (q[t] * k[s] * la[s + 1:t + 1].sum(0).exp()).sum(-1)
            out[t] += a[:, None] * v[s]
    out = torch.nn.functional.rms_norm(out, (V,), w["norm"], 1e-6).reshape(n, -1)
    want = (out * torch.nn.functional.silu(h @ w["g"].T)) @ w["o"].T
    assert torch.allclose(got, want, rtol=1e-10, atol=1e-10)


def test_latent_attention_equals_torch_attention_with_a_sink_column():
    gen = torch.Generator().manual_seed(2)
    n, C, H, D, R, V, rank = 11, 10, 3, 4, 6, 5, 8
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": rank, "scale": 0.7,
         "rot": {"base": 100.0, "dims": R, "scaling": cases.YARN}}
    w = {k: torch.randn(*s, generator=gen, dtype=torch.float64) for k, s in
         {"q": (H * (D + R), C), "dkv": (rank + R, C), "dkv.norm": (rank,), "uk": (H * D, rank), "uv": (H * V, rank),
          "g": (H * V, C), "o": (C, H * V), "sink": (H,)}.items()}
    h = torch.randn(n, C, generator=gen, dtype=torch.float64)
    got = oracle.latent_attention(h, w, m, 1e-5)
    freqs, factor = yarn_frequencies(R, 100.0, cases.YARN)
    z = torch.polar(torch.full((n, R // 2), factor, dtype=torch.float64), torch.arange(n, dtype=torch.float64)[:, None] * freqs)

    def turn(x):  # [n, .., R] as complex numbers
        c = torch.complex(x[..., :R // 2], x[..., R // 2:]) * z.view(n, *[1] * (x.dim() - 2), -1)
        return torch.cat([c.real, c.imag], -1)

    q = (h @ w["q"].T).view(n, H, D + R)
    kv = h @ w["dkv"].T
    c = torch.nn.functional.rms_norm(kv[:, :rank], (rank,), w["dkv.norm"], 1e-5)
    q = torch.cat([q[..., :D], turn(q[..., D:])], -1)
    k = torch.cat([(c @ w["uk"].T).view(n, H, D), turn(kv[:, rank:])[:, None].expand(n, H, R)], -1)
    s = torch.einsum("ihd,jhd->hij", q, k) * 0.7
    s = s.masked_fill(torch.ones(n, n, dtype=torch.bool).triu(1), -torch.inf)
    p = torch.cat([s, w["sink"].view(H, 1, 1).expand(H, n, 1)], -1).softmax(-1)[..., :-1]
    o = torch.einsum("hij,jhv->ihv", p, (c @ w["uv"].T).view(n, H, V)).reshape(n, -1)
    assert torch.allclose(got, (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T, rtol=1e-9, atol=1e-9)


def test_activations():
    z = torch.linspace(-6, 6, 101, dtype=torch.float64)
    assert torch.allclose(oracle.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)
    assert torch.allclose(oracle.silu(z), torch.nn.functional.silu(z), atol=1e-12)


@pytest.mark.parametrize("mistake", ["no sink", "sink scaled", "late key", "first key lost", "rotation off by one", "no yarn factor",
                                     "state lost", "decay late", "own weights for a shared layer", "plain residual"])
def test_a_planted_mistake_exceeds_the_gpu_tests_tolerance(mistake, monkeypatch):
    """Each mistake changes the oracle's logits by more than what the GPU comparisons allow (in bf16, the looser ones)."""
    cfg = json.loads(json.dumps(cases.CONFIGS["ragged"]))
    state, toks = cases.random_state(cfg, 5), cases.tokens(cfg, 40, 6)
    want = oracle.forward(toks, cfg, state)
    softmax, rotate, gla = oracle.sink_softmax, oracle.rotate, oracle.gated_linear_attention

    def drop(index):
        def weights(scores, sink):
            if len(scores) > 1:
                scores = scores.clone()
                scores[index] = -torch.inf
            return softmax(scores, sink)
        return weights

    def lost_state(h, w, m, eps):
        cut = len(h) // 2
        return torch.cat([gla(h[:cut], w, m, eps), gla(h[cut:], w, m, eps)])

    if mistake == "no sink":
        monkeypatch.setattr(oracle, "sink_softmax", lambda s, sink: torch.softmax(s, -1))
    elif mistake == "sink scaled":
        monkeypatch.setattr(oracle, "sink_softmax", lambda s, sink: softmax(s, 0.35 * float(sink)))
    elif mistake == "late key":
        monkeypatch.setattr(oracle, "sink_softmax", drop(-1))
    elif mistake == "first key lost":
        monkeypatch.setattr(oracle, "sink_softmax", drop(0))
    elif mistake == "rotation off by one":
        calls = []
        monkeypatch.setattr(oracle, "rotate", lambda x, p, r: (calls.append(0), rotate(x, p + (len(calls) % 2), r))[1])
    elif mistake == "no yarn factor":
        f = oracle.rotary_frequencies
        monkeypatch.setattr(oracle, "rotary_frequencies", lambda r: (f(r)[0], 1.0))
    elif mistake == "state lost":
        monkeypatch.setitem(oracle.MIXERS, "gla", lost_state)
    elif mistake == "decay late":
        monkeypatch.setitem(oracle.MIXERS, "gla", lambda h, w, m, eps: gla(h, {**w, "a2.b": w["a2.b"].roll(1)}, m, eps))
    elif mistake == "own weights for a shared layer":
        other = cases.random_state(cases.config([cases.latent()] * 4), 77)
        state = {**state, **{k: v for k, v in other.items() if k.startswith("l3.")}}
        del cfg["layers"][3]["weights_of"]
    elif mistake == "plain residual":
        cfg["residual_mult"] = 0.5
    assert cases.relative_error(oracle.forward(toks, cfg, state), want) > BF16_TOLERANCE


# ---- tables, files, configuration ---------------------------------------------------------------------------------------

def test_rotary_tables_follow_the_oracles_frequencies():
    for rot in ({"dims": 24, "base": 10000.0, "scaling": cases.YARN}, {"dims": 2, "base": 500.0},
                {"dims": 64, "base": 20.0, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}):
        want, factor = oracle.rotary_frequencies(rot)
        got, gf = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        assert torch.allclose(got, want, rtol=1e-13) and gf == pytest.approx(factor, rel=1e-14)
        padded = (rot["dims"] + 15) // 16 * 16
        cos, sin = half_tables(70, rot["dims"], rot["base"], rot.get("scaling"), padded, "cpu")
        assert cos.shape == (70, padded // 2) and cos.dtype == torch.float32
        assert float(cos[69, 0]) == pytest.approx(math.cos(69 * float(want[0])) * factor, abs=1e-6)
        assert float(sin[69, rot["dims"] // 2 - 1]) == pytest.approx(math.sin(69 * float(want[-1])) * factor, abs=1e-6)
        assert (sin[:, rot["dims"] // 2:] == 0).all()


def test_checkpoint_reader(tmp_path):
    cfg = cases.CONFIGS["ones"]
    state = cases.random_state(cfg, 3)
    state["table"] = torch.tensor([3, -1, 7], dtype=torch.int32)
    cases.write_folder(tmp_path, cfg, state)
    got_cfg, got = checkpoint.read_folder(tmp_path)
    assert got_cfg == cfg and set(got) == set(state)
    assert all(torch.equal(got[k], state[k]) and got[k].dtype == state[k].dtype for k in state)
    head = json.dumps({"x": {"dtype": "F32", "shape": [4], "data_offsets": [0, 12]}}).encode()
    (tmp_path / "bad.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + bytes(16))
    with pytest.raises(ValueError):
        checkpoint.read_safetensors(tmp_path / "bad.safetensors")
    with pytest.raises(FileNotFoundError):
        checkpoint.read_folder(tmp_path / "nothing")


def test_configuration_and_registry():
    cfg = HybridConfig.from_pudisun(cases.CONFIGS["ragged"], max_len=100)
    assert [s.kind for s in cfg.layers] == ["latent_attention", "gla", "latent_attention", "latent_attention", "gla"]
    assert [s.weights_of for s in cfg.layers] == [0, 1, 2, 0, 1] and [s.ff for s in cfg.layers] == [160, 160, 0, 160, 160]
    assert (cfg.width, cfg.vocab, cfg.eps, cfg.residual_mult, cfg.logit_scale) == (104, 333, 1e-5, 0.45, 0.7)
    # 128 cached positions: three latent layers of (96 + 32), (96 + 32), (96 + 32) bf16 values, two states of 2 x 32 x 48 fp32
    assert cfg.slot_bytes() - (16 * 128 + 8 * 384 + 8 * 129) == 3 * 128 * 128 * 2 + 2 * 2 * 32 * 48 * 4
    for change in ({"type": "other"}, {"mlp": {"kind": "sparse", "ff": 8}}, {"weights_of": 3}):
        broken = json.loads(json.dumps(cases.CONFIGS["ragged"]))
        broken["layers"][1].update(change)
        with pytest.raises(ValueError):
            HybridConfig.from_pudisun(broken, 64)
    assert torch.float32 in registry.architecture_of(cases.CONFIGS["ones"]).dtypes
    assert registry.architecture_of({"architectures": ["NanochatForCausalLM"]}).dtypes == (torch.bfloat16,)
    assert registry.architecture_of({"model_type": "nanochat"}) is not None
    with pytest.raises(ValueError):
        registry.architecture_of({"architecture": "Unheard"})


def test_command_line_lists_models_and_refuses_a_number_format(tmp_path, capsys):
    assert main(["models"]) == 0
    assert "Pudisun bfloat16 float32" in capsys.readouterr().out
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["NanochatForCausalLM"]}))
    assert main(["trace", "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "8"]) == DTYPE_REFUSED == 3


def test_structures_match_the_header():
    """Field names and order of the ctypes structures against the C declarations."""
    text = re.sub(r"/\*.*?\*/", "", (ROOT / "include" / "nanochat_b200.h").read_text(), flags=re.S)
    for cls, name in ((native.GemmRs, "ncb_gemm_rs"), (native.Latent, "ncb_latent"), (native.Gla, "ncb_gla")):
        body = re.search(r"typedef struct \{([^}]*)\} " + name + ";", text).group(1)
        fields = [f for decl in re.sub(r"\[[^]]*\]", "", body).split(";") if decl.strip()
                  for f in re.findall(r"(\w+)\s*(?:,|$)", decl.strip() + ",")]
        assert fields == [f.rstrip("_") for f, _ in cls._fields_], name


def test_row_plans():
    slots = [4, 4, 4, 1, 1, 7, 7, 7, 7]
    positions = [0, 1, 2, 9, 10, 5, 6, 7, 8]
    plan = RowPlan(slots, positions, "cpu")
    assert plan.n_segments == 3 and plan.longest == 4
    assert plan.first.tolist() == [0, 3, 5] and plan.count.tolist() == [3, 2, 4]
    (seg_chunk, first, count, within), n = plan.chunks(2)
    assert n == 5 and seg_chunk.tolist() == [0, 2, 3, 5] and first.tolist() == [0, 2, 3, 5, 7] and count.tolist() == [2, 1, 2, 2, 2]
    ctx_slot, ctx_first = plan.contexts()
    assert ctx_slot.tolist() == [4, 1, 7] and ctx_first.tolist() == [0, 3, 14, 23]
    (row, rows, ctx, pos), n = plan.row_tiles(2)
    assert n == 5
    assert sorted(zip(row.tolist(), rows.tolist(), ctx.tolist(), pos.tolist())) == [(0, 2, 0, 0), (2, 1, 0, 2), (3, 2, 3, 9), (5, 2, 14, 5),
                                                                                     (7, 2, 14, 7)]
    assert pos.tolist() == sorted(pos.tolist(), reverse=True)
    gap = RowPlan([2, 2, 2], [0, 1, 3], "cpu")  # a jump in positions starts a segment
    assert gap.count.tolist() == [2, 1] and np.array_equal(gap.starts, [0, 3])
