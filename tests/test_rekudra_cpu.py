"""Rekudra without a GPU: the oracle's own mechanisms against independent statements of them (and against planted mistakes, so
that the tolerances of the GPU tests are known to catch them), tables, weight preparation, configuration, registry."""

import ctypes
import json
import math
import re
from pathlib import Path

import pytest
import torch

from nanochat_b200 import checkpoint, native, registry
from nanochat_b200.__main__ import main
from nanochat_b200.hybrid import HybridConfig, HybridWeights, HyperConnection
from nanochat_b200.kv_cache import HeadCache, RingCache
from nanochat_b200.mixers import ChannelDelta, GroupedAttention, RowPlan
from nanochat_b200.prompt_store import PromptStore
from nanochat_b200.rotary import frequencies, half_tables
from oracle import rekudra as oracle
from tests import rekudra_cases as cases

ROOT = Path(__file__).resolve().parent.parent
F64 = torch.float64
BF16_TOLERANCE = 0.05  # of the GPU tests, on relative_error of a bf16 run


# ---- the oracle -------------------------------------------------------------------------------------------------------

def test_short_convolution_equals_torch_conv():
    gen = torch.Generator().manual_seed(1)
    for taps in (1, 2, 3, 5):
        u, w = torch.randn(9, 6, generator=gen, dtype=F64), torch.randn(6, taps, generator=gen, dtype=F64)
        want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T[None], (taps - 1, 0)), w[:, None], groups=6)[0].T
        assert torch.allclose(oracle.short_convolution(u, w), want, atol=1e-12)


def test_delta_rule_equals_products_of_transition_matrices():
    """S_t = (I - beta k k^T) diag(g) S_(t-1) + beta k v^T, read out as a sum over earlier tokens without a state."""
    gen = torch.Generator().manual_seed(2)
    n, D, V = 8, 4, 3
    q, k = (oracle.unit(torch.randn(n, D, generator=gen, dtype=F64)) for _ in range(2))
    v, g, beta = torch.randn(n, V, generator=gen, dtype=F64), torch.rand(n, D, generator=gen, dtype=F64), torch.rand(n, generator=gen, dtype=F64)
    step = [(torch.eye(D, dtype=F64) - beta[t] * torch.outer(k[t], k[t])) @ torch.diag(g[t]) for t in range(n)]
    want = torch.zeros(n, V, dtype=F64)
    for t in range(n):
        for s in range(t + 1):
            moved = beta[s] * k[s]
            for j in range(s + 1, t + 1):
                moved = step[j] @ moved
            want[t] += (q[t] @ moved) * v[s]
    assert torch.allclose(oracle.delta_rule(q, k, v, g, beta), want, atol=1e-12)


def test_decays_and_activations():
    z = torch.linspace(-30, 30, 241, dtype=F64)
    assert torch.allclose(oracle.softplus(z), torch.nn.functional.softplus(z, threshold=1000), atol=1e-12)
    assert torch.allclose(oracle.silu(z), torch.nn.functional.silu(z), atol=1e-12)
    h = torch.randn(5, 7, dtype=F64)
    w = {"a1": torch.randn(3, 7, dtype=F64), "a2": torch.randn(8, 3, dtype=F64), "dt_bias": torch.randn(8, dtype=F64), "A_log": torch.randn(2, dtype=F64)}
    want = torch.sigmoid(-((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"])).view(5, 2, 4) ** w["A_log"].exp()[:, None]
    assert torch.allclose(oracle.channel_decay(h, w, 2), want, atol=1e-12)  # exp(-a softplus(z)) = sigmoid(-z)^a


def test_attention_equals_torch_attention_with_complex_rotation():
    gen = torch.Generator().manual_seed(3)
    n, C = 11, 10
    m = cases.attention(heads=6, kv_heads=2, dim=8, vdim=5, rot_dims=6, scale=0.7)["mixer"]
    w = {k: torch.randn(*s, generator=gen, dtype=F64) for k, s in
         {"q": (48, C), "k": (16, C), "v": (10, C), "q.conv": (48, 3), "k.conv": (16, 3), "v.conv": (10, 3), "g": (6, C), "o": (C, 30)}.items()}
    h = torch.randn(n, C, generator=gen, dtype=F64)
    z = torch.polar(torch.ones(n, 3, dtype=F64), torch.arange(n, dtype=F64)[:, None] * oracle.banded_frequencies(m["rot"]))[:, None]

    def heads(name, count, dim):
        return oracle.short_convolution(h @ w[name].T, w[name + ".conv"]).view(n, count, dim)

    def turned(x):
        c = torch.complex(x[..., :3], x[..., 3:6]) * z
        x = torch.cat([c.real, c.imag, x[..., 6:]], -1)
        return torch.nn.functional.rms_norm(x, (8,), eps=1e-5).transpose(0, 1)

    k, v = (x.repeat_interleave(3, 0) for x in (turned(heads("k", 2, 8)), heads("v", 2, 5).transpose(0, 1)))
    o = torch.nn.functional.scaled_dot_product_attention(turned(heads("q", 6, 8)), k, v, is_causal=True, scale=0.7)
    want = (o * torch.sigmoid(h @ w["g"].T).T[..., None]).transpose(0, 1).reshape(n, 30) @ w["o"].T
    assert torch.allclose(oracle.attention(h, w, m, 1e-5, oracle.keys_and_values(h, w, m, 1e-5)), want, atol=1e-10)


def test_frequency_bands():
    """Kept, divided and in between, by the wavelength; the ends of the band meet both."""
    rot = {"dims": 32, "base": 5000.0, "scaling": {"factor": 4.0, "high": 4.0, "low": 1.0, "original": 96}}
    plain, got = oracle.banded_frequencies({**rot, "scaling": None}), oracle.banded_frequencies(rot)
    wavelength = 2 * math.pi / plain
    assert torch.equal(got[wavelength < 24], plain[wavelength < 24]) and (wavelength < 24).sum() > 1
    assert torch.equal(got[wavelength > 96], plain[wavelength > 96] / 4) and (wavelength > 96).sum() > 1
    between = (wavelength > 24) & (wavelength < 96)
    assert between.sum() > 1 and ((got < plain) & (got > plain / 4))[between].all()


def test_streams_are_written_from_the_old_ones():
    x, y = torch.randn(3, 4, 5, dtype=F64), torch.randn(4, 5, dtype=F64)
    w = {"mix": torch.randn(3, 3, dtype=F64), "out": torch.randn(3, dtype=F64), "in": torch.randn(3, dtype=F64)}
    want = torch.einsum("st,snc->tnc", w["mix"], x) + w["out"][:, None, None] * y
    assert torch.allclose(oracle.write_streams(x, y, w), want)
    assert torch.allclose(oracle.read_streams(x, w), torch.einsum("s,snc->nc", w["in"], x))


MISTAKES = ["late key", "first key lost", "rotation off by one", "no bands", "norm before the rotation", "head gate left out", "convolution shifted",
            "convolution without its past", "own keys for a shared layer", "state lost", "no decay", "decay after the write", "read before the write",
            "old value not taken out", "streams mixed the other way", "streams not mixed", "plain norm weight", "embedding not scaled",
            "mean of the streams", "gelu for silu"]


@pytest.mark.parametrize("mistake", MISTAKES)
def test_a_planted_mistake_exceeds_the_gpu_tests_tolerance(mistake, monkeypatch):
    """Each mistake changes the oracle's logits by more than what the GPU comparisons allow (in bf16, the looser ones)."""
    cfg = json.loads(json.dumps(cases.CONFIGS["ragged"]))
    state, toks = cases.random_state(cfg, 5), cases.tokens(cfg, 40, 6)
    want = oracle.forward(toks, cfg, state)
    conv, rotate, attend, rms, delta = (oracle.short_convolution, oracle.rotate, oracle.attention, oracle.root_mean_square, oracle.channel_delta)

    def rule(order):
        def delta_rule(q, k, v, g, beta):
            s, out = torch.zeros(q.shape[1], v.shape[1], dtype=F64), torch.zeros_like(v)
            for t in range(len(q)):
                if order == "read before the write":
                    s = g[t][:, None] * s
                    out[t] = s.T @ q[t]
                    s = s + torch.outer(k[t], beta[t] * (v[t] - s.T @ k[t]))
                    continue
                if order == "decay after the write":
                    s = g[t][:, None] * (s + torch.outer(k[t], beta[t] * (v[t] - s.T @ k[t])))
                else:
                    s = (1 if order == "no decay" else g[t][:, None]) * s
                    s = s + torch.outer(k[t], beta[t] * (v[t] - (0 if order == "old value not taken out" else s.T @ k[t])))
                out[t] = s.T @ q[t]
            return out
        return delta_rule

    def without_key(index):
        def attention(h, w, m, eps, kv):
            scores = torch.softmax
            k = kv[0].clone()
            if index == 0:
                k[0] = -k[0]
                return attend(h, w, m, eps, (k, kv[1]))
            late = (torch.cat([kv[0][:1], kv[0][:-1]]), torch.cat([kv[1][:1], kv[1][:-1]]))  # every row sees one key less
            del scores
            return attend(h, w, m, eps, late)
        return attention

    if mistake in ("late key", "first key lost"):
        monkeypatch.setattr(oracle, "attention", without_key(0 if mistake == "first key lost" else -1))
    elif mistake == "rotation off by one":  # of the queries against the keys
        calls = []

        def shifted(x, rot):
            calls.append(0)
            return rotate(torch.cat([x[:1], x]), rot)[1:] if len(calls) % 2 else rotate(x, rot)
        monkeypatch.setattr(oracle, "rotate", shifted)
    elif mistake == "no bands":
        for e in cfg["layers"]:
            e["mixer"].get("rot", {}).pop("scaling", None)
    elif mistake == "norm before the rotation":  # the same for a whole head, not for one that is turned in parts of it and normed by those
        monkeypatch.setattr(oracle, "rotate", lambda x, rot: torch.cat([rotate(x, rot)[..., :rot["dims"]], 2 * x[..., rot["dims"]:]], -1))
    elif mistake == "head gate left out":
        state = {k: torch.zeros_like(v) if re.fullmatch(r"l\d+\.mix\.g", k) else v for k, v in state.items()}
    elif mistake == "convolution shifted":
        monkeypatch.setattr(oracle, "short_convolution", lambda u, w: conv(u, w.roll(1, 1)))
    elif mistake == "convolution without its past":
        monkeypatch.setattr(oracle, "short_convolution", lambda u, w: torch.cat([conv(u[:20], w), conv(u[20:], w)]))
    elif mistake == "own keys for a shared layer":
        for i in (3, 4):
            j = cfg["layers"][i]["mixer"].pop("kv_from")
            state.update({k.replace(f"l{j}.", f"l{i}."): v for k, v in state.items() if re.match(rf"l{j}\.mix\.[kv]", k)})
    elif mistake == "state lost":
        monkeypatch.setattr(oracle, "channel_delta", lambda h, w, m, eps: torch.cat([delta(h[:20], w, m, eps), delta(h[20:], w, m, eps)]))
    elif mistake in ("no decay", "decay after the write", "read before the write", "old value not taken out"):
        monkeypatch.setattr(oracle, "delta_rule", rule(mistake))
    elif mistake == "streams mixed the other way":
        state = {k: v.T.contiguous() if k.endswith(".mix") else v for k, v in state.items()}
    elif mistake == "streams not mixed":
        state = {k: torch.eye(3).bfloat16() if k.endswith(".mix") else v for k, v in state.items()}
    elif mistake == "plain norm weight":
        monkeypatch.setattr(oracle, "zero_centred_norm", lambda x, w, eps: x / rms(x, eps) * (1.0 + 2.0 * w))
    elif mistake == "embedding not scaled":
        cfg["embedding"]["scale"] = 1.0
    elif mistake == "mean of the streams":  # (alone it would vanish in the norm: the last stream is left out as well)
        cfg2 = cfg["streams"]
        read = oracle.write_streams
        monkeypatch.setattr(oracle, "write_streams", lambda x, y, w: read(x, y, w) * torch.tensor([1.0] * (cfg2 - 1) + [0.0], dtype=F64)[:, None, None])
    elif mistake == "gelu for silu":
        monkeypatch.setattr(oracle, "dense_feed_forward",
                            lambda h, w: (torch.nn.functional.gelu(h @ w["gate"].T, approximate="tanh") * (h @ w["up"].T)) @ w["down"].T)
    assert cases.relative_error(oracle.forward(toks, cfg, state), want) > BF16_TOLERANCE


# ---- tables, weights, configuration -------------------------------------------------------------------------------------

def test_rotary_tables_follow_the_oracles_frequencies():
    for rot in ({"dims": 24, "base": 10000.0, "scaling": cases.BANDS}, {"dims": 2, "base": 500.0},
                {"dims": 64, "base": 300000.0, "scaling": {"factor": 8.0, "original": 2048, "high": 3.0, "low": 0.5}}):
        want = oracle.banded_frequencies(rot)
        got, factor = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        assert torch.allclose(got, want, rtol=1e-13) and factor == 1.0
        cos, sin = half_tables(70, rot["dims"], rot["base"], rot.get("scaling"), rot["dims"], "cpu")
        assert cos.shape == (70, rot["dims"] // 2) and cos.dtype == torch.float32
        assert torch.allclose(cos[69].double(), torch.cos(69 * want), atol=1e-6) and torch.allclose(sin[69].double(), torch.sin(69 * want), atol=1e-6)


def test_weights_are_prepared_with_zeros_where_they_are_padded():
    cfg = cases.CONFIGS["ragged"]
    state = cases.random_state(cfg, 3)
    c = HybridConfig.from_rekudra(cfg, 64)
    w = HybridWeights.from_state_dict(state, c, torch.float32, "cpu")
    assert w.head is not w.embed and torch.equal(w.head[:333, :104], state["head"].float()) and not w.head[333:].any()
    assert torch.equal(w.final_gain[:104], 1 + state["final.norm"].float()) and torch.equal(w.layers[0].gain2[:104], 1 + state["l0.norm2"].float())
    a = w.layers[0].mixer
    assert isinstance(a, GroupedAttention) and (a.dim, a.vdim, a.rot) == (48, 32, 24)
    q = a.w_in[a.off_q:a.off_q + 4 * 48].view(4, 48, -1)
    assert torch.equal(q[:, :40, :104], state["l0.mix.q"].float().view(4, 40, 104)) and not q[:, 40:].any()
    taps = a.conv.w.T[a.off_v:a.off_v + 2 * 32].view(2, 32, 3)
    assert torch.equal(taps[:, :24], state["l0.mix.v.conv"].float().view(2, 24, 3)) and not taps[:, 24:].any()
    shared = w.layers[3].mixer
    assert shared.kv_from == 0 and shared.in_width < a.in_width and shared.conv.width == 4 * 48
    d = w.layers[1].mixer
    assert isinstance(d, ChannelDelta) and (d.rank_a, d.rank_g) == (16, 16) and d.a2.shape == (4, 16, 32)
    assert torch.equal(d.a2[:, :5, :24], state["l1.mix.a2"].float().view(4, 24, 5).transpose(1, 2)) and not d.a2[:, 5:].any()
    hc = w.layers[0].hc2
    assert [hc.read[i] for i in range(3)] == state["l0.hc2.in"].float().tolist() and hc.read[3] == 0
    assert hc.mix[1 * native.MAX_STREAMS + 2] == float(state["l0.hc2.mix"][1, 2]) and w.layers[1].hc2 is None


def test_caches_and_what_a_prompt_store_copies():
    cfg = cases.CONFIGS["ragged"]
    c = HybridConfig.from_rekudra(cfg, 100)
    w = HybridWeights.from_state_dict(cases.random_state(cfg, 3), c, torch.bfloat16, "cpu")
    caches = []
    for layer in w.layers:
        of = layer.mixer.kv_from
        caches.append(layer.mixer.new_cache(2, 100, None if of is None else caches[of]))
    assert caches[3].kv is caches[0].kv and [len(cache.parts) for cache in caches] == [2, 2, 2, 1, 1, 2]
    parts = [part for cache in caches for part in cache.parts]
    assert isinstance(parts[0], HeadCache) and parts[0].rows.shape == (2, 2, 128, 48 + 32) and isinstance(parts[1], RingCache)
    assert c.slot_bytes() - HybridConfig(c.width, c.vocab, [], 1e-5, max_len=100, streams=3).slot_bytes() == sum(p.nbytes() for p in parts) // 2
    for part in parts:
        part.pages.random_(0, 100)
    store, before = PromptStore(parts, 256), [part.pages.clone() for part in parts]
    assert store.save(1, list(range(71))) and store.load(0, list(range(71)))
    for part, old in zip(parts, before):
        k = part.pages_for(70)
        assert torch.equal(part.pages[0, :, :k], old[1, :, :k]) and torch.equal(part.pages[1], old[1])
    with pytest.raises(ValueError):
        w.layers[3].mixer.new_cache(2, 100)


def test_configuration_and_registry(tmp_path, capsys):
    cfg = HybridConfig.from_rekudra(cases.CONFIGS["ragged"], max_len=100)
    assert [s.kind for s in cfg.layers] == ["attention", "channel_delta", "attention", "attention", "attention", "channel_delta"]
    assert [s.ff for s in cfg.layers] == [160, 0, 0, 160, 160, 72]
    assert (cfg.width, cfg.vocab, cfg.eps, cfg.streams, cfg.embed_scale, cfg.tied_head) == (104, 333, 1e-5, 3, 3.7, False)
    for where, change in ((1, {"type": "other"}), (1, {"mlp": {"kind": "sparse", "ff": 8}}), (3, {"mixer": {**cases.attention()["mixer"], "kv_from": 3}}),
                          (4, {"mixer": {**cases.attention()["mixer"], "kv_from": 3}}), (3, {"mixer": {**cases.attention()["mixer"], "kv_from": 1}})):
        broken = json.loads(json.dumps(cases.CONFIGS["ragged"]))
        broken["layers"][where].update(change)
        with pytest.raises(ValueError):
            HybridConfig.from_rekudra(broken, 64)
    assert registry.architecture_of(cases.CONFIGS["ones"]).dtypes == (torch.bfloat16, torch.float32)
    assert main(["models"]) == 0
    assert "Rekudra bfloat16 float32" in capsys.readouterr().out
    state = cases.random_state(cases.CONFIGS["ones"], 3)
    cases.write_folder(tmp_path, cases.CONFIGS["ones"], state)
    got_cfg, got = checkpoint.read_folder(tmp_path)
    assert got_cfg == cases.CONFIGS["ones"] and all(torch.equal(got[k], state[k]) for k in state)
    with pytest.raises(ValueError):  # connections of another number of streams
        HybridWeights.from_state_dict({**state, "l0.hc1.in": torch.ones(2)}, HybridConfig.from_rekudra(cases.CONFIGS["ones"], 64), torch.float32, "cpu")


def test_random_weights_fit_the_configuration():
    for name in cases.CONFIGS:
        cfg = HybridConfig.from_rekudra(cases.CONFIGS[name], 64)
        state = HybridWeights.random_state(cfg, 1)
        wanted = cases.random_state(cases.CONFIGS[name], 1)
        assert set(state) == set(wanted)
        HybridWeights.from_state_dict(state, cfg, torch.bfloat16, "cpu")


def test_hyper_connections_as_the_kernels_take_them():
    read, write, mix = torch.tensor([1.0, 2.0]), torch.tensor([3.0, 4.0]), torch.tensor([[5.0, 6.0], [7.0, 8.0]])
    hc = HyperConnection.of(read, write, mix)
    a = native.GemmRs()
    a.in_, a.out, a.mix = hc.read, hc.write, hc.mix
    assert (a.in_[1], a.out[0], a.mix[1], a.mix[native.MAX_STREAMS], a.mix[2], hc.read_sum) == (2.0, 3.0, 6.0, 7.0, 0.0, 3.0)


def test_structures_match_the_header():
    """Field names and order of the ctypes structures against the C declarations, and the sizes of their arrays."""
    text = re.sub(r"/\*.*?\*/", "", (ROOT / "include" / "nanochat_b200.h").read_text(), flags=re.S)
    for cls, name in ((native.Conv, "ncb_conv"), (native.Gqa, "ncb_gqa"), (native.Delta, "ncb_delta")):
        body = re.search(r"typedef struct \{([^}]*)\} " + name + ";", text).group(1)
        fields = [f for decl in body.split(";") if decl.strip() for f in re.findall(r"(\w+)\s*(?:,|$)", decl.strip() + ",")]
        assert fields == [f for f, _ in cls._fields_], name
    assert int(re.search(r"#define NCB_MAX_STREAMS (\d+)", text).group(1)) == native.MAX_STREAMS
    assert ctypes.sizeof(native.GemmRs) % 8 == 0


def test_chunks_know_what_of_their_segment_lies_before_them():
    plan = RowPlan([4, 4, 4, 1, 1], [0, 1, 2, 9, 10], "cpu")
    (seg_chunk, first, count, within), n = plan.chunks(2)
    assert n == 3 and first.tolist() == [0, 2, 3] and count.tolist() == [2, 1, 2] and within.tolist() == [0, 2, 0] and seg_chunk.tolist() == [0, 2, 3]


def test_sizes_of_the_chunked_delta_rule():
    lib = native.cuda_library("delta_rule")
    assert lib.delta_chunk_tokens(128, 128, 4, 128, 128) == 64 and lib.delta_chunk_tokens(256, 256, 4, 128, 128) == 32
    assert lib.delta_chunk_tokens(272, 64, 4, 16, 16) == 0 and lib.delta_chunk_tokens(128, 128, 4, 4096, 16) == 0
