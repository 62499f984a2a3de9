"""Rekudra on the GPU against the plain oracle (oracle/rekudra.py): each mechanism alone, whole prompts, portions, decoding,
batches, slots used again, generation through the scheduler, the command line and the trace runner."""

import ctypes
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from nanochat_b200 import native
from nanochat_b200.hybrid import STREAMS, SWIGLU, HybridConfig, HybridDecoder, HyperConnection, HybridWeights, Stream
from nanochat_b200.mixers import ChannelDelta, GroupedAttention, RowPlan, Rows, ShortConv, up
from nanochat_b200.serving import NativeDecoder, Request
from oracle import rekudra as oracle
from tests import rekudra_cases as cases

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
F32, BF16 = torch.float32, torch.bfloat16
# relative_error of logits or mixer outputs: fp32 rounding through a few layers, and bf16 products and activations (planted
# mistakes, tests/test_rekudra_cpu.py, all exceed the larger one)
TOLERANCE = {F32: 2e-5, BF16: 0.05}
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def decoder(cfg: dict, state: dict, dtype, n_slots=3, max_len=256, **kw) -> HybridDecoder:
    c = HybridConfig.from_rekudra(cfg, max_len)
    c.itemsize = dtype.itemsize
    return HybridDecoder(c, HybridWeights.from_state_dict(state, c, dtype), n_slots, **kw)


_oracle: dict = {}


def case(name: str, n: int, seed: int = 1):
    """(configuration, weights, tokens, the oracle's logits), computed once per test run."""
    if (name, n, seed) not in _oracle:
        cfg = cases.CONFIGS[name]
        state, toks = cases.random_state(cfg, seed), cases.tokens(cfg, n, seed + 50)
        _oracle[name, n, seed] = cfg, state, toks, oracle.forward(toks, cfg, state)
    return _oracle[name, n, seed]


def close(got: torch.Tensor, want: torch.Tensor, dtype) -> None:
    err = cases.relative_error(got, want)
    assert err < TOLERANCE[dtype], err


# ---- mechanisms alone -----------------------------------------------------------------------------------------------

def rows_of(slots, positions, status, plan=True, **kw) -> Rows:
    pos = torch.tensor(positions, dtype=torch.int32, device="cuda")
    slot_map = torch.tensor(slots, dtype=torch.int32, device="cuda")
    return Rows(len(slots), pos, slot_map, max(positions) + 1, status, RowPlan(slots, positions, "cuda") if plan else None, **kw)


def part(state: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in state.items() if k.startswith(prefix)}


def run_mixer(mixer, cache, h, dtype, pieces, rank=2):
    """The mixer's output projection applied to its launches' output for h [n, C], run in `pieces` (row counts)."""
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    x = torch.zeros((len(h), mixer.w_in.shape[1]), dtype=dtype, device="cuda")
    x[:, :h.shape[1]] = h.to(dtype)
    got, at = [], 0
    for n in pieces:
        proj = (x[at:at + n].float() @ mixer.w_in.float().T).to(dtype)
        out = torch.zeros((n, mixer.out_width), dtype=dtype, device="cuda")
        mixer.run(proj, cache, rows_of([rank] * n, list(range(at, at + n)), status, plan=n > 1), out)
        got.append(out.double() @ mixer.w_out.double().T)
        at += n
    assert int(status.item()) == 0 and at == len(h)
    return torch.cat(got)[:, :h.shape[1]]


def new_mixer(cls, entry, state, dtype, columns, layer=0):
    return cls(entry["mixer"], part(state, f"l{layer}.mix."), 1e-5, columns, dtype, "cuda")


def fresh_cache(mixer, positions: int, of=None):
    cache = mixer.new_cache(3, positions, of)
    for one in cache.parts:  # what was never written must not be read into a result
        getattr(one, "rows", getattr(one, "state", None)).fill_(float("nan"))
    return cache


ATTENTION_SIZES = {
    "ragged": cases.attention(), "one head": cases.attention(heads=1, kv_heads=1, dim=16, vdim=16, conv=1, rot_dims=2, scale=1.0, scaling=None),
    "two head tiles": cases.attention(heads=20, kv_heads=1, dim=32, vdim=32, rot_dims=32),
    "64": cases.attention(heads=6, kv_heads=2, dim=64, vdim=64, rot_dims=64), "128": cases.attention(heads=4, kv_heads=1, dim=128, vdim=128, conv=4, rot_dims=32, scale=0.2),
    "wide key": cases.attention(heads=2, kv_heads=2, dim=192, vdim=64, conv=2, rot_dims=96, scale=0.2),
    "wide value": cases.attention(heads=2, kv_heads=1, dim=48, vdim=256, rot_dims=48), "256": cases.attention(heads=4, kv_heads=2, dim=256, vdim=208, rot_dims=64, scale=0.1),
    "beyond the tensor-core forms": cases.attention(heads=2, kv_heads=2, dim=272, vdim=288, conv=5, rot_dims=256, scale=0.1)}


@DTYPES
@pytest.mark.parametrize("sizes", list(ATTENTION_SIZES))
@pytest.mark.parametrize("mode", ["tiled", "rows", "decoded", "mixed"])
def test_attention_alone(dtype, sizes, mode):
    entry, n, C = ATTENTION_SIZES[sizes], 150, 64
    state = cases.random_state(cases.config([entry], width=C), 7)
    h = torch.randn(n, C, generator=torch.Generator().manual_seed(8)).to(dtype)
    w = oracle.part(state, "l0.mix.")
    want = oracle.attention(h.double(), w, entry["mixer"], 1e-5, oracle.keys_and_values(h.double(), w, entry["mixer"], 1e-5))
    mixer = new_mixer(GroupedAttention, entry, state, dtype, 128)
    if mode != "mixed":
        mixer.tiled = mixer.tiled and mode == "tiled"
    pieces = {"tiled": [66, 2, n - 68], "rows": [33, 2, n - 35], "decoded": [1] * n, "mixed": [1, 2, 1, 60, 1, 8, 64, 3, 1, 9]}[mode]
    close(run_mixer(mixer, fresh_cache(mixer, n), h, dtype, pieces), want, dtype)


@DTYPES
@pytest.mark.parametrize("mode", ["tiled", "rows", "decoded"])
def test_a_key_that_stands_out_is_found_wherever_it_lies(dtype, mode):
    """One earlier row's key is made to dominate a later row's score: the query's projection is the key's with its columns
    rolled, and the later row's inputs (over all taps) are the earlier row's, rolled as well, so that the two meet and the later
    row's own key does not. At tile, page and chunk borders, first and last positions."""
    entry = cases.attention(heads=4, kv_heads=2, dim=32, vdim=32, conv=2, rot_dims=16, scale=1.2, base=1e6, scaling=None)
    C, n = 64, 200
    state = cases.random_state(cases.config([entry], width=C), 17)
    for name, size in (("", C), (".conv", 2)):
        k = state["l0.mix.k" + name].reshape(2, 32, size).repeat_interleave(2, 0).reshape(128, size)
        state["l0.mix.q" + name] = k if name else k.roll(5, 1)
    h = torch.randn(n, C, generator=torch.Generator().manual_seed(18))
    pairs = ((1, 199), (16, 196), (31, 193), (33, 190), (64, 187), (66, 184), (128, 181), (129, 132), (176, 178))
    for key, query in pairs:
        h[query - 1:query + 1] = h[key - 1:key + 1].roll(5, 1)
    h = h.to(dtype)
    w = oracle.part(state, "l0.mix.")
    want = oracle.attention(h.double(), w, entry["mixer"], 1e-5, oracle.keys_and_values(h.double(), w, entry["mixer"], 1e-5))
    mixer = new_mixer(GroupedAttention, entry, state, dtype, 128)
    mixer.tiled = mixer.tiled and mode == "tiled"
    pieces = [120] + [1] * 80 if mode == "decoded" else [64, 65, 71]
    close(run_mixer(mixer, fresh_cache(mixer, n), h, dtype, pieces), want, dtype)
    for key, query in pairs:  # (the test would see any of these keys missing)
        kv = without(oracle.keys_and_values(h.double(), w, entry["mixer"], 1e-5), key)
        assert (oracle.attention(h.double(), w, entry["mixer"], 1e-5, kv) - want)[query].norm() > 0.3 * want[query].norm()


def without(kv, position: int):
    k, v = kv[0].clone(), kv[1].clone()
    k[position] = -k[position]
    return k, v


@DTYPES
def test_attention_over_another_layers_keys_and_values(dtype):
    first, second = cases.attention(), cases.attention(scale=0.9, kv_from=0)
    C, n = 64, 90
    state = cases.random_state(cases.config([first, second], width=C), 27)
    assert "l1.mix.k" not in state
    gen = torch.Generator().manual_seed(28)
    h0, h1 = (torch.randn(n, C, generator=gen).to(dtype) for _ in range(2))
    w0, w1 = oracle.part(state, "l0.mix."), oracle.part(state, "l1.mix.")
    kv = oracle.keys_and_values(h0.double(), w0, first["mixer"], 1e-5)
    want = oracle.attention(h1.double(), w1, second["mixer"], 1e-5, kv)
    a, b = new_mixer(GroupedAttention, first, state, dtype, 128), new_mixer(GroupedAttention, second, state, dtype, 128, 1)
    cache = fresh_cache(a, n)
    shared = fresh_cache(b, n, cache)
    assert shared.kv is cache.kv and len(shared.parts) == 1
    got, at = [], 0
    for m in (30, 2, 1, 1, 40, 1, 15):
        run = lambda mixer, c, h: run_at(mixer, c, h, dtype, at, m)  # noqa: E731
        run(a, cache, h0)
        got.append(run(b, shared, h1))
        at += m
    close(torch.cat(got)[:, :C], want, dtype)


def run_at(mixer, cache, h, dtype, at, m, slot=1):
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    x = torch.zeros((m, mixer.w_in.shape[1]), dtype=dtype, device="cuda")
    x[:, :h.shape[1]] = h[at:at + m].to(dtype)
    proj = (x.float() @ mixer.w_in.float().T).to(dtype)
    out = torch.zeros((m, mixer.out_width), dtype=dtype, device="cuda")
    mixer.run(proj, cache, rows_of([slot] * m, list(range(at, at + m)), status, plan=m > 1), out)
    assert int(status.item()) == 0
    return out.double() @ mixer.w_out.double().T


DELTA_SIZES = {"ragged": cases.delta(), "one": cases.delta(heads=1, kv_heads=1, dim=16, vdim=16, conv=1), "64": cases.delta(heads=2, kv_heads=2, dim=64, vdim=64),
               "128": cases.delta(heads=3, kv_heads=1, dim=128, vdim=128), "wide value": cases.delta(heads=2, kv_heads=1, dim=32, vdim=272, conv=2),
               "wide": cases.delta(heads=2, kv_heads=2, dim=160, vdim=256), "widest": cases.delta(heads=1, kv_heads=1, dim=272, vdim=96, conv=6),
               "token by token only": cases.delta(heads=1, kv_heads=1, dim=528, vdim=32)}


@DTYPES
@pytest.mark.parametrize("sizes", list(DELTA_SIZES))
@pytest.mark.parametrize("mode", ["step", "chunked", "mixed", "decoded"])
def test_delta_rule_alone(dtype, sizes, mode):
    entry, n, C = DELTA_SIZES[sizes], 150, 64
    state = cases.random_state(cases.config([entry], width=C), 37)
    h = torch.randn(n, C, generator=torch.Generator().manual_seed(38)).to(dtype)
    want = oracle.channel_delta(h.double(), oracle.part(state, "l0.mix."), entry["mixer"], 1e-5)
    mixer = new_mixer(ChannelDelta, entry, state, dtype, 128)
    if mode != "mixed":
        mixer.CHUNKED_FROM = 1 if mode == "chunked" else 10 ** 9
    pieces = {"step": [40, 2, 1, 107], "chunked": [66, 2, 82], "mixed": [64, 1, 1, 2, 63, 19], "decoded": [1] * n}[mode]
    close(run_mixer(mixer, fresh_cache(mixer, n), h, dtype, pieces), want, dtype)


@DTYPES
@pytest.mark.parametrize("decay", ["strong", "none", "uneven"])
def test_delta_rule_with_decays_at_the_extremes(dtype, decay):
    """Decays that leave nothing after a token, that forget nothing, and both side by side in one head."""
    entry, n, C = cases.delta(heads=2, kv_heads=1, dim=64, vdim=48), 200, 64
    state = cases.random_state(cases.config([entry], width=C), 47)
    bias = state["l0.mix.dt_bias"]
    state["l0.mix.dt_bias"] = {"strong": torch.full_like(bias, 40.0), "none": torch.full_like(bias, -30.0),
                               "uneven": torch.where(torch.arange(len(bias)) % 3 == 0, 30.0, -12.0).bfloat16()}[decay]
    h = torch.randn(n, C, generator=torch.Generator().manual_seed(48)).to(dtype)
    want = oracle.channel_delta(h.double(), oracle.part(state, "l0.mix."), entry["mixer"], 1e-5)
    mixer = new_mixer(ChannelDelta, entry, state, dtype, 128)
    mixer.CHUNKED_FROM = 1
    close(run_mixer(mixer, fresh_cache(mixer, n), h, dtype, [130, 70]), want, dtype)
    mixer.CHUNKED_FROM = 10 ** 9
    close(run_mixer(mixer, fresh_cache(mixer, n), h, dtype, [150] + [1] * 50), want, dtype)


@DTYPES
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_the_ring_of_a_convolution_holds_the_last_rows(dtype, taps):
    """After portions of every size around the number of taps: position p's row at p % taps, other slots untouched."""
    conv = ShortConv([(torch.randn(24, taps), 0)], 24, dtype, "cuda")
    ring, n = conv.new_ring(3), 40
    ring.rows.fill_(7.0)
    x = torch.randn(n, 40, device="cuda").to(dtype)
    status, at = torch.zeros(1, dtype=torch.int32, device="cuda"), 0
    for m in (2, 3, 2, 9, 4, 5, 7, 8):
        rows = rows_of([1] * m, list(range(at, at + m)), status)
        conv.keep_tail(conv.args(x[at:at + m], ring, rows), rows)
        at += m
        for back in range(1, min(taps, at + 1)):
            assert torch.equal(ring.rows[1, (at - back) % taps], x[at - back, :24])
    assert (ring.rows[[0, 2]] == 7).all() and int(status.item()) == 0


@DTYPES
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8])
@pytest.mark.parametrize("rows", [1, 9, 16, 17, 40, 65, 300])
def test_gemms_on_several_streams(dtype, rows, streams):
    """The kernels (by rows) with hyper-connections: the scaled embedding as the first streams, a branch's result and the old
    streams as the new ones with what the next norm reads; the silu-gated unit."""
    width, C, F, V = 300, 384, 256, 520
    cfg = HybridConfig(width=width, vocab=V, layers=[], eps=1e-3, streams=streams)
    dec = HybridDecoder.__new__(HybridDecoder)
    dec.cfg, dec.f32, dec.status = cfg, dtype == F32, torch.zeros(1, dtype=torch.int32, device="cuda")
    gen = torch.Generator(device="cuda").manual_seed(rows)

    def r(*shape, std=1.0, dt=dtype):
        return (torch.randn(*shape, generator=gen, device="cuda") * std).to(dt)

    def connection():
        read, write, mix = r(streams, dt=F32), r(streams, dt=F32), r(streams, streams, dt=F32)
        return HyperConnection.of(read.cpu(), write.cpu(), mix.cpu()), read, write, mix

    embed, gain, gain2 = r(V, C), r(C, dt=F32), r(C, dt=F32)
    embed[:, width:], gain[width:], gain2[width:] = 0, 0, 0
    toks = torch.randint(0, V, (rows,), generator=gen, device="cuda")
    st = Stream(rows, C, dtype, "cuda", streams)
    hc, read, write, mix = connection()
    lib = native.cuda_library("decode_step")
    native.check(lib.embed_streams(*map(native.pointer, (embed, toks, st.h, gain, st.x, st.ss)), rows, C, V, int(dtype == F32), streams, 1.7,
                                   hc.read_sum, native.stream()), "embed_streams")
    h = (1.7 * embed[toks].float())[:, None].expand(rows, streams, C)
    tol = 1e-5 if dtype == F32 else 2e-2

    def same(got, want, tol=tol):
        err = (got.float() - want).abs().max() / want.abs().max()
        assert float(err) < tol, float(err)

    def norm(u, g):
        return u / (u.square().sum(-1, keepdim=True) / width + 1e-3).sqrt() * g

    same(st.h.view(rows, streams, C), h, 1e-6)
    u = torch.empty((rows, F), dtype=dtype, device="cuda")
    wu = r(2 * F, C, std=0.05)
    dec.gemm(rows, st.x, wu, SWIGLU, st, out=u, normed=True)
    z = norm((read[:, None] * h).sum(1), gain) @ wu.float().T
    same(u, torch.nn.functional.silu(z[:, 0::2]) * z[:, 1::2])
    for _ in range(2):  # from equal streams, then from different ones
        nxt = connection()
        x, wo = r(rows, F), r(C, F, std=0.05)
        wo[width:] = 0
        dec.gemm(rows, x, wo, STREAMS, st, gain=gain2, hc=(hc, nxt[0]))
        y = x.float() @ wo.float().T
        h = torch.einsum("st,rsc->rtc", mix, h) + write[:, None] * y[:, None]
        read_next = (nxt[1][:, None] * h).sum(1)
        same(st.h.view(rows, streams, C), h)
        same(st.x, read_next * gain2)
        parts = st.ss.view(-1)[:rows * st.parts].view(rows, st.parts)
        same(parts.sum(-1), read_next.square().sum(-1))
        hc, read, write, mix = nxt
    assert int(dec.status.item()) == 0


def test_arguments_out_of_range_are_refused_on_the_host():
    lib, a = native.cuda_library("decode_step"), native.GemmRs()
    x = torch.zeros(8, 256, device="cuda", dtype=BF16)
    a.x = a.w = a.h = a.gain = a.x_next = a.ss_next = x.data_ptr()
    a.rows, a.N, a.K, a.epilogue = 1, 8, 256, STREAMS
    for streams in (0, 9):
        a.streams = streams
        assert lib.skinny_gemm_rs(ctypes.byref(a), native.stream()) == 1
    with pytest.raises(ValueError):
        HybridConfig.from_rekudra(cases.config([cases.attention()], streams=9), 64)
    with pytest.raises(ValueError):
        HybridConfig.from_rekudra(cases.config([cases.attention(), cases.attention(kv_from=1)]), 64)


# ---- the whole model ------------------------------------------------------------------------------------------------

@DTYPES
@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_whole_prompts_portions_and_decoding(dtype, name):
    cfg, state, toks, want = case(name, 150)
    dec = decoder(cfg, state, dtype)
    every = list(range(len(toks)))
    close(dec.feed(0, toks, 0, every), want, dtype)
    for size in (2, 3, 17, 64, 65):  # slot 0 and 1 alternate: both have been used before
        got, at = [], 0
        while at < len(toks):
            n = min(size, len(toks) - at)
            got.append(dec.feed(size % 2, toks[at:at + n], at, list(range(n))))
            at += n
        close(torch.cat(got), want, dtype)
    got = [dec.feed(2, toks[:37], 0, list(range(37)))]
    got += [dec.feed(2, [t], 37 + i, [0]) for i, t in enumerate(toks[37:])]  # 113 steps, over page and tile borders
    close(torch.cat(got), want, dtype)
    assert int(dec.status.item()) == 0


@DTYPES
def test_first_tokens_and_prompts_of_one_token(dtype):
    for name in ("ragged", "ones"):
        cfg, state, toks, want = case(name, 6)
        dec = decoder(cfg, state, dtype)
        for n in (6, 1, 2, 3, 6):
            close(dec.feed(1, toks[:n], 0, list(range(n))), want[:n], dtype)
        for i, t in enumerate(toks):
            close(dec.feed(0, [t], i, [0]), want[i:i + 1], dtype)


@DTYPES
def test_long_prompts_far_keys_and_passes_of_a_prompt(dtype):
    """A prompt longer than any chunk, tile or page, in one pass and in several, then decoding on; small heads for the oracle."""
    cfg = cases.config([cases.attention(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=16, ff=None, scaling={**cases.BANDS, "original": 256}),
                        cases.delta(heads=1, kv_heads=1, dim=16, vdim=16, ff=96)], width=64, vocab=96)
    state, toks = cases.random_state(cfg, 9), cases.tokens(cfg, 700, 10)
    want = oracle.forward(toks, cfg, state)
    dec = decoder(cfg, state, dtype, max_len=720)
    every = list(range(len(toks)))
    close(dec.feed(0, toks, 0, every), want, dtype)
    close(dec.feed(1, toks, 0, every, rows_per_pass=256), want, dtype)
    dec.feed(2, toks[:600], 0, [])
    close(torch.cat([dec.feed(2, [t], 600 + i, [0]) for i, t in enumerate(toks[600:])]), want[600:], dtype)
    assert int(dec.status.item()) == 0


@DTYPES
def test_batches_of_unequal_requests_match_each_request_alone(dtype):
    """Prompts of different lengths in one pass (also cut by the pass's size), then decode steps over all slots in another
    order than the slots', against the oracle; an idle slot's cache and state stay as they are."""
    name = "ragged"
    lens = (5, 71, 1, 130, 64)
    seqs = [case(name, n + 9, seed=s) for s, n in enumerate(lens)]
    cfg, state = seqs[0][0], seqs[0][1]
    seqs = [(toks, oracle.forward(toks, cfg, state)) for _, _, toks, _ in seqs]
    for per_pass in (4096, 50):
        dec = decoder(cfg, state, dtype, n_slots=6)
        slots = [3, 0, 5, 1, 4]
        dec.prefill([toks[:n] for (toks, _), n in zip(seqs, lens)], slots, rows_per_pass=per_pass)
        order = [4, 2, 0, 3, 1]
        slot_map = torch.tensor([slots[i] for i in order], dtype=torch.int32, device="cuda")
        buf = dec.step_buffers(len(order))
        for step in range(9):
            idle = order[step % 3]  # one sequence pauses and continues: its row is idle for this step
            tokens = torch.tensor([seqs[i][0][lens[i] - 1 + (step if i != idle or step < 6 else 0)] for i in order], device="cuda")
            pos = torch.tensor([lens[i] - 1 + step for i in order], dtype=torch.int32, device="cuda")
            if step >= 6:
                pos[step % 3] = -1
            dec.run_step(tokens, pos, slot_map, buf)
            live = [r for r in range(len(order)) if int(pos[r]) >= 0]
            want = torch.stack([seqs[order[r]][1][lens[order[r]] - 1 + step] for r in live])
            close(buf["logits"][live], want, dtype)
            if step >= 6:  # catch the idle sequence up, alone
                i = idle
                got = dec.feed(slots[i], [seqs[i][0][lens[i] - 1 + step]], lens[i] - 1 + step, [0])
                close(got, seqs[i][1][lens[i] - 1 + step][None], dtype)
        assert int(dec.status.item()) == 0


def test_long_decoding_stays_with_the_oracle():
    """600 steps in 32-bit, the recurrent state carried all the way, the ring turning around 150 times and more."""
    cfg = cases.config([cases.delta(heads=2, kv_heads=1, dim=16, vdim=16, ff=None), cases.attention(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=8, ff=48)],
                       width=48, vocab=64)
    state, toks = cases.random_state(cfg, 19), cases.tokens(cfg, 600, 20)
    want = oracle.forward(toks, cfg, state)
    dec = decoder(cfg, state, F32, max_len=640)
    close(torch.cat([dec.feed(1, [t], i, [0]) for i, t in enumerate(toks)]), want, F32)


def greedy(cfg, state, prompt, n) -> list[int]:
    out = list(prompt)
    for _ in range(n):
        out.append(int(oracle.forward(out, cfg, state)[-1].argmax()))
    return out[len(prompt):]


def test_greedy_generation_through_the_scheduler_matches_the_oracle():
    """Seven requests through three slots (slots are freed and used again while others run), and generate(); 32-bit, where the
    choice is the oracle's."""
    cfg = cases.CONFIGS["ones"]
    state = cases.random_state(cfg, 31)
    prompts = [cases.tokens(cfg, n, 60 + n) for n in (1, 30, 7, 66, 2, 64, 12)]
    lengths = [4, 9, 3, 6, 8, 2, 5]
    want = [greedy(cfg, state, p, n) for p, n in zip(prompts, lengths)]
    dec = decoder(cfg, state, F32)
    served = dict(NativeDecoder(dec, end_token=-1).generate(
        [Request(input_ids=p, max_new_tokens=n) for p, n in zip(prompts, lengths)]))
    assert [served[i] for i in range(7)] == want
    out, times = decoder(cfg, state, F32).generate(prompts[:3], 3)
    assert [o[:3] for o in out] == [w[:3] for w in want[:3]] and times["tokens_per_s"] > 0
    cfg = cases.CONFIGS["ragged"]
    state, prompt = cases.random_state(cfg, 34), cases.tokens(cfg, 21, 35)
    assert decoder(cfg, state, F32).generate([prompt], 4)[0] == [greedy(cfg, state, prompt, 4)]


def test_served_requests_do_not_depend_on_the_batch_and_prompts_come_from_the_store():
    """bf16: the same streams alone, in a full batch, sampled and greedy; a prompt seen before is copied from the store (keys and
    values, rings, states) instead of being prefilled."""
    cfg = cases.CONFIGS["aligned"]
    state = cases.random_state(cfg, 32)
    prompts = [cases.tokens(cfg, n, 80 + n) for n in (40, 3, 90, 17)]
    reqs = [Request(input_ids=p, max_new_tokens=10, temperature=0.8 * (i % 2), top_p=0.9, seed=i) for i, p in enumerate(prompts)]
    alone = [dict(NativeDecoder(decoder(cfg, state, BF16), end_token=-1).generate([r]))[0] for r in reqs]
    nd = NativeDecoder(decoder(cfg, state, BF16, prompt_store=512), end_token=-1)
    passes = []
    prefill = nd.decoder.prefill
    nd.decoder.prefill = lambda prompts, slots, **kw: (passes.append(len(prompts)), prefill(prompts, slots, **kw))
    first = dict(nd.generate(reqs))
    again = dict(nd.generate(reqs[::-1]))
    assert sum(passes) == 4
    # a pass holds other rows than a prompt alone, and batches other GEMM shapes: equal up to rounding, which random logits
    # rarely turn into another choice
    same = sum(first[i] == alone[i] for i in range(4)) + sum(again[3 - i] == first[i] for i in range(4))
    assert same >= 7, (alone, first, again)


def test_positions_and_slots_outside_the_cache_are_refused_and_flagged():
    cfg = cases.CONFIGS["ones"]
    dec = decoder(cfg, cases.random_state(cfg, 33), BF16, n_slots=2, max_len=64)
    with pytest.raises(ValueError):
        dec.feed(0, [1, 2], 63, [])
    with pytest.raises(ValueError):
        dec.feed(2, [1], 0, [])
    buf = dec.step_buffers(2)
    tokens, slot_map = torch.zeros(2, dtype=torch.long, device="cuda"), torch.tensor([0, 9], dtype=torch.int32, device="cuda")
    dec.run_step(tokens, torch.tensor([0, 0], dtype=torch.int32, device="cuda"), slot_map, buf)
    assert int(dec.status.item()) & 1


# ---- programs -------------------------------------------------------------------------------------------------------

@DTYPES
def test_trace_runner_and_command_line(tmp_path, dtype):
    cfg, state, toks, want = case("ragged", 90)
    cases.write_folder(tmp_path / "model", cfg, state)
    name = str(dtype).removeprefix("torch.")
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[50:52], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[52:53], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks[:1], "want": [0]}], "end": []},
             {"step": 4, "entries": [{"id": "b", "tokens": toks[1:90], "want": [88]}], "end": ["b"]}]
    out = tmp_path / "out"
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "model"), "--dtype", name, "--out", str(out),
                          "--max-tokens", "96"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(5)]
    for step, places in ((0, [0, 49]), (2, [52]), (3, [0]), (4, [89])):
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4")).view(len(places), cfg["vocab"])
        close(got, want[places], dtype)
    assert not (out / "1.f32").exists()
    if dtype == F32:
        prompt = toks[:12]
        run = subprocess.run([sys.executable, "-m", "nanochat_b200", "generate", "--model", str(tmp_path / "model"), "--dtype", name,
                              "--prompt", ",".join(map(str, prompt)), "--max-new-tokens", "5"], cwd=ROOT, capture_output=True, text=True,
                             timeout=600, env=dict(os.environ))
        assert run.returncode == 0, run.stderr[-2000:]
        assert json.loads(run.stdout.splitlines()[-1]) == {"prompt": 0, "tokens": greedy(cfg, state, prompt, 5)}
