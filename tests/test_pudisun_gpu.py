"""Pudisun on the GPU against the plain oracle (oracle/pudisun.py): each mechanism alone, whole prompts, portions, decoding,
batches, slots used again, generation through the scheduler, the command line and the trace runner."""

import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from nanochat_b200 import checkpoint, native
from nanochat_b200.hybrid import GEGLU, STORE, STORE_F32, STREAM, HybridConfig, HybridDecoder, HybridWeights, Stream
from nanochat_b200.mixers import GatedLinearAttention, LatentAttention, RowPlan, Rows, up
from nanochat_b200.serving import NativeDecoder, Request
from oracle import pudisun as oracle
from tests import pudisun_cases as cases

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
F32, BF16 = torch.float32, torch.bfloat16
# relative_error of logits or mixer outputs: fp32 rounding through a few layers, and bf16 products and activations (planted
# mistakes, tests/test_pudisun_cpu.py, all exceed the larger one)
TOLERANCE = {F32: 2e-5, BF16: 0.05}
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def decoder(cfg: dict, state: dict, dtype, n_slots=3, max_len=256, **kw) -> HybridDecoder:
    c = HybridConfig.from_pudisun(cfg, max_len)
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

def rows_of(slots, positions, dtype, status, plan=True, **kw) -> Rows:
    pos = torch.tensor(positions, dtype=torch.int32, device="cuda")
    slot_map = torch.tensor(slots, dtype=torch.int32, device="cuda")
    return Rows(len(slots), pos, slot_map, max(positions) + 1, status, RowPlan(slots, positions, "cuda") if plan else None, **kw)


def run_mixer(cls, entry, state, h, dtype, pieces, eps=1e-5, mode=None):
    """The mixer's output projection applied to its launches' output for h [n, C], run in `pieces` (row counts)."""
    columns = up(h.shape[1], 128)
    mixer = cls(entry["mixer"], {k[len("l0.mix."):]: v for k, v in state.items() if k.startswith("l0.mix.")}, eps, columns, dtype, "cuda")
    cache = mixer.new_cache(3, len(h))
    if cls is LatentAttention:
        cache.rows.fill_(float("nan"))  # what was never appended must not be read into a result
        if mode is not None:
            mixer.expands = lambda plan: mode == "expanded"
    else:
        cache.state.fill_(float("nan"))
        if mode is not None:
            mixer.CHUNKED_FROM = 1 if mode == "chunked" else 10 ** 9
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    x = torch.zeros((len(h), columns), dtype=dtype, device="cuda")
    x[:, :h.shape[1]] = h.to(dtype)
    got, at = [], 0
    for n in pieces:
        proj = (x[at:at + n].float() @ mixer.w_in.float().T).to(dtype)
        out = torch.zeros((n, mixer.out_width), dtype=dtype, device="cuda")
        mixer.run(proj, cache, rows_of([2] * n, list(range(at, at + n)), dtype, status, plan=n > 1), out)
        got.append(out.double() @ mixer.w_out.double().T)
        at += n
    assert int(status.item()) == 0
    return torch.cat(got)[:, :h.shape[1]]


LATENT_SIZES = {"ragged": cases.latent(), "one head": cases.latent(heads=1, dim=32, rot_dim=2, vdim=16, kv_rank=32, scale=1.0, scaling=None),
                "two head tiles": cases.latent(heads=18, dim=32, rot_dim=16, vdim=32, kv_rank=160),
                "rank 256": cases.latent(heads=4, dim=64, rot_dim=64, vdim=64, kv_rank=256),
                "rank 512": cases.latent(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=0.1),
                "beyond the tensor-core forms": cases.latent(heads=2, dim=224, rot_dim=32, vdim=160, kv_rank=704, scale=0.1)}


@DTYPES
@pytest.mark.parametrize("sizes", list(LATENT_SIZES))
@pytest.mark.parametrize("mode", ["absorbed", "expanded", "decoded"])
def test_latent_attention_alone(dtype, sizes, mode):
    entry = LATENT_SIZES[sizes]
    big = entry["mixer"]["kv_rank"] >= 512
    n, C = (70, 64) if big else (150, 64)
    state = cases.random_state(cases.config([entry], width=C), 7)
    h = torch.randn(n, C, generator=torch.Generator().manual_seed(8)).to(dtype)
    want = oracle.latent_attention(h.double(), oracle.part(state, "l0.mix."), entry["mixer"], 1e-5)
    if mode == "expanded":
        if dtype == F32 or entry["mixer"]["dim"] > 128:
            pytest.skip("no expanded form for these")
        got = run_mixer(LatentAttention, entry, state, h, dtype, [n - 67, 67], mode=mode)
    elif mode == "absorbed":
        got = run_mixer(LatentAttention, entry, state, h, dtype, [33, 2, n - 35], mode=mode)
    else:
        got = run_mixer(LatentAttention, entry, state, h, dtype, [1] * n)
    close(got, want, dtype)


@DTYPES
@pytest.mark.parametrize("mode", ["absorbed", "expanded", "decoded"])
def test_a_key_that_stands_out_is_found_wherever_it_lies(dtype, mode):
    """One earlier row's key is made to dominate a later row's score (same input, large scale), at tile, page and chunk
    borders, first and last positions; the outputs are those of the oracle."""
    if mode == "expanded" and dtype == F32:
        pytest.skip("no expanded form in 32-bit")
    entry = cases.latent(heads=2, dim=32, rot_dim=16, vdim=32, kv_rank=64, scale=1.5, scaling=None)
    C, n = 64, 200
    state = cases.random_state(cases.config([entry], width=C), 17)
    h = torch.randn(n, C, generator=torch.Generator().manual_seed(18))
    for key, query in ((0, 199), (31, 198), (32, 197), (63, 196), (64, 195), (127, 194), (128, 129), (191, 192), (150, 193)):
        h[key] *= 2.0  # only its direction counts for the key (the latent is normed), its size makes the query's scores sharp
        h[query] = h[key] + 0.1 * h[query]
    h = h.to(dtype)
    want = oracle.latent_attention(h.double(), oracle.part(state, "l0.mix."), entry["mixer"], 1e-5)
    pieces = {"absorbed": [64, 65, 71], "expanded": [64, 65, 71], "decoded": [120] + [1] * 80}[mode]
    got = run_mixer(LatentAttention, entry, state, h, dtype, pieces, mode="absorbed" if mode == "decoded" else mode)
    close(got, want, dtype)


GLA_SIZES = {"ragged": cases.gla(), "one": cases.gla(heads=1, dim=16, vdim=16, tau=1.0), "strong decay": cases.gla(heads=2, dim=48, vdim=32, tau=0.02),
             "long memory": cases.gla(heads=2, dim=32, vdim=64, tau=400.0), "wide": cases.gla(heads=2, dim=160, vdim=256, tau=16.0),
             "widest": cases.gla(heads=1, dim=272, vdim=96, tau=4.0), "value slices": cases.gla(heads=2, dim=64, vdim=1280, tau=4.0),
             "token by token only": cases.gla(heads=1, dim=528, vdim=32, tau=4.0)}


@DTYPES
@pytest.mark.parametrize("sizes", list(GLA_SIZES))
@pytest.mark.parametrize("mode", ["step", "chunked", "mixed"])
def test_gated_linear_attention_alone(dtype, sizes, mode):
    entry = GLA_SIZES[sizes]
    n, C = 150, 64
    state = cases.random_state(cases.config([entry], width=C), 27)
    h = torch.randn(n, C, generator=torch.Generator().manual_seed(28)).to(dtype)
    want = oracle.gated_linear_attention(h.double(), oracle.part(state, "l0.mix."), entry["mixer"], 1e-5)
    pieces = {"step": [40, 2, 1, 107], "chunked": [66, 2, 82], "mixed": [64, 1, 1, 2, 63, 19]}[mode]
    got = run_mixer(GatedLinearAttention, entry, state, h, dtype, pieces, mode=None if mode == "mixed" else mode)
    # a norm over few values of o amplifies rounding where they nearly cancel: the row error is taken over all rows' rms
    close(got, want, dtype)


@DTYPES
@pytest.mark.parametrize("rows", [1, 5, 16, 17, 40, 64, 65, 300])
def test_gemms_on_the_residual_stream(dtype, rows):
    """The four kernels (by rows) and their epilogues against fp32 torch: normed input, plain and fp32 store with a column
    limit, gated unit, stream update with what the next norm reads."""
    width, C, F, V = 300, 384, 256, 520
    cfg = HybridConfig(width=width, vocab=V, layers=[], eps=1e-3, residual_mult=0.3)
    dec = HybridDecoder.__new__(HybridDecoder)
    dec.cfg, dec.f32, dec.status = cfg, dtype == F32, torch.zeros(1, dtype=torch.int32, device="cuda")
    gen = torch.Generator(device="cuda").manual_seed(rows)

    def r(*shape, std=1.0, dt=dtype):
        return (torch.randn(*shape, generator=gen, device="cuda") * std).to(dt)

    embed, gain, gain2 = r(V, C), r(C, dt=F32), r(C, dt=F32)
    embed[:, width:], gain[width:], gain2[width:] = 0, 0, 0
    toks = torch.randint(0, V, (rows,), generator=gen, device="cuda")
    st = Stream(rows, C, dtype, "cuda")
    lib = native.cuda_library("decode_step")
    native.check(lib.embed_rs(*map(native.pointer, (embed, toks, st.h, gain, st.x, st.ss)), rows, C, V, int(dtype == F32), native.stream()), "")
    h = embed[toks].float()
    assert torch.equal(st.h, h)
    tol = 1e-5 if dtype == F32 else 2e-2

    def norm(h, g):
        return h / (h.square().sum(-1, keepdim=True) / width + 1e-3).sqrt() * g

    def same(got, want):
        err = (got.float() - want).abs().max() / want.abs().max()
        assert float(err) < tol, float(err)

    w = r(640, C, std=0.05)
    y = torch.full((rows, 648), 7.0, dtype=dtype, device="cuda")
    dec.gemm(rows, st.x, w, STORE, st, out=y, normed=True, n_store=600)
    same(y[:, :600], norm(h, gain) @ w.float().T[:, :600])
    assert (y[:, 600:] == 7).all()
    logits = torch.full((rows, V), 7.0, device="cuda")
    big = torch.zeros((640, C), dtype=dtype, device="cuda")
    big[:V] = embed
    dec.gemm(rows, st.x, big, STORE_F32, st, out=logits, normed=True, n_store=V, scale=0.25)
    same(logits, 0.25 * norm(h, gain) @ embed.float().T)
    u = torch.empty((rows, F), dtype=dtype, device="cuda")
    wu = r(2 * F, C, std=0.05)
    dec.gemm(rows, st.x, wu, GEGLU, st, out=u, normed=True)
    z = norm(h, gain) @ wu.float().T
    same(u, torch.nn.functional.gelu(z[:, 0::2], approximate="tanh") * z[:, 1::2])
    x, wo = r(rows, F), r(C, F, std=0.05)
    wo[width:] = 0
    dec.gemm(rows, x, wo, STREAM, st, gain=gain2)
    want = h + 0.3 * (x.float() @ wo.float().T)
    same(st.h, want)
    same(st.x, want * gain2)
    parts = st.ss.view(-1)[:rows * st.parts].view(rows, st.parts)
    same(parts.sum(-1), want.square().sum(-1))
    assert int(dec.status.item()) == 0


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
        for n in (1, 2, 3, 6):
            close(dec.feed(1, toks[:n], 0, list(range(n))), want[:n], dtype)
        for i, t in enumerate(toks):
            close(dec.feed(0, [t], i, [0]), want[i:i + 1], dtype)


@DTYPES
def test_long_prompts_far_keys_and_passes_of_a_prompt(dtype):
    """A prompt longer than any chunk, tile or page, in one pass and in several."""
    cfg = cases.config([cases.latent(heads=2, ff=None, scaling={**cases.YARN, "original": 256}), cases.gla(ff=96)], width=64, vocab=96)
    state, toks = cases.random_state(cfg, 9), cases.tokens(cfg, 700, 10)
    want = oracle.forward(toks, cfg, state)
    dec = decoder(cfg, state, dtype, max_len=720)
    every = list(range(len(toks)))
    close(dec.feed(0, toks, 0, every), want, dtype)
    close(dec.feed(1, toks, 0, every, rows_per_pass=256), want, dtype)
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


def greedy(cfg, state, prompt, n) -> list[int]:
    out = list(prompt)
    for _ in range(n):
        out.append(int(oracle.forward(out, cfg, state)[-1].argmax()))
    return out[len(prompt):]


def test_greedy_generation_through_the_scheduler_matches_the_oracle():
    """Seven requests through three slots (slots are freed and used again while others run), and generate(); 32-bit, where the
    choice is the oracle's."""
    cfg = cases.CONFIGS["ragged"]
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


def test_served_requests_do_not_depend_on_the_batch_and_prompts_come_from_the_store():
    """bf16: the same streams alone, in a full batch, sampled and greedy; a prompt seen before is copied from the store (rows
    of the latent layers, the state of the recurrent ones) instead of being prefilled."""
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
    assert checkpoint.read_config(tmp_path / "model") == cfg
    if dtype == F32:
        prompt = toks[:12]
        run = subprocess.run([sys.executable, "-m", "nanochat_b200", "generate", "--model", str(tmp_path / "model"), "--dtype", name,
                              "--prompt", ",".join(map(str, prompt)), "--max-new-tokens", "5"], cwd=ROOT, capture_output=True, text=True,
                             timeout=600, env=dict(os.environ))
        assert run.returncode == 0, run.stderr[-2000:]
        assert json.loads(run.stdout.splitlines()[-1]) == {"prompt": 0, "tokens": greedy(cfg, state, prompt, 5)}
