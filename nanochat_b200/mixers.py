"""Token mixers of models whose layers differ in kind: weights prepared for the kernels, the cache or state each needs, and
the launches between the input projection and the output projection. A mixer is built from its sizes and a dict of
checkpoint tensors, so any model whose layers use it can share it. A decoder only sees

    w_in, w_out                    fused input projection [in_width, C], output projection [C, out_width]
    new_cache(n_slots, max_len)    one layer's cache; its `parts` are what a prompt store copies
    kv_from                        the layer whose keys and values this one reads (None: its own); that layer's cache is then
                                   new_cache's third argument
    run(proj, cache, rows, out)    proj [rows, in_width] -> out [rows, out_width]; out None: only fill the cache

Sizes the kernels want as multiples (of 16, 32 or 128) are reached by zero-padding weights here: padded values are zero
everywhere they appear, so they change nothing, and no kernel has ragged edges."""

import functools
from dataclasses import dataclass, field

import numpy as np
import torch
from torch import Tensor

from .kv_cache import HeadCache, LatentCache, RingCache, StateCache
from .native import Conv, Delta, GemmRs, Gla, Gqa, Latent, check, cuda_library, pointer, stream
from .rotary import half_tables

LATENT_TILE = 32  # NCB_LATENT_TILE
GQA_TILE = 16     # NCB_GQA_TILE
SM_COUNT = 148


def up(n: int, multiple: int) -> int:
    return (n + multiple - 1) // multiple * multiple


def pad_to(t: Tensor, *shape: int) -> Tensor:
    """t with zeros appended to each axis up to `shape`."""
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def split_halves(t: Tensor, padded: int) -> Tensor:
    """Rows of a rotated part [.., dims, C] -> [.., padded, C] with each half at the start of its padded half."""
    half = t.shape[-2] // 2
    out = torch.zeros((*t.shape[:-2], padded, t.shape[-1]), dtype=t.dtype, device=t.device)
    out[..., :half, :] = t[..., :half, :]
    out[..., padded // 2:padded // 2 + half, :] = t[..., half:, :]
    return out


def stack_fields(fields: list[Tensor], width: int, columns: int) -> tuple[Tensor, list[int]]:
    """Fields [n_i, C] stacked into [width multiple, columns], each starting at a multiple of 8 rows; their offsets."""
    offsets, at = [], 0
    for f in fields:
        offsets.append(at)
        at += up(f.shape[0], 8)
    if at >= 1024:  # the widest tiles of tile_gemm take multiples of 256
        width = up(width, 256)
    out = torch.zeros((up(at, width), columns), dtype=fields[0].dtype, device=fields[0].device)
    for f, o in zip(fields, offsets):
        out[o:o + f.shape[0], :f.shape[1]] = f
    return out, offsets


class RowPlan:
    """The segments of one prefill pass (runs of rows of one slot at ascending positions) and their chunks for recurrent
    layers, on the device. Built once per pass, shared by the layers."""

    def __init__(self, slots, positions, device):
        slots, positions = np.asarray(slots, dtype=np.int32), np.asarray(positions, dtype=np.int32)
        n = len(slots)
        cut = np.ones(n, dtype=bool)
        cut[1:] = (slots[1:] != slots[:-1]) | (positions[1:] != positions[:-1] + 1)
        first = np.flatnonzero(cut).astype(np.int32)
        self.first, self.count = first, np.diff(np.append(first, n)).astype(np.int32)
        self.slots, self.starts, self.device = slots[first], positions[first], device
        self._on_device: dict = {}

    @property
    def n_segments(self) -> int:
        return len(self.first)

    @property
    def longest(self) -> int:
        return int(self.count.max())

    def upload(self, key, arrays: list[np.ndarray]) -> list[Tensor]:
        """The arrays on the device (one copy), kept under `key` for the pass's other layers."""
        if key not in self._on_device:
            flat = torch.from_numpy(np.concatenate([np.asarray(a, dtype=np.int32) for a in arrays])).to(self.device)
            self._on_device[key] = list(flat.split([len(a) for a in arrays]))
        return self._on_device[key]

    def segments(self) -> list[Tensor]:
        return self.upload("segments", [self.first, self.count])

    def contexts(self) -> list[Tensor]:
        """[segment's slot, first row of its context (n + 1)]: the contexts (all positions up to the segment's end) laid
        out one after the other."""
        return self.upload("contexts", [self.slots, np.concatenate([[0], np.cumsum(self.starts + self.count)])])

    def row_tiles(self, size: int) -> tuple[list[Tensor], int]:
        """([tile's first row, its rows, its context's first row, its first position], number of tiles) of at most `size`
        rows of one segment, those that reach furthest into their sequences first."""
        per = (self.count + size - 1) // size
        within = np.arange(per.sum(), dtype=np.int32) - np.repeat(np.cumsum(per) - per, per)
        first = np.repeat(self.first, per) + within * size
        rows = np.minimum(size, np.repeat(self.first + self.count, per) - first)
        context = np.repeat(np.cumsum(self.starts + self.count) - (self.starts + self.count), per)
        pos = np.repeat(self.starts, per) + within * size
        order = np.argsort(-pos.astype(np.int64), kind="stable")
        return self.upload(("tiles", size), [v[order] for v in (first, rows, context, pos)]), len(first)

    def chunks(self, size: int) -> tuple[list[Tensor], int]:
        """([segment's first chunk (n + 1), chunk's first row, chunk's rows, the segment's rows before it], number of chunks) for
        chunks of `size` rows."""
        per = (self.count + size - 1) // size
        base = np.concatenate([[0], np.cumsum(per)]).astype(np.int32)
        within = np.arange(base[-1], dtype=np.int32) - np.repeat(base[:-1], per)
        rows = np.repeat(self.first, per) + within * size
        count = np.minimum(size, np.repeat(self.first + self.count, per) - rows)
        return self.upload(("chunks", size), [base, rows, count, within * size]), int(base[-1])


@dataclass
class Rows:
    """The rows of one pass or decode step: positions and slots on the device, a bound of every position + 1, and the
    segments (None: a decode step, every row a slot of its own)."""
    n: int
    pos: Tensor
    slot_map: Tensor
    max_len: int
    status: Tensor
    plan: "RowPlan | None" = None
    chunk_tiles: int = 0
    scratch: dict = field(default_factory=dict)  # name -> tensor, reused by the layers of one pass

    def buffer(self, name: str, numel: int, dtype: torch.dtype, device) -> Tensor:
        t = self.scratch.get((name, dtype))
        if t is None or t.numel() < numel:
            t = self.scratch[(name, dtype)] = torch.empty(numel, dtype=dtype, device=device)
        return t


def padded_heads(w: Tensor, heads: int, size: int, padded: int) -> Tensor:
    """[heads size, n] -> [heads padded, n]: zero rows at the end of every head."""
    return pad_to(w.reshape(heads, size, -1), heads, padded, w.shape[-1]).reshape(heads * padded, -1)


class ShortConv:
    """The short causal convolution on the first channels of a mixer's projection: fields [(channels x taps weights or None where
    there are none, the field's offset)]; channels outside the fields are zero."""

    def __init__(self, fields: list, width: int, dtype: torch.dtype, device):
        self.width, self.dtype, self.device = width, dtype, torch.device(device)
        self.taps = max((w.shape[1] for w, _ in fields), default=1)
        self.w = torch.zeros((self.taps, width), dtype=torch.float32, device=device)
        for w, at in fields:
            if w.shape[1] != self.taps:
                raise ValueError(f"convolutions of {w.shape[1]} and {self.taps} taps in one layer")
            self.w[:, at:at + w.shape[0]] = w.float().T

    def new_ring(self, n_slots: int) -> RingCache:
        return RingCache(n_slots, self.taps, self.width, self.dtype, self.device)

    def args(self, proj: Tensor, ring: RingCache, rows: "Rows") -> Conv:
        return Conv(proj=proj.data_ptr(), ring=ring.rows.data_ptr(), w=self.w.data_ptr(), rows=rows.n, ldp=proj.stride(0),
                    taps=self.taps, width=self.width, n_slots=ring.n_slots, pos=rows.pos.data_ptr(),
                    slot_map=rows.slot_map.data_ptr())

    def keep_tail(self, conv: Conv, rows: "Rows") -> None:
        """After a pass of several rows per slot; a decode step's kernels keep their rows themselves."""
        if rows.plan is not None:
            check(cuda_library("short_conv").short_conv_tail(pointer_to(conv), int(self.dtype == torch.float32),
                                                             pointer(rows.status), stream()), "short_conv_tail")


@dataclass
class AttentionCache:
    kv: HeadCache
    ring: RingCache
    own: bool

    @property
    def parts(self) -> list:
        return [self.kv, self.ring] if self.own else [self.ring]


@dataclass
class RecurrentCache:
    state: StateCache
    ring: RingCache

    @property
    def parts(self) -> list:
        return [self.state, self.ring]


class GroupedAttention:
    """Softmax attention of grouped query heads: short convolutions, rotation, norm of queries and keys, a gate per head
    (csrc/gqa_attn.cu). sizes: heads, kv_heads, dim, vdim, scale, rot (dims, base, scaling; may be absent), kv_from. tensors: q,
    q.conv, g, o and, unless another layer's are read, k, k.conv, v, v.conv."""

    def __init__(self, sizes: dict, tensors: dict, eps: float, columns: int, dtype: torch.dtype, device):
        H, G, D, V = (int(sizes[n]) for n in ("heads", "kv_heads", "dim", "vdim"))
        if H % G:
            raise ValueError(f"{H} query heads over {G} key/value heads")
        self.heads, self.kv_heads, self.true_dim, self.rot_spec = H, G, D, sizes.get("rot")
        self.rot = int(self.rot_spec["dims"]) if self.rot_spec else 0
        if self.rot % 2 or self.rot > D:
            raise ValueError(f"rotation of {self.rot} of {D} dimensions")
        self.dim, self.vdim, self.kv_from = up(D, 16), up(V, 16), sizes.get("kv_from")
        self.scale, self.eps, self.dtype, self.device = float(sizes["scale"]), float(eps), dtype, torch.device(device)
        t = {k: v.to(device) for k, v in tensors.items()}
        heads = [("q", H, D, self.dim)] + ([("k", G, D, self.dim), ("v", G, V, self.vdim)] if self.kv_from is None else [])
        fields = [padded_heads(t[n], h, d, p).to(dtype) for n, h, d, p in heads] + [t["g"].to(dtype)]
        self.w_in, offsets = stack_fields(fields, 128, columns)
        self.off_q, self.off_g = offsets[0], offsets[-1]
        self.off_k, self.off_v = offsets[1:3] if self.kv_from is None else (0, 0)
        self.conv = ShortConv([(padded_heads(t[n + ".conv"], h, d, p), at) for (n, h, d, p), at in zip(heads, offsets)], self.off_g,
                              dtype, device)
        o = pad_to(t["o"].reshape(-1, H, V), columns, H, self.vdim).reshape(columns, H * self.vdim)
        self.out_width = up(H * self.vdim, 128)
        self.w_out = pad_to(o, columns, self.out_width).to(dtype)
        self.in_width = self.w_in.shape[0]
        self.tables: "tuple[Tensor, Tensor] | None" = None
        self._chunks: dict[tuple[int, int], int] = {}
        lib, bf = cuda_library("gqa_attn"), dtype == torch.bfloat16
        self.fused = bf and bool(lib.gqa_split_fused(self.dim, self.vdim))
        self.tiled = bf and bool(lib.gqa_prefill_supported(self.dim, self.vdim))

    ROW_TILE = 64     # rows per tile of gqa_prefill
    TILED_FROM = 8    # shorter segments run as rows on their own

    def new_cache(self, n_slots: int, max_len: int, of: "AttentionCache | None" = None) -> AttentionCache:
        if (of is None) != (self.kv_from is None):
            raise ValueError("a layer reads its own keys and values or another layer's")
        kv = HeadCache(n_slots, self.kv_heads, self.dim + self.vdim, max_len, self.dtype, self.device) if of is None else of.kv
        if kv.width != self.dim + self.vdim or kv.kv_heads != self.kv_heads:
            raise ValueError("layers that share keys and values differ in their heads")
        if self.rot and (self.tables is None or self.tables[0].shape[0] < kv.capacity):
            self.tables = shared_tables(kv.capacity, self.rot, float(self.rot_spec["base"]),
                                        tuple(sorted((self.rot_spec.get("scaling") or {}).items())), self.device)
        return AttentionCache(kv, self.conv.new_ring(n_slots), of is None)

    @staticmethod
    def cache_bytes(sizes: dict, max_len: int, itemsize: int) -> int:
        H, G, dim, vdim = int(sizes["heads"]), int(sizes["kv_heads"]), up(int(sizes["dim"]), 16), up(int(sizes["vdim"]), 16)
        own = sizes.get("kv_from") is None
        ring = int(sizes.get("conv", 1)) * (H * dim + (G * (dim + vdim) if own else 0))
        return (ring + (up(max_len, 64) * G * (dim + vdim) if own else 0)) * itemsize

    def chunk_for(self, lens: "list[int]", most: int) -> int:
        """Tiles per chunk of the split kernel for rows of these lengths, at most 128 chunks for `most` positions: enough blocks
        to fill the GPU twice over, chunks long enough to be worth a state."""
        tiles = np.maximum((np.asarray(lens, dtype=np.int64) + GQA_TILE - 1) // GQA_TILE, 1)
        top, least = int(tiles.max()), max(8, ((most + GQA_TILE - 1) // GQA_TILE + 127) // 128)
        per_chunk = self.kv_heads * ((self.heads // self.kv_heads + 15) // 16)
        best, cost = least, float("inf")
        c = least
        while c < 2 * max(top, least):
            blocks = int(((tiles + c - 1) // c).sum()) * per_chunk
            now = -(-blocks // (2 * SM_COUNT)) * (min(c, top) + 8.0)
            if now < cost:
                best, cost = c, now
            c += max(1, c // 8)
        return best

    def default_chunk(self, rows: int, max_len: int) -> int:
        if (rows, max_len) not in self._chunks:
            self._chunks[rows, max_len] = self.chunk_for([max_len] * rows, max_len)
        return self._chunks[rows, max_len]

    def run(self, proj: Tensor, cache: AttentionCache, rows: Rows, out: "Tensor | None") -> None:
        n, f32, lib, kv = rows.n, int(self.dtype == torch.float32), cuda_library("gqa_attn"), cache.kv
        a = Gqa(conv=self.conv.args(proj, cache.ring, rows), kv=kv.rows.data_ptr(), off_q=self.off_q, off_k=self.off_k, off_v=self.off_v,
                off_g=self.off_g, own_kv=int(cache.own), keep=int(rows.plan is None and self.conv.taps > 1), heads=self.heads,
                kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, norm_count=self.true_dim, rot=self.rot, capacity=kv.capacity,
                table_len=kv.capacity, scale=self.scale, eps=self.eps, status=rows.status.data_ptr())
        if self.rot:
            a.cos, a.sin = (t.data_ptr() for t in self.tables)
        fused = self.fused and rows.plan is None and out is not None
        if not fused:
            if out is not None:
                a.q = rows.buffer("gqa_q", n * self.heads * self.dim, self.dtype, self.device).data_ptr()
            check(lib.gqa_rows(pointer_to(a), f32, stream()), "gqa_rows")
        if out is not None:
            a.out, a.ldo = out.data_ptr(), out.stride(0)
        if out is not None and self.tiled and rows.plan is not None and rows.plan.longest >= self.TILED_FROM:
            tiles, a.n_tiles = rows.plan.row_tiles(self.ROW_TILE)
            a.tile_row, a.tile_rows, a.tile_pos = (tiles[i].data_ptr() for i in (0, 1, 3))
            check(lib.gqa_prefill(pointer_to(a), stream()), "gqa_prefill")
        elif out is not None:
            max_len = min(rows.max_len, kv.capacity)
            tiles = (max_len + GQA_TILE - 1) // GQA_TILE
            a.max_len, a.chunk_tiles = max_len, rows.chunk_tiles or self.default_chunk(n, max_len)
            a.max_chunks = (tiles + a.chunk_tiles - 1) // a.chunk_tiles
            a.parts = rows.buffer("gqa_parts", n * self.heads * a.max_chunks * (self.vdim + 4), torch.float32, self.device).data_ptr()
            check(lib.gqa_split(pointer_to(a), f32, stream()), "gqa_split")
            check(lib.gqa_merge(pointer_to(a), f32, stream()), "gqa_merge")
        self.conv.keep_tail(a.conv, rows)


class ChannelDelta:
    """Gated delta rule with a decay per key channel, short convolutions, per-head output norm and a low-rank sigmoid gate
    (csrc/delta_rule.cu). sizes: heads, kv_heads, dim, vdim. tensors: q, k, v and their .conv, b, A_log, a1, a2, dt_bias, g1, g2,
    norm, o."""

    kv_from = None
    CHUNKED_FROM = 24  # shorter segments run token by token

    def __init__(self, sizes: dict, tensors: dict, eps: float, columns: int, dtype: torch.dtype, device):
        H, G, D, V = (int(sizes[n]) for n in ("heads", "kv_heads", "dim", "vdim"))
        if H % G:
            raise ValueError(f"{H} value heads over {G} query/key heads")
        self.heads, self.kv_heads, self.true_vdim = H, G, V
        self.dim, self.vdim, self.q_scale = up(D, 16), up(V, 16), float(D) ** -0.5
        self.eps, self.dtype, self.device = float(eps), dtype, torch.device(device)
        t = {k: v.to(device) for k, v in tensors.items()}
        heads = [("q", G, D, self.dim), ("k", G, D, self.dim), ("v", H, V, self.vdim)]
        fields = [padded_heads(t[n], h, d, p).to(dtype) for n, h, d, p in heads] + [t["b"].to(dtype)] + \
            [pad_to(t[n], up(t[n].shape[0], 16), t[n].shape[1]).to(dtype) for n in ("a1", "g1")]
        self.w_in, self.offsets = stack_fields(fields, 128, columns)
        self.conv = ShortConv([(padded_heads(t[n + ".conv"], h, d, p), at) for (n, h, d, p), at in zip(heads, self.offsets)],
                              self.offsets[3], dtype, device)
        self.rank_a, self.rank_g = (up(t[n].shape[0], 16) for n in ("a1", "g1"))
        self.a2_rows = pad_to(t["a2"].reshape(H, D, -1), H, self.dim, self.rank_a).to(dtype)
        self.g2_rows = pad_to(t["g2"].reshape(H, V, -1), H, self.vdim, self.rank_g).to(dtype)
        self.a2, self.g2 = (w.transpose(1, 2).contiguous() for w in (self.a2_rows, self.g2_rows))
        self.chunk = cuda_library("delta_rule").delta_chunk_tokens(self.dim, self.vdim, self.conv.taps, self.rank_a, self.rank_g) if dtype == torch.bfloat16 else 0
        self.dt_bias = pad_to(t["dt_bias"].float().reshape(H, D), H, self.dim).contiguous()
        self.a_exp = t["A_log"].float().exp()
        self.norm = pad_to(t["norm"].float(), self.vdim)
        o = pad_to(t["o"].reshape(-1, H, V), columns, H, self.vdim).reshape(columns, H * self.vdim)
        self.out_width = up(H * self.vdim, 128)
        self.w_out = pad_to(o, columns, self.out_width).to(dtype)
        self.in_width = self.w_in.shape[0]

    def new_cache(self, n_slots: int, max_len: int, of: None = None) -> RecurrentCache:
        return RecurrentCache(StateCache(n_slots, self.heads, self.dim, self.vdim, device=self.device), self.conv.new_ring(n_slots))

    @staticmethod
    def cache_bytes(sizes: dict, max_len: int, itemsize: int) -> int:
        H, G, dim, vdim = int(sizes["heads"]), int(sizes["kv_heads"]), up(int(sizes["dim"]), 16), up(int(sizes["vdim"]), 16)
        return H * dim * vdim * 4 + int(sizes.get("conv", 1)) * (2 * G * dim + H * vdim) * itemsize

    def run(self, proj: Tensor, cache: RecurrentCache, rows: Rows, out: "Tensor | None") -> None:
        f32, lib, plan = int(self.dtype == torch.float32), cuda_library("delta_rule"), rows.plan
        a = Delta(conv=self.conv.args(proj, cache.ring, rows), out=None if out is None else out.data_ptr(),
                  ldo=0 if out is None else out.stride(0), keep=int(plan is None and self.conv.taps > 1), heads=self.heads,
                  kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, rank_a=self.rank_a, rank_g=self.rank_g,
                  norm_count=self.true_vdim, q_scale=self.q_scale, eps=self.eps, a2=self.a2.data_ptr(), g2=self.g2.data_ptr(),
                  dt_bias=self.dt_bias.data_ptr(), a_exp=self.a_exp.data_ptr(), norm=self.norm.data_ptr(),
                  state=cache.state.state.data_ptr(), status=rows.status.data_ptr())
        a.off_q, a.off_k, a.off_v, a.off_b, a.off_a, a.off_g = self.offsets
        if plan is not None:
            first, count = plan.segments()
            a.seg_first, a.seg_count, a.n_segments = first.data_ptr(), count.data_ptr(), plan.n_segments
        if plan is None or self.chunk == 0 or plan.longest < self.CHUNKED_FROM:
            check(lib.delta_step(pointer_to(a), f32, stream()), "delta_step")
        else:
            self.run_chunked(a, rows)
        self.conv.keep_tail(a.conv, rows)

    def run_chunked(self, a: Delta, rows: Rows) -> None:
        arrays, n = rows.plan.chunks(self.chunk)
        a.seg_chunk, a.chunk_first, a.chunk_count, a.chunk_within = (t.data_ptr() for t in arrays)
        a.n_chunks, a.chunk, a.a2_rows, a.g2_rows = n, self.chunk, self.a2_rows.data_ptr(), self.g2_rows.data_ptr()
        C, D, V, each, bf, f = self.chunk, self.dim, self.vdim, n * self.heads, torch.bfloat16, torch.float32
        for name, size, kind in (("w_terms", 2 * C * (D + 8), bf), ("kd_terms", 2 * C * (D + 8), bf), ("q_terms", 2 * C * (D + 8), bf),
                                 ("b_terms", 2 * C * (C + 8), bf), ("s_terms", 2 * V * (D + 8), bf), ("u_terms", 2 * V * (C + 8), bf),
                                 ("u0", V * (C + 4), f), ("chunk_decay", D, f)):
            setattr(a, name, rows.buffer("delta_" + name, each * size, kind, self.device).data_ptr())
        # values beyond one tile of the output kernel pass through memory for the norm
        a.raw = rows.buffer("delta_raw", rows.n * self.heads * V if V > 128 else 4, f, self.device).data_ptr()
        check(cuda_library("delta_rule").delta_chunked(pointer_to(a), stream()), "delta_chunked")


class GatedLinearAttention:
    """Linear attention with a decay per key channel, per-head output norm and silu gate (csrc/gla.cu).
    sizes: heads, dim, vdim, tau. tensors: q, k, v, g, o, a1, a2, a2.b, norm."""

    kv_from = None
    CHUNKED_FROM = 24  # shorter segments run token by token

    def __init__(self, sizes: dict, tensors: dict, eps: float, columns: int, dtype: torch.dtype, device):
        H, D, V = int(sizes["heads"]), int(sizes["dim"]), int(sizes["vdim"])
        self.heads, self.true_vdim, self.eps, self.dtype, self.device = H, V, float(eps), dtype, torch.device(device)
        self.dim, self.vdim = up(D, 16), up(V, 16)
        self.q_scale, self.inv_tau = float(D) ** -0.5, 1.0 / float(sizes["tau"])
        t = {k: v.to(device) for k, v in tensors.items()}
        C = t["q"].shape[1]

        def per_head(w: Tensor, n: int, padded: int) -> Tensor:
            return pad_to(w.reshape(H, n, C), H, padded, C).reshape(H * padded, C).to(dtype)

        self.rank = t["a1"].shape[0]
        fields = [per_head(t["q"], D, self.dim), per_head(t["k"], D, self.dim), per_head(t["v"], V, self.vdim),
                  per_head(t["g"], V, self.vdim), t["a1"].to(dtype)]
        self.w_in, self.offsets = stack_fields(fields, 128, columns)
        self.a2 = pad_to(t["a2"].float().reshape(H, D, self.rank), H, self.dim, self.rank).contiguous()
        self.a2_bias = pad_to(t["a2.b"].float().reshape(H, D), H, self.dim).contiguous()
        self.norm = pad_to(t["norm"].float(), self.vdim)
        o = pad_to(t["o"].reshape(-1, H, V), columns, H, self.vdim).reshape(columns, H * self.vdim)
        self.out_width = up(H * self.vdim, 128)
        self.w_out = pad_to(o, columns, self.out_width).to(dtype)
        self.in_width = self.w_in.shape[0]
        self.chunk = cuda_library("gla").gla_chunk_tokens(self.dim)

    def new_cache(self, n_slots: int, max_len: int, of: None = None) -> StateCache:
        return StateCache(n_slots, self.heads, self.dim, self.vdim, device=self.device)

    @staticmethod
    def cache_bytes(sizes: dict, max_len: int, itemsize: int) -> int:
        return int(sizes["heads"]) * up(int(sizes["dim"]), 16) * up(int(sizes["vdim"]), 16) * 4

    def run(self, proj: Tensor, cache: StateCache, rows: Rows, out: "Tensor | None") -> None:
        n, f32 = rows.n, int(self.dtype == torch.float32)
        a = Gla(proj=proj.data_ptr(), out=None if out is None else out.data_ptr(), rows=n, ldp=proj.stride(0),
                ldo=0 if out is None else out.stride(0), heads=self.heads, dim=self.dim, vdim=self.vdim, rank=self.rank,
                norm_count=self.true_vdim, n_slots=cache.n_slots, q_scale=self.q_scale, inv_tau=self.inv_tau, eps=self.eps,
                a2=self.a2.data_ptr(), a2_bias=self.a2_bias.data_ptr(), norm=self.norm.data_ptr(),
                state=cache.state.data_ptr(), pos=rows.pos.data_ptr(), slot_map=rows.slot_map.data_ptr(),
                status=rows.status.data_ptr())
        a.off_q, a.off_k, a.off_v, a.off_g, a.off_a = self.offsets
        lib, plan = cuda_library("gla"), rows.plan
        if plan is not None:
            first, count = plan.segments()
            a.seg_first, a.seg_count, a.n_segments = first.data_ptr(), count.data_ptr(), plan.n_segments
        if plan is None or self.chunk == 0 or plan.longest < self.CHUNKED_FROM:
            check(lib.gla_step(pointer_to(a), f32, stream()), "gla_step")
            return
        (seg_chunk, chunk_first, chunk_count, _), n_chunks = plan.chunks(self.chunk)
        HD, HV, f = self.heads * self.dim, self.heads * self.vdim, torch.float32
        a.seg_chunk, a.chunk_first, a.chunk_count = seg_chunk.data_ptr(), chunk_first.data_ptr(), chunk_count.data_ptr()
        a.n_chunks, a.chunk = n_chunks, self.chunk
        a.decay = rows.buffer("gla_decay", n * HD, f, self.device).data_ptr()
        a.chunk_decay = rows.buffer("gla_chunk_decay", n_chunks * HD, f, self.device).data_ptr()
        a.states = rows.buffer("gla_states", n_chunks * HD * self.vdim, f, self.device).data_ptr()
        a.raw = rows.buffer("gla_raw", n * HV, f, self.device).data_ptr()
        check(lib.gla_chunked(pointer_to(a), f32, stream()), "gla_chunked")


class LatentAttention:
    """Attention over a cache of latent rows shared by the heads (csrc/latent_attn.cu).
    sizes: heads, dim, rot_dim, vdim, kv_rank, scale, rot (dims, base, scaling). tensors: q, dkv, dkv.norm, uk, uv, o and
    optionally g (output gate) and sink."""

    kv_from = None

    def __init__(self, sizes: dict, tensors: dict, eps: float, columns: int, dtype: torch.dtype, device):
        H, D, R = int(sizes["heads"]), int(sizes["dim"]), int(sizes["rot_dim"])
        V, rank, rot = int(sizes["vdim"]), int(sizes["kv_rank"]), sizes["rot"]
        if int(rot["dims"]) != R or R % 2:
            raise ValueError(f"the rotated part has {R} dimensions, rot.dims is {rot['dims']}: they have to be equal and even")
        self.heads, self.rank_count, self.rot, self.rot_spec = H, rank, up(R, 16), rot
        self.dim, self.vdim, self.rank = up(D, 32), up(V, 16), up(rank, 32)
        self.scale, self.eps, self.dtype, self.device = float(sizes["scale"]), float(eps), dtype, torch.device(device)
        t = {k: v.to(device) for k, v in tensors.items()}
        C = t["q"].shape[1]
        q = t["q"].reshape(H, D + R, C)
        q = torch.cat([pad_to(q[:, :D], H, self.dim, C), split_halves(q[:, D:], self.rot)], 1).reshape(-1, C)
        kv = torch.cat([pad_to(t["dkv"][:rank], self.rank, C), split_halves(t["dkv"][rank:], self.rot)], 0)
        fields = [q.to(dtype), kv.to(dtype)]
        self.gated = "g" in t
        if self.gated:
            fields.append(pad_to(t["g"].reshape(H, V, C), H, self.vdim, C).reshape(-1, C).to(dtype))
        self.w_in, offsets = stack_fields(fields, 128, columns)
        self.off_q, self.off_kv, self.off_g = offsets[0], offsets[1], offsets[2] if self.gated else 0
        self.norm = pad_to(t["dkv.norm"].float(), self.rank)
        uk = pad_to(t["uk"].reshape(H, D, rank), H, self.dim, self.rank)
        uv = pad_to(t["uv"].reshape(H, V, rank), H, self.vdim, self.rank)
        self.expanded = dtype == torch.bfloat16 and bool(
            cuda_library("latent_attn").latent_prefill_supported(self.dim, self.rot, self.vdim))
        if self.expanded:  # both expansions of a latent row as one GEMM: per head the key's rows, then the value's
            both = torch.cat([uk, uv], 1).reshape(H * (self.dim + self.vdim), self.rank)
            self.w_ukv = pad_to(both, up(both.shape[0], 128), up(self.rank, 64)).to(dtype)
        self.w_uk_t = uk.transpose(1, 2).contiguous().to(dtype)
        self.w_uv = uv.contiguous().to(dtype)
        self.sink = t["sink"].float().contiguous() if "sink" in t else None
        o = pad_to(t["o"].reshape(-1, H, V), columns, H, self.vdim).reshape(columns, H * self.vdim)
        self.out_width = up(H * self.vdim, 128)
        self.w_out = pad_to(o, columns, self.out_width).to(dtype)
        self.in_width = self.w_in.shape[0]
        self.tables: "tuple[Tensor, Tensor] | None" = None
        self._chunks: dict[tuple[int, int], int] = {}

    def new_cache(self, n_slots: int, max_len: int, of: None = None) -> LatentCache:
        cache = LatentCache(n_slots, self.rank + self.rot, max_len, self.dtype, device=self.device)
        if self.tables is None or self.tables[0].shape[0] < cache.capacity:
            self.tables = half_tables(cache.capacity, int(self.rot_spec["dims"]), float(self.rot_spec["base"]),
                                      self.rot_spec.get("scaling"), self.rot, self.device)
        return cache

    @staticmethod
    def cache_bytes(sizes: dict, max_len: int, itemsize: int) -> int:
        return up(max_len, 64) * (up(int(sizes["kv_rank"]), 32) + up(int(sizes["rot_dim"]), 16)) * itemsize

    def chunk_for(self, lens: "list[int]", most: int) -> int:
        """Tiles per chunk of the split kernel for rows of these lengths: the size with the least modelled time, waves of the
        blocks that fit the GPU (two per SM) times a block's tiles plus a fixed cost. At most 128 chunks for `most` positions
        (a bound of every length)."""
        tiles = np.maximum((np.asarray(lens, dtype=np.int64) + LATENT_TILE - 1) // LATENT_TILE, 1)
        top, least = int(tiles.max()), max(2, ((most + LATENT_TILE - 1) // LATENT_TILE + 127) // 128)
        best, cost = least, float("inf")
        for c in range(least, max(top, least) + 1):
            blocks = int(((tiles + c - 1) // c).sum()) * ((self.heads + 15) // 16)
            now = -(-blocks // (2 * SM_COUNT)) * (min(c, top) + 2.0)
            if now < cost:
                best, cost = c, now
        return best

    def default_chunk(self, rows: int, max_len: int) -> int:
        """chunk_for rows that all have max_len positions, remembered (it only depends on these)."""
        if (rows, max_len) not in self._chunks:
            self._chunks[rows, max_len] = self.chunk_for([max_len] * rows, max_len)
        return self._chunks[rows, max_len]

    ROW_TILE = 64  # rows per tile of latent_prefill

    def expands(self, plan: RowPlan) -> bool:
        """Whether a pass is cheaper with expanded keys and values: expanding every context once and attending in head
        space, against attending in latent space (whose kernel reads the cache once per row and head tile)."""
        if not self.expanded:
            return False
        count, length = plan.count.astype(np.float64), (plan.starts + plan.count).astype(np.float64)
        pairs = float((count * (length - count / 2)).sum())
        expanded = float(length.sum()) * self.rank * (self.dim + self.vdim) + pairs * (self.dim + self.rot + self.vdim)
        return expanded < 2.0 * pairs * (2 * self.rank + self.rot)

    def run_expanded(self, a: Latent, rows: Rows) -> None:
        plan, lib, bf = rows.plan, cuda_library("latent_attn"), torch.bfloat16
        n_ctx = int((plan.starts + plan.count).sum())
        (slots, first), (tiles, a.n_tiles) = plan.contexts(), plan.row_tiles(self.ROW_TILE)
        N, K = self.w_ukv.shape
        a.rotate_q, a.max_len, a.n_contexts = 1, int((plan.starts + plan.count).max()), plan.n_segments
        a.ctx_slot, a.ctx_first = slots.data_ptr(), first.data_ptr()
        a.tile_row, a.tile_rows, a.tile_ctx, a.tile_pos = (t.data_ptr() for t in tiles)
        a.ctx_ld, a.ctx_kv_ld = K, N
        a.ctx = rows.buffer("latent_ctx", n_ctx * K, bf, self.device).data_ptr()
        a.ctx_rot = rows.buffer("latent_ctx_rot", n_ctx * self.rot, bf, self.device).data_ptr()
        a.ctx_kv = rows.buffer("latent_ctx_kv", n_ctx * N, bf, self.device).data_ptr()
        check(lib.latent_append(pointer_to(a), 0, stream()), "latent_append")
        check(lib.latent_gather(pointer_to(a), stream()), "latent_gather")
        g = GemmRs(x=a.ctx, w=self.w_ukv.data_ptr(), y=a.ctx_kv, rows=n_ctx, ldy=N, N=N, K=K, n_store=N, epilogue=0, scale=1.0,
                   status=a.status)
        check(cuda_library("tile_gemm").tile_gemm_rs(pointer_to(g), stream()), "tile_gemm_rs")
        check(lib.latent_prefill(pointer_to(a), stream()), "latent_prefill")

    def run(self, proj: Tensor, cache: LatentCache, rows: Rows, out: "Tensor | None") -> None:
        n, f32, lib = rows.n, int(self.dtype == torch.float32), cuda_library("latent_attn")
        cos, sin = self.tables
        a = Latent(proj=proj.data_ptr(), cache=cache.rows.data_ptr(), rows=n, ldp=proj.stride(0), off_q=self.off_q,
                   off_kv=self.off_kv, off_g=self.off_g, gated=int(self.gated), rotate_q=0, heads=self.heads, dim=self.dim,
                   rot=self.rot, vdim=self.vdim, rank=self.rank, norm_count=self.rank_count, n_slots=cache.n_slots,
                   capacity=cache.capacity, table_len=cos.shape[0], scale=self.scale, eps=self.eps,
                   norm=self.norm.data_ptr(), cos=cos.data_ptr(), sin=sin.data_ptr(),
                   sink=None if self.sink is None else self.sink.data_ptr(), pos=rows.pos.data_ptr(),
                   slot_map=rows.slot_map.data_ptr(), status=rows.status.data_ptr())
        if out is None:
            check(lib.latent_append(pointer_to(a), f32, stream()), "latent_append")
            return
        max_len = min(rows.max_len, cache.capacity)
        a.out, a.ldo = out.data_ptr(), out.stride(0)
        if rows.plan is not None and self.expands(rows.plan):
            self.run_expanded(a, rows)
            return
        tiles = (max_len + LATENT_TILE - 1) // LATENT_TILE
        a.max_len, a.chunk_tiles = max_len, rows.chunk_tiles or self.default_chunk(n, max_len)
        a.max_chunks = (tiles + a.chunk_tiles - 1) // a.chunk_tiles
        a.w_uk_t, a.w_uv = self.w_uk_t.data_ptr(), self.w_uv.data_ptr()
        a.q_abs = rows.buffer("latent_q", n * self.heads * (self.rank + self.rot), self.dtype, self.device).data_ptr()
        a.parts = rows.buffer("latent_parts", n * self.heads * a.max_chunks * (self.rank + 4), torch.float32,
                              self.device).data_ptr()
        check(lib.latent_query(pointer_to(a), f32, stream()), "latent_query")
        check(lib.latent_split(pointer_to(a), f32, stream()), "latent_split")
        check(lib.latent_out(pointer_to(a), f32, stream()), "latent_out")


@functools.lru_cache(maxsize=4)
def shared_tables(positions: int, dims: int, base: float, scaling: tuple, device) -> tuple[Tensor, Tensor]:
    """half_tables, one pair for all layers of a kind."""
    return half_tables(positions, dims, base, dict(scaling) or None, dims, device)


def pointer_to(struct):
    import ctypes

    return ctypes.byref(struct)


MIXERS = {"latent_attention": LatentAttention, "gla": GatedLinearAttention, "attention": GroupedAttention,
          "channel_delta": ChannelDelta}
