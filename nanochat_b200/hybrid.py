"""Decoder for models whose layers differ in kind: each layer a mixer (mixers.MIXERS) and optionally a gated feed-forward,
pre-norm, around a residual stream kept in fp32. Layers may share another layer's weights with a cache of their own, or read
another layer's keys and values. In place of the one stream there may be several with hyper-connections: a branch reads a
weighted sum of them, and its result and the old streams make the new ones (HyperConnection).

One layer is
    input projection (norm as a row scale) -> mixer's launches -> output projection, stream update ->
    gate / up projection with the gated unit in its epilogue -> down projection, stream update
and every GEMM that ends a branch also writes what the next norm needs (the gained stream and partial sums of squares), so
there are no norm launches. The same sequence runs a decode step (one row per slot, captured in a graph) and a prefill pass
(rows of prompts); only the GEMM kernel (by rows, as in decoder.py) and the mixers' kernels differ. dtype float32 runs
everything in 32-bit on gemm_f32 and the mixers' fp32 forms."""

import ctypes
from dataclasses import dataclass

import torch
from torch import Tensor

from .decoder import StepDecoder
from .kv_cache import cache_pages
from .mixers import MIXERS, RowPlan, Rows, pad_to, up
from .native import MAX_STREAMS, GemmRs, check, cuda_library, pointer, stream
from .prompt_store import PromptStore

STORE, STORE_F32, GEGLU, STREAM, STREAMS, SWIGLU = 0, 3, 5, 6, 7, 8


@dataclass(frozen=True)
class LayerSpec:
    """One layer: the kind of mixer and its sizes, the feed-forward's width (0: none), and whose weights it uses."""
    kind: str
    mixer: dict
    ff: int
    weights_of: int


@dataclass
class HybridConfig:
    width: int
    vocab: int
    layers: list[LayerSpec]
    eps: float
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    max_len: int = 1024
    itemsize: int = 2  # bytes of a cached value
    streams: int = 0   # streams with hyper-connections; 0: one plain residual stream
    embed_scale: float = 1.0
    tied_head: bool = True      # the head is the embedding; else the checkpoint's "head"
    norm_base: float = 0.0      # norms multiply by norm_base + weight
    unit: int = GEGLU           # the feed-forward's gated unit: GEGLU or SWIGLU

    @staticmethod
    def from_pudisun(config: dict, max_len: int) -> "HybridConfig":
        """From the config.json of a Pudisun model."""
        layers = []
        for i, entry in enumerate(config["layers"]):
            kind, mlp, of = entry["type"], entry.get("mlp"), int(entry.get("weights_of", i))
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: no mixer '{kind}' (known: {', '.join(sorted(MIXERS))})")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: no feed-forward '{mlp['kind']}'")
            if not 0 <= of < len(config["layers"]) or "weights_of" in config["layers"][of]:
                raise ValueError(f"layer {i}: weights of layer {of}, which has none of its own")
            layers.append(LayerSpec(kind, entry["mixer"], 0 if mlp is None else int(mlp["ff"]), of))
        return HybridConfig(width=int(config["width"]), vocab=int(config["vocab"]), layers=layers,
                            eps=float(config["norm"]["eps"]), residual_mult=float(config["residual_mult"]),
                            logit_scale=float(config["logit_scale"]), max_len=max_len)

    @staticmethod
    def from_rekudra(config: dict, max_len: int) -> "HybridConfig":
        """From the config.json of a Rekudra model."""
        entries, layers = config["layers"], []
        for i, entry in enumerate(entries):
            kind, mixer, mlp = entry["type"], entry["mixer"], entry.get("mlp")
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: no mixer '{kind}' (known: {', '.join(sorted(MIXERS))})")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: no feed-forward '{mlp['kind']}'")
            of = mixer.get("kv_from")
            if of is not None and not (0 <= of < i and entries[of]["type"] == kind and entries[of]["mixer"].get("kv_from") is None):
                raise ValueError(f"layer {i}: keys and values of layer {of}, which has none of its own")
            layers.append(LayerSpec(kind, mixer, 0 if mlp is None else int(mlp["ff"]), i))
        streams = int(config["streams"])
        if not 1 <= streams <= MAX_STREAMS:
            raise ValueError(f"{streams} streams: the kernels take up to {MAX_STREAMS}")
        return HybridConfig(width=int(config["width"]), vocab=int(config["vocab"]), layers=layers, eps=float(config["norm"]["eps"]),
                            max_len=max_len, streams=streams, embed_scale=float(config["embedding"]["scale"]), tied_head=False,
                            norm_base=1.0, unit=SWIGLU)

    def slot_bytes(self) -> int:
        """Device bytes one more slot costs: its rows and states in every layer's cache and its rows of a decode step."""
        cache = sum(MIXERS[s.kind].cache_bytes(s.mixer, self.max_len, self.itemsize) for s in self.layers)
        columns = up(self.width, 128)
        rows = (16 + 4 * max(self.streams - 1, 0)) * columns + 8 * up(self.vocab, 64) + 8 * (cache_pages(self.max_len) * 64 + 1)
        return cache + rows


@dataclass
class HyperConnection:
    """How one branch reads and writes the streams, as the arrays a GEMM's epilogue takes: u = sum_s read[s] x_s,
    x_t <- sum_s mix[s, t] x_s + write[t] y."""
    read: ctypes.Array
    write: ctypes.Array
    mix: ctypes.Array
    read_sum: float

    @staticmethod
    def of(read: Tensor, write: Tensor, mix: Tensor) -> "HyperConnection":
        full = torch.zeros((MAX_STREAMS, MAX_STREAMS))
        full[:mix.shape[0], :mix.shape[1]] = mix.float()
        row, square = ctypes.c_float * MAX_STREAMS, ctypes.c_float * (MAX_STREAMS * MAX_STREAMS)
        return HyperConnection(row(*read.float().tolist()), row(*write.float().tolist()), square(*full.flatten().tolist()),
                               float(read.float().sum()))


@dataclass
class LayerWeights:
    gain1: Tensor  # fp32 [C]
    mixer: object
    gain2: "Tensor | None" = None
    w_up: "Tensor | None" = None    # [2 F, C]: gate and up rows alternating
    w_down: "Tensor | None" = None  # [C, F]
    hc1: "HyperConnection | None" = None
    hc2: "HyperConnection | None" = None


@dataclass
class HybridWeights:
    """C = width and every other GEMM size padded with zeros to what the kernels tile."""
    embed: Tensor        # [vocab up to 128, C]
    head: Tensor         # the same shape, maybe the same tensor
    final_gain: Tensor   # fp32 [C]
    layers: list[LayerWeights]
    dtype: torch.dtype

    @staticmethod
    def from_state_dict(state: dict, cfg: HybridConfig, dtype: torch.dtype = torch.bfloat16,
                        device: "torch.device | str" = "cuda") -> "HybridWeights":
        """From a checkpoint's tensors by name: embed, final.norm, and per layer l<i>.norm1 / norm2, l<i>.mix.*, l<i>.mlp.gate
        / up / down; with several streams l<i>.hc1 / hc2.in / out / mix; the head where it is not the embedding. A layer that uses another one's weights has no tensors of its own and shares the prepared ones."""
        C = up(cfg.width, 128)

        def gain(name: str) -> Tensor:
            return pad_to(cfg.norm_base + state[name].to(device).float(), C)

        def connection(name: str) -> "HyperConnection | None":
            if not cfg.streams:
                return None
            read, write, mix = (state[name + part].cpu() for part in (".in", ".out", ".mix"))
            if read.shape != (cfg.streams,) or write.shape != (cfg.streams,) or mix.shape != (cfg.streams, cfg.streams):
                raise ValueError(f"{name}: not of {cfg.streams} streams")
            return HyperConnection.of(read, write, mix)

        layers: list[LayerWeights] = [None] * len(cfg.layers)
        for i, spec in enumerate(cfg.layers):
            if spec.weights_of != i:
                continue
            p = f"l{i}."
            mix = {name[len(p) + 4:]: t for name, t in state.items() if name.startswith(p + "mix.")}
            layer = LayerWeights(gain(p + "norm1"), MIXERS[spec.kind](spec.mixer, mix, cfg.eps, C, dtype, device),
                                 hc1=connection(p + "hc1"))
            if spec.ff:
                F = up(spec.ff, 128)
                w = torch.zeros((F, 2, C), dtype=dtype, device=device)
                for j, name in enumerate(("gate", "up")):
                    w[:spec.ff, j, :cfg.width] = state[p + "mlp." + name].to(device=device, dtype=dtype)
                layer.hc2 = connection(p + "hc2")
                layer.gain2, layer.w_up = gain(p + "norm2"), w.view(2 * F, C)
                layer.w_down = pad_to(state[p + "mlp.down"].to(device=device, dtype=dtype), C, F)
            layers[i] = layer
        for i, spec in enumerate(cfg.layers):
            layers[i] = layers[spec.weights_of]
        embed, head = (pad_to(state[name].to(device=device, dtype=dtype), up(cfg.vocab, 128), C) if name else None
                       for name in ("embed", None if cfg.tied_head else "head"))
        return HybridWeights(embed, embed if head is None else head, gain("final.norm"), layers, dtype)

    @staticmethod
    def random_state(cfg: HybridConfig, seed: int, device: "torch.device | str" = "cpu", std: float = 0.02) -> dict:
        """Random checkpoint tensors of this configuration (bf16): matrices ~ N(0, std), norms multiply by about 1, sinks and
        decay biases ~ N(0, 1), convolutions pass mostly the current token on, streams mix gently. For benchmarks and tests."""
        gen = torch.Generator(device=device).manual_seed(seed)

        def w(*shape, scale=std, base=0.0):
            return (torch.randn(*shape, generator=gen, device=device) * scale + base).bfloat16()

        C = cfg.width
        around = 1.0 - cfg.norm_base
        state = {"embed": w(cfg.vocab, C), "final.norm": w(C, scale=0.1, base=around)}
        if not cfg.tied_head:
            state["head"] = w(cfg.vocab, C)
        for i, spec in enumerate(cfg.layers):
            if spec.weights_of != i:
                continue
            m, p = spec.mixer, f"l{i}."
            H, D, V = m["heads"], m["dim"], m["vdim"]
            state[p + "norm1"] = w(C, scale=0.1, base=around)
            if cfg.streams:
                for q in (1, 2) if spec.ff else (1,):
                    state.update({p + f"hc{q}.in": w(cfg.streams, scale=0.1, base=1.0 / cfg.streams), p + f"hc{q}.out": w(cfg.streams, scale=0.1, base=1.0),
                                  p + f"hc{q}.mix": (w(cfg.streams, cfg.streams, scale=0.05) + torch.eye(cfg.streams, device=device)).bfloat16()})
            if spec.kind == "gla":
                rank = m.get("decay_rank", 16)
                shapes = {"q": (H * D, C), "k": (H * D, C), "v": (H * V, C), "g": (H * V, C), "o": (C, H * V),
                          "a1": (rank, C), "a2": (H * D, rank)}
                state[p + "mix.a2.b"] = w(H * D, scale=1.0, base=2.0)
                state[p + "mix.norm"] = w(V, scale=0.1, base=1.0)
            elif spec.kind in ("attention", "channel_delta"):
                G, delta = m["kv_heads"], spec.kind == "channel_delta"
                rows = {"q": (G if delta else H) * D, "k": G * D, "v": (H if delta else G) * V}
                if m.get("kv_from") is not None:
                    rows = {"q": rows["q"]}
                shapes = {**{n: (count, C) for n, count in rows.items()}, "o": (C, H * V)}
                for n, count in rows.items():
                    taps = w(count, m["conv"], scale=0.2)
                    taps[:, -1] += 1.0
                    state[p + f"mix.{n}.conv"] = taps
                if delta:
                    rank = m.get("low_rank", 128)
                    shapes.update({"b": (H, C), "a1": (rank, C), "a2": (H * D, rank), "g1": (rank, C), "g2": (H * V, rank)})
                    state.update({p + "mix.A_log": w(H, scale=0.5), p + "mix.dt_bias": w(H * D, scale=1.0, base=-4.0),
                                  p + "mix.norm": w(V, scale=0.1, base=1.0)})
                else:
                    shapes["g"] = (H, C)
            else:
                R, rank = m["rot_dim"], m["kv_rank"]
                shapes = {"q": (H * (D + R), C), "dkv": (rank + R, C), "uk": (H * D, rank), "uv": (H * V, rank),
                          "g": (H * V, C), "o": (C, H * V)}
                state[p + "mix.dkv.norm"] = w(rank, scale=0.1, base=1.0)
                state[p + "mix.sink"] = w(H, scale=1.0)
            state.update({p + "mix." + n: w(*s) for n, s in shapes.items()})
            if spec.ff:
                state[p + "norm2"] = w(C, scale=0.1, base=around)
                state.update({p + "mlp.gate": w(spec.ff, C), p + "mlp.up": w(spec.ff, C), p + "mlp.down": w(C, spec.ff)})
        return state


class Stream:
    """The fp32 residual stream of some rows (or several streams) and what the next norm reads: h, x = h * gain (of several: of
    their weighted sum), partial sums of squares."""

    def __init__(self, rows: int, columns: int, dtype: torch.dtype, device, streams: int = 1):
        self.h = torch.empty((rows, streams, columns) if streams > 1 else (rows, columns), dtype=torch.float32, device=device)
        self.x = torch.empty((rows, columns), dtype=dtype, device=device)
        self.ss = torch.empty((rows, columns // 8), dtype=torch.float32, device=device)
        self.parts = 1


class HybridDecoder(StepDecoder):
    """Decoding of up to n_slots sequences of a HybridConfig model."""

    def __init__(self, cfg: HybridConfig, weights: HybridWeights, n_slots: int, device: "torch.device | str" = "cuda",
                 prompt_store: int = 0, softcap: float = 0.0):
        self._start(cfg, weights, n_slots, device, softcap)
        self.dtype, self.f32 = weights.dtype, weights.dtype == torch.float32
        self.caches = []
        for layer in weights.layers:
            of = layer.mixer.kv_from
            self.caches.append(layer.mixer.new_cache(n_slots, cfg.max_len, None if of is None else self.caches[of]))
        self.capacity = cache_pages(cfg.max_len) * 64
        self.sum_of_streams = HyperConnection.of(*(torch.ones(cfg.streams),) * 2, torch.zeros(cfg.streams, cfg.streams))
        self.store = PromptStore([part for cache in self.caches for part in cache.parts], prompt_store) if prompt_store > 0 else None
        self.columns = up(cfg.width, 128)
        self.in_width = max(layer.mixer.in_width for layer in weights.layers)
        self.out_width = max(layer.mixer.out_width for layer in weights.layers)
        self.ff_width = max([l.w_down.shape[1] for l in weights.layers if l.w_down is not None], default=0)
        self._pass: "tuple[int, dict] | None" = None
        self._scratch: dict = {}

    # ---- GEMMs on the stream ------------------------------------------------------------------------------------------

    def gemm_kernel(self, rows: int, N: int, K: int) -> str:
        """As in decoder.py: up to 16 rows skinny_gemm where it is instantiated for the depth, up to 64 stream_gemm, else
        tile_gemm; gemm_f32 for a 32-bit model."""
        if self.f32:
            return "f32"
        if rows <= 16 and cuda_library("decode_step").skinny_gemm_supported(rows, N, K, 0):
            return "skinny"
        return "stream" if rows <= 64 else "tile"

    ENTRY = {"f32": ("gemm_f32", "gemm_f32_rs", 64), "skinny": ("decode_step", "skinny_gemm_rs", 8),
             "stream": ("stream_gemm", "stream_gemm_rs", 128), "tile": ("tile_gemm", "tile_gemm_rs", 32)}

    def gemm(self, rows: int, x: Tensor, w: Tensor, epilogue: int, st: Stream, out: "Tensor | None" = None,
             gain: "Tensor | None" = None, n_store: int = 0, scale: float = 1.0, normed: bool = False,
             then: "Tensor | None" = None, hc: "tuple | None" = None) -> None:
        """epilogue(x . w^T): see ncb_gemm_rs. normed: x is the stream's and its norm is applied; gain: the next norm's
        (epilogues STREAM, STREAMS); then: the weights the next GEMM reads (prefetched into L2 by stream_gemm); hc: this branch's
        and the next one's hyper-connections (STREAMS)."""
        N, K = w.shape
        kind = self.gemm_kernel(rows, N, K)
        lib, entry, part = self.ENTRY[kind]
        a = GemmRs(x=x.data_ptr(), w=w.data_ptr(), rows=rows, N=N, K=K, n_store=n_store or N, epilogue=epilogue, scale=scale,
                   eps=self.cfg.eps, norm_count=self.cfg.width, mult=self.cfg.residual_mult, status=self.status.data_ptr())
        if normed:
            a.ss, a.ss_parts = st.ss.data_ptr(), st.parts
        if epilogue == STREAMS:
            a.streams, a.out, a.mix, a.in_ = self.cfg.streams, hc[0].write, hc[0].mix, hc[1].read
        if epilogue in (STREAM, STREAMS):
            a.h, a.gain, a.x_next, a.ss_next = st.h.data_ptr(), gain.data_ptr(), st.x.data_ptr(), st.ss.data_ptr()
            st.parts = N // part
        else:
            a.y, a.ldy = out.data_ptr(), out.stride(0)
        if kind == "stream" and then is not None:
            a.next_w, a.next_bytes = then.data_ptr(), then.numel() * 2
        check(getattr(cuda_library(lib), entry)(ctypes.byref(a), stream()), entry)

    # ---- one pass over rows -------------------------------------------------------------------------------------------

    def buffers(self, rows: int) -> dict:
        dev, d = self.device, self.dtype
        buf = {"stream": Stream(rows, self.columns, d, dev, max(self.cfg.streams, 1)),
               "proj": torch.empty((rows, self.in_width), dtype=d, device=dev),
               # columns past a mixer's heads are padding that the output projection multiplies by zero weights
               "mixed": torch.zeros((rows, self.out_width), dtype=d, device=dev)}
        if self.ff_width:
            buf["u"] = torch.empty((rows, self.ff_width), dtype=d, device=dev)
        return buf

    def run_layers(self, tokens: Tensor, rows: Rows, buf: dict, fill_only: bool = False) -> Stream:
        """The stream after the last layer, with x = h * final gain; fill_only: stop when the last layer's cache is filled."""
        cfg, w, st, n = self.cfg, self.w, buf["stream"], rows.n
        layers = w.layers
        many = cfg.streams > 0
        write = STREAMS if many else STREAM
        check(cuda_library("decode_step").embed_streams(pointer(w.embed), pointer(tokens), pointer(st.h), pointer(layers[0].gain1),
                                                        pointer(st.x), pointer(st.ss), n, self.columns, cfg.vocab, int(self.f32),
                                                        max(cfg.streams, 1), cfg.embed_scale,
                                                        layers[0].hc1.read_sum if many else 1.0, stream()), "embed_streams")
        st.parts = 1
        for i, layer in enumerate(layers):
            mixer, last = layer.mixer, i + 1 == len(layers)
            after = w.final_gain if last else layers[i + 1].gain1
            proj = buf["proj"].view(-1)[:n * mixer.in_width].view(n, mixer.in_width)
            mixed = buf["mixed"].view(-1)[:n * mixer.out_width].view(n, mixer.out_width)
            self.gemm(n, st.x, mixer.w_in, STORE, st, out=proj, normed=True, then=mixer.w_out)
            if last and fill_only:
                mixer.run(proj, self.caches[i], rows, None)
                return st
            mixer.run(proj, self.caches[i], rows, mixed)
            dense = layer.w_up is not None
            following = layer.w_up if dense else w.head if last else layers[i + 1].mixer.w_in
            read = self.sum_of_streams if last else layers[i + 1].hc1
            self.gemm(n, mixed, mixer.w_out, write, st, gain=layer.gain2 if dense else after, then=following,
                      hc=(layer.hc1, layer.hc2 if dense else read))
            if dense:
                u = buf["u"].view(-1)[:n * layer.w_down.shape[1]].view(n, layer.w_down.shape[1])
                self.gemm(n, st.x, layer.w_up, cfg.unit, st, out=u, normed=True, then=layer.w_down)
                self.gemm(n, u, layer.w_down, write, st, gain=after, then=None if last else layers[i + 1].mixer.w_in,
                          hc=(layer.hc2, read))
        return st

    def head(self, st: Stream, rows: int, out: Tensor) -> None:
        self.gemm(rows, st.x, self.w.head, STORE_F32, st, out=out, n_store=self.cfg.vocab, scale=self.cfg.logit_scale,
                  normed=True)

    # ---- what StepDecoder drives ----------------------------------------------------------------------------------------

    def _pass_rows(self, pos: Tensor, slot_map: Tensor, max_kv_len: int, host_rows: tuple) -> tuple[Rows, dict]:
        n = pos.shape[0]
        if self._pass is None or self._pass[0] < n:
            self._pass = (n, self.buffers(n))
        return Rows(n, pos, slot_map, max_kv_len, self.status, RowPlan(host_rows[0], host_rows[1], self.device),
                    scratch=self._scratch), self._pass[1]

    def fill_rows(self, tokens: Tensor, pos: Tensor, slot_map: Tensor, max_kv_len: int, host_rows: tuple) -> None:
        rows, buf = self._pass_rows(pos, slot_map, max_kv_len, host_rows)
        self.run_layers(tokens, rows, buf, fill_only=True)

    def place_logits(self, tokens: Tensor, pos: Tensor, slot_map: Tensor, max_kv_len: int, host_rows: tuple,
                     places: list[int]) -> Tensor:
        rows, buf = self._pass_rows(pos, slot_map, max_kv_len, host_rows)
        st = self.run_layers(tokens, rows, buf)
        picked = Stream.__new__(Stream)
        at = torch.tensor(places, device=self.device)
        picked.x, picked.parts = st.x[at], st.parts
        picked.ss = st.ss.view(-1)[:rows.n * st.parts].view(rows.n, st.parts)[at]
        out = torch.empty((len(places), self.cfg.vocab), dtype=torch.float32, device=self.device)
        self.head(picked, len(places), out)
        return out

    def step_buffers(self, batch: int) -> dict:
        buf = self.buffers(batch)
        buf["logits"] = torch.empty((batch, self.cfg.vocab), dtype=torch.float32, device=self.device)
        buf["trace"] = torch.zeros((batch, self.capacity + 1), dtype=torch.long, device=self.device)
        buf["scratch"] = {}
        return buf

    def run_step(self, tokens: Tensor, pos: Tensor, slot_map: Tensor, buf: dict) -> None:
        n = tokens.shape[0]
        rows = Rows(n, pos, slot_map, self.capacity, self.status, chunk_tiles=self.chunk_pages, scratch=buf["scratch"])
        self.head(self.run_layers(tokens, rows, buf), n, buf["logits"])

    def planned_chunk(self, positions: list[int], steps: int) -> int:
        """Tiles per chunk of the attention layers' split kernel (the first such layer's choice) for lengths half way through
        the run."""
        attention = next((l.mixer for l in self.w.layers if hasattr(l.mixer, "chunk_for")), None)
        if attention is None:
            return 0
        lens = [min(p + 1 + steps // 2, self.capacity) for p in positions]
        return attention.chunk_for(lens, self.capacity)
