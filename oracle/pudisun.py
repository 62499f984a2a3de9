"""TEST INFRASTRUCTURE: a plain, slow restatement of the Pudisun model on the CPU, one function per mechanism.

Everything runs in float64 on weights as they are stored, one whole sequence at a time, with no cache: token t's row is
computed from rows 0 .. t of the same call. Weights are a dict of tensors under their checkpoint names; cfg is the
parsed config.json. Nothing here is imported by the package, and nothing of the package is imported here."""

import math

import torch

F64 = torch.float64


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def rotary_frequencies(rot: dict) -> tuple[torch.Tensor, float]:
    """(frequency of each pair, factor of both cos and sin), with the optional YaRN interpolation of rot["scaling"]."""
    dims, base = rot["dims"], float(rot["base"])
    freqs, mscale = [], 1.0
    for i in range(dims // 2):
        freqs.append(base ** (-2.0 * i / dims))
    s = rot.get("scaling")
    if s:
        def dim_of(turns: float) -> float:
            return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        lo = max(math.floor(dim_of(s["fast"])), 0)
        hi = min(math.ceil(dim_of(s["slow"])), dims - 1)
        for i in range(dims // 2):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            freqs[i] = freqs[i] / s["factor"] * ramp + freqs[i] * (1.0 - ramp)
        mscale = 0.1 * math.log(s["factor"]) + 1.0
    return torch.tensor(freqs, dtype=F64), mscale


def rotate(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [n, ..., dims at least rot dims]: element i of the first half turns with element i of the second half."""
    freqs, mscale = rotary_frequencies(rot)
    half = rot["dims"] // 2
    out = x.clone()
    for t in range(x.shape[0]):
        angle = float(positions[t]) * freqs
        c, s = torch.cos(angle) * mscale, torch.sin(angle) * mscale
        u, v = x[t, ..., :half], x[t, ..., half:2 * half]
        out[t, ..., :half] = u * c - v * s
        out[t, ..., half:2 * half] = v * c + u * s
    return out


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor | float) -> torch.Tensor:
    """Softmax weights over the last axis with exp(sink) added to the denominator."""
    m = torch.clamp(scores.max(), min=float(sink))
    e = torch.exp(scores - m)
    return e / (e.sum() + math.exp(float(sink) - float(m)))


def latent_attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """h [n, width] -> [n, width]; w: the mixer's tensors without their prefix."""
    n, H, D, R, Vd, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(n)
    q = (h @ w["q"].T).view(n, H, D + R)
    q_plain, q_rot = q[..., :D], rotate(q[..., D:], pos, m["rot"])
    kv = h @ w["dkv"].T
    c = rms_norm(kv[:, :rank], w["dkv.norm"], eps)
    k_rot = rotate(kv[:, rank:], pos, m["rot"])
    k = (c @ w["uk"].T).view(n, H, D)
    v = (c @ w["uv"].T).view(n, H, Vd)
    out = torch.zeros(n, H, Vd, dtype=F64)
    for t in range(n):
        for a in range(H):
            s = (k[:t + 1, a] @ q_plain[t, a] + k_rot[:t + 1] @ q_rot[t, a]) * m["scale"]
            out[t, a] = sink_softmax(s, w["sink"][a]) @ v[:t + 1, a]
    gate = 1.0 / (1.0 + torch.exp(-(h @ w["g"].T)))
    return (out.reshape(n, H * Vd) * gate) @ w["o"].T


def gated_linear_attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    n, H, D, Vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(n, H, D) * D ** -0.5
    k = (h @ w["k"].T).view(n, H, D)
    v = (h @ w["v"].T).view(n, H, Vd)
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    alpha = ((1.0 / (1.0 + torch.exp(-z))) ** (1.0 / m["tau"])).view(n, H, D)
    state = torch.zeros(H, D, Vd, dtype=F64)
    out = torch.zeros(n, H, Vd, dtype=F64)
    for t in range(n):
        for a in range(H):
            state[a] = alpha[t, a][:, None] * state[a] + torch.outer(k[t, a], v[t, a])
            out[t, a] = state[a].T @ q[t, a]
    out = rms_norm(out, w["norm"], eps).reshape(n, H * Vd)
    return (out * silu(h @ w["g"].T)) @ w["o"].T


def dense_feed_forward(h: torch.Tensor, w: dict) -> torch.Tensor:
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"latent_attention": latent_attention, "gla": gated_linear_attention}


def part(weights: dict, prefix: str) -> dict:
    return {name[len(prefix):]: t.to(F64) for name, t in weights.items() if name.startswith(prefix)}


def layer(x: torch.Tensor, i: int, cfg: dict, weights: dict) -> torch.Tensor:
    entry, eps, m = cfg["layers"][i], cfg["norm"]["eps"], cfg["residual_mult"]
    w = part(weights, f"l{entry.get('weights_of', i)}.")
    h = rms_norm(x, w["norm1"], eps)
    x = x + m * MIXERS[entry["type"]](h, part(w, "mix."), entry["mixer"], eps)
    if entry.get("mlp") is not None:
        x = x + m * dense_feed_forward(rms_norm(x, w["norm2"], eps), part(w, "mlp."))
    return x


def forward(tokens: list[int], cfg: dict, weights: dict, streams: list | None = None) -> torch.Tensor:
    """Logits [n, vocab] in float64; `streams` collects the residual stream after every layer."""
    embed = weights["embed"].to(F64)
    x = embed[torch.tensor(tokens)]
    for i in range(len(cfg["layers"])):
        x = layer(x, i, cfg, weights)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, weights["final.norm"].to(F64), cfg["norm"]["eps"]) @ embed.T * cfg["logit_scale"]
