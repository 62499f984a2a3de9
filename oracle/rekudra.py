"""TEST INFRASTRUCTURE: a plain, slow restatement of the Rekudra model on the CPU, one function per mechanism.

Everything runs in float64 on weights as they are stored, one whole sequence at a time, with no cache: token t's row is
computed from rows 0 .. t of the same call. Weights are a dict of tensors under their checkpoint names; cfg is the
parsed config.json. Nothing here is imported by the package, and nothing of the package is imported here."""

import math

import torch

F64 = torch.float64


def root_mean_square(x: torch.Tensor, eps: float) -> torch.Tensor:
    return torch.sqrt((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps)


def zero_centred_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return x / root_mean_square(x, eps) * (1.0 + weight)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 0, z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def short_convolution(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [n, channels], w [channels, taps]: y_t = sum over j of w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    n, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(n):
        for j in range(taps):
            at = t - taps + 1 + j
            if at >= 0:
                y[t] += w[:, j] * u[at]
    return y


def banded_frequencies(rot: dict) -> torch.Tensor:
    """The angle per position of every pair: short wavelengths keep theirs, long ones turn `factor` times slower, and between
    the two the two frequencies are mixed by how often the wavelength fits into the original context."""
    out = []
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            fits = s["original"] * f / (2.0 * math.pi)  # original / wavelength
            if fits < s["low"]:
                f = f / s["factor"]
            elif fits <= s["high"]:
                share = (fits - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - share) * f / s["factor"] + share * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [n, heads, dim]: row t is at position t; dimension i < dims / 2 turns with i + dims / 2, the rest pass."""
    f, half, out = banded_frequencies(rot), rot["dims"] // 2, x.clone()
    for t in range(x.shape[0]):
        c, s = torch.cos(t * f), torch.sin(t * f)
        u, v = x[t, :, :half], x[t, :, half:2 * half]
        out[t, :, :half] = u * c - v * s
        out[t, :, half:2 * half] = v * c + u * s
    return out


def keys_and_values(h: torch.Tensor, w: dict, m: dict, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """([n, kv_heads, dim] as a cache holds them, [n, kv_heads, vdim])."""
    n, G = h.shape[0], m["kv_heads"]
    k = rotate(short_convolution(h @ w["k"].T, w["k.conv"]).view(n, G, m["dim"]), m["rot"])
    v = short_convolution(h @ w["v"].T, w["v.conv"]).view(n, G, m["vdim"])
    return k / root_mean_square(k, eps), v


def attention(h: torch.Tensor, w: dict, m: dict, eps: float, kv: tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
    """h [n, width] -> [n, width], over keys and values of the same positions (this layer's or another's)."""
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    keys, values = kv
    q = rotate(short_convolution(h @ w["q"].T, w["q.conv"]).view(n, H, m["dim"]), m["rot"])
    q = q / root_mean_square(q, eps)
    gate = sigmoid(h @ w["g"].T)
    out = torch.zeros(n, H, m["vdim"], dtype=F64)
    for a in range(H):
        score = q[:, a] @ keys[:, a // (H // G)].T * m["scale"]
        score = score.masked_fill(torch.ones(n, n, dtype=torch.bool).triu(1), -math.inf)
        e = torch.exp(score - score.max(-1, keepdim=True).values)
        out[:, a] = e / e.sum(-1, keepdim=True) @ values[:, a // (H // G)] * gate[:, a:a + 1]
    return out.reshape(n, -1) @ w["o"].T


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """One head: q, k, g [n, dim], v [n, vdim], beta [n] -> what each token reads [n, vdim]."""
    state = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros_like(v)
    for t in range(len(q)):
        state = g[t][:, None] * state
        state = state + torch.outer(k[t], beta[t] * (v[t] - state.T @ k[t]))
        out[t] = state.T @ q[t]
    return out


def channel_decay(h: torch.Tensor, w: dict, heads: int) -> torch.Tensor:
    """[n, heads, dim], each in (0, 1)."""
    z = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).view(h.shape[0], heads, -1)
    return torch.exp(-torch.exp(w["A_log"])[:, None] * z)


def channel_delta(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ w[x].T, w[x + ".conv"])).view(n, -1, d) for x, d in (("q", D), ("k", D), ("v", V)))
    q, k = unit(q) * D ** -0.5, unit(k)
    g, beta = channel_decay(h, w, H), sigmoid(h @ w["b"].T)
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T).view(n, H, V)
    out = torch.zeros(n, H, V, dtype=F64)
    for a in range(H):
        j = a // (H // G)
        o = delta_rule(q[:, j], k[:, j], v[:, a], g[:, a], beta[:, a])
        out[:, a] = o / root_mean_square(o, eps) * w["norm"] * gate[:, a]
    return out.reshape(n, -1) @ w["o"].T


def dense_feed_forward(h: torch.Tensor, w: dict) -> torch.Tensor:
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def read_streams(x: torch.Tensor, w: dict) -> torch.Tensor:
    """x [streams, n, width] -> what a sublayer reads."""
    return sum(w["in"][s] * x[s] for s in range(len(x)))


def write_streams(x: torch.Tensor, y: torch.Tensor, w: dict) -> torch.Tensor:
    """Every stream from all the old ones and the sublayer's result; w["mix"] is [from, to]."""
    return torch.stack([sum(w["mix"][s, t] * x[s] for s in range(len(x))) + w["out"][t] * y for t in range(len(x))])


def part(weights: dict, prefix: str) -> dict:
    return {name[len(prefix):]: t.to(F64) for name, t in weights.items() if name.startswith(prefix)}


def layer(x: torch.Tensor, i: int, cfg: dict, weights: dict, kv: dict) -> torch.Tensor:
    """kv: layer -> its keys and values, filled by the layers that have their own."""
    entry, eps, w = cfg["layers"][i], cfg["norm"]["eps"], part(weights, f"l{i}.")
    m, mix = entry["mixer"], part(w, "mix.")
    h = zero_centred_norm(read_streams(x, part(w, "hc1.")), w["norm1"], eps)
    if entry["type"] == "attention":
        if "kv_from" not in m:
            kv[i] = keys_and_values(h, mix, m, eps)
        y = attention(h, mix, m, eps, kv[m.get("kv_from", i)])
    else:
        y = channel_delta(h, mix, m, eps)
    x = write_streams(x, y, part(w, "hc1."))
    if entry.get("mlp") is not None:
        h = zero_centred_norm(read_streams(x, part(w, "hc2.")), w["norm2"], eps)
        x = write_streams(x, dense_feed_forward(h, part(w, "mlp.")), part(w, "hc2."))
    return x


def forward(tokens: list[int], cfg: dict, weights: dict, streams: list | None = None) -> torch.Tensor:
    """Logits [n, vocab] in float64; `streams` collects the sum of the streams after every layer."""
    x = weights["embed"].to(F64)[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    x = torch.stack([x] * cfg["streams"])
    kv: dict = {}
    for i in range(len(cfg["layers"])):
        x = layer(x, i, cfg, weights, kv)
        if streams is not None:
            streams.append(x.sum(0))
    return zero_centred_norm(x.sum(0), weights["final.norm"].to(F64), cfg["norm"]["eps"]) @ weights["head"].to(F64).T
