"""Plain, slow restatement of the hybrid designs' mathematics, one function per mechanism, for tests.

Token by token where a mechanism is a recurrence, a full score matrix where it is attention; CPU
tensors in float64 (or the dtype the caller passes). Nothing here is shared with the product path.

Notation: a sequence is a [T, width] tensor; W is [out, in]; a head layout [T, H * D] is read as
[T, H, D]; `first` is the position of the first row given.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor


def rms_norm(x: Tensor, weight: Optional[Tensor], eps: float, weight_offset: float = 0.0) -> Tensor:
    """x / sqrt(mean(x^2) + eps), times (weight_offset + weight) where there is a weight."""
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * (weight_offset + weight)


def silu(x: Tensor) -> Tensor:
    return x / (1.0 + torch.exp(-x))


def sigmoid(x: Tensor) -> Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def softplus(x: Tensor) -> Tensor:
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def rotate_half(x: Tensor, base: float, dims: int, first: int = 0) -> Tensor:
    """x [T, H, D]: pair (i, i + dims / 2) of the first `dims` dimensions turned by
    (first + t) * base^(-2 i / dims); dimensions from `dims` on unchanged."""
    y = x.clone()
    half = dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            angle = (first + t) * base ** (-2.0 * i / dims)
            c, s = math.cos(angle), math.sin(angle)
            u, v = x[t, :, i], x[t, :, i + half]
            y[t, :, i] = u * c - v * s
            y[t, :, i + half] = v * c + u * s
    return y


def causal_conv(x: Tensor, taps: Tensor) -> Tensor:
    """Per-channel filter over time: y[t, c] = sum_j taps[c, j] x[t - (n - 1) + j, c], x = 0 before
    the start."""
    n = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            source = t - (n - 1) + j
            if source >= 0:
                y[t] += taps[:, j] * x[source]
    return y


def unit(x: Tensor, eps: float = 1e-6) -> Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def retention_scan(q: Tensor, k: Tensor, v: Tensor, decay: List[float]) -> Tensor:
    """S' = gamma_h S + k v^T, read-out S'^T q. q, k [T, H, D], v [T, H, V] -> [T, H, V]."""
    tokens, heads, dim = q.shape
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        state = torch.zeros(dim, v.shape[2], dtype=q.dtype)
        for t in range(tokens):
            state = decay[h] * state + torch.outer(k[t, h], v[t, h])
            out[t, h] = state.T @ q[t, h]
    return out


def delta_scan(q: Tensor, k: Tensor, v: Tensor, g: Tensor, beta: Tensor) -> Tensor:
    """P = diag(g) S, S' = P + k (beta (v - P^T k))^T, read-out S'^T q.
    q, k, g [T, H, D], v [T, H, V], beta [T, H] -> [T, H, V]."""
    tokens, heads, dim = q.shape
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        state = torch.zeros(dim, v.shape[2], dtype=q.dtype)
        for t in range(tokens):
            state = g[t, h][:, None] * state
            u = beta[t, h] * (v[t, h] - state.T @ k[t, h])
            state = state + torch.outer(k[t, h], u)
            out[t, h] = state.T @ q[t, h]
    return out


def sink_attention(q: Tensor, k: Tensor, v: Tensor, scale: float, sink: Optional[Tensor]) -> Tensor:
    """Causal softmax attention; the denominator of head h also holds exp(sink[h]).
    q, k [T, H, D], v [T, H, V] -> [T, H, V]."""
    tokens, heads, _ = q.shape
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        scores = (q[:, h] @ k[:, h].T) * scale
        for i in range(tokens):
            row = scores[i, :i + 1]
            top = row.max() if sink is None else torch.maximum(row.max(), sink[h])
            weights = torch.exp(row - top)
            total = weights.sum() + (0.0 if sink is None else torch.exp(sink[h] - top))
            out[i, h] = (weights / total) @ v[:i + 1, h]
    return out


# ------------------------------------------------------------------------------- mixers ----
def retention(w: Dict[str, Tensor], spec: dict, h: Tensor, eps: float) -> Tensor:
    tokens = h.shape[0]
    heads, dim, vdim = spec["heads"], spec["dim"], spec["vdim"]
    q = (h @ w["q"].T).view(tokens, heads, dim)
    k = (h @ w["k"].T).view(tokens, heads, dim)
    v = (h @ w["v"].T).view(tokens, heads, vdim)
    q = rotate_half(q, spec["rot"]["base"], spec["rot"]["dims"])
    k = rotate_half(k, spec["rot"]["base"], spec["rot"]["dims"]) * dim ** -0.5
    o = rms_norm(retention_scan(q, k, v, spec["decay"]), None, eps)
    return (o.reshape(tokens, heads * vdim) * silu(h @ w["g"].T)) @ w["o"].T


def latent_rows(w: Dict[str, Tensor], h: Tensor, eps: float) -> Tensor:
    return rms_norm(h @ w["dkv"].T, w["dkv.norm"], eps)


def latent_attention(w: Dict[str, Tensor], spec: dict, h: Tensor, latent: Tensor, eps: float) -> Tensor:
    tokens = h.shape[0]
    heads, dim, vdim = spec["heads"], spec["dim"], spec["vdim"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(tokens, heads, dim)
    k = (latent @ w["uk"].T).view(tokens, heads, dim)
    v = (latent @ w["uv"].T).view(tokens, heads, vdim)
    o = sink_attention(q, k, v, spec["scale"], w["sink"])
    return o.reshape(tokens, heads * vdim) @ w["o"].T


def channel_delta(w: Dict[str, Tensor], spec: dict, h: Tensor, eps: float) -> Tensor:
    tokens = h.shape[0]
    heads, kv_heads, dim, vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = silu(causal_conv(h @ w["q"].T, w["q.conv"])).view(tokens, kv_heads, dim)
    k = silu(causal_conv(h @ w["k"].T, w["k.conv"])).view(tokens, kv_heads, dim)
    v = silu(causal_conv(h @ w["v"].T, w["v.conv"])).view(tokens, heads, vdim)
    shared = heads // kv_heads
    q = (unit(q) * dim ** -0.5).repeat_interleave(shared, dim=1)
    k = unit(k).repeat_interleave(shared, dim=1)
    beta = sigmoid(h @ w["b"].T)
    step = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).view(tokens, heads, dim)
    g = torch.exp(-torch.exp(w["A_log"])[None, :, None] * step)
    o = rms_norm(delta_scan(q, k, v, g, beta), w["norm"], eps)
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T).view(tokens, heads, vdim)
    return (o * gate).reshape(tokens, heads * vdim) @ w["o"].T


def dense_mlp(w: Dict[str, Tensor], h: Tensor) -> Tensor:
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


# -------------------------------------------------------------------------------- model ----
def _under(weights: Dict[str, Tensor], prefix: str) -> Dict[str, Tensor]:
    return {name[len(prefix):]: value for name, value in weights.items() if name.startswith(prefix)}


def forward(config: dict, weights: Dict[str, Tensor], tokens: List[int], *,
            streams: Optional[list] = None, dtype: torch.dtype = torch.float64) -> Tensor:
    """Logits [T, vocab] of one sequence from the start; `streams` receives the residual stream
    after every layer."""
    w = {name: value.to(dtype) for name, value in weights.items()}
    eps = config["norm"]["eps"]

    def norm(x, name):
        return rms_norm(x, w[name], eps, 1.0)

    x = w["embed"][torch.tensor(tokens, dtype=torch.int64)]
    latents: Dict[int, Tensor] = {}
    for i, layer in enumerate(config["layers"]):
        p, spec = f"l{i}.", layer["mixer"]
        mix = _under(w, p + "mix.")
        h = norm(x, p + "norm1")
        if layer["type"] == "retention":
            y = retention(mix, spec, h, eps)
        elif layer["type"] == "channel_delta":
            y = channel_delta(mix, spec, h, eps)
        elif layer["type"] == "latent_attention":
            source = spec.get("kv_from")
            latents[i] = latent_rows(mix, h, eps) if source is None else latents[source]
            y = latent_attention(mix, spec, h, latents[i], eps)
        else:
            raise ValueError(f"unknown mixer {layer['type']!r}")
        x = x + norm(y, p + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(dense_mlp(_under(w, p + "mlp."), norm(x, p + "norm2")), p + "norm2b")
        if streams is not None:
            streams.append(x)
    return norm(x, "final.norm") @ w["head"].T


def greedy(config: dict, weights: Dict[str, Tensor], prompt: List[int], steps: int) -> List[int]:
    """Greedy continuation, the whole sequence recomputed at every step."""
    tokens = list(prompt)
    for _ in range(steps):
        tokens.append(int(forward(config, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


# ------------------------------------------------------------- mechanisms of Lozanex ----
def chunk_attention(q: Tensor, k: Tensor, v: Tensor, scale: float, chunk: Optional[int]) -> Tensor:
    """Causal softmax attention with grouped heads (H query heads on G key heads); with `chunk` a row sees
    only the keys of its own chunk of `chunk` positions. q [T, H, D], k [T, G, D], v [T, G, V]."""
    tokens, heads, _ = q.shape
    group = heads // k.shape[1]
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        keys, values = k[:, h // group], v[:, h // group]
        for i in range(tokens):
            first = 0 if chunk is None else i // chunk * chunk
            scores = (keys[first:i + 1] @ q[i, h]) * scale
            weights = torch.exp(scores - scores.max())
            out[i, h] = (weights / weights.sum()) @ values[first:i + 1]
    return out


def attention_keys(w: Dict[str, Tensor], spec: dict, h: Tensor, eps: float):
    """Keys (normed over the whole projection, then rotated) and values of every token."""
    tokens, groups = h.shape[0], spec["kv_heads"]
    k = rms_norm(h @ w["k"].T + w["k.b"], w["k.norm"], eps).view(tokens, groups, spec["dim"])
    rot = spec.get("rot")
    if rot is not None:
        k = rotate_half(k, rot["base"], rot["dims"])
    return k, (h @ w["v"].T + w["v.b"]).view(tokens, groups, spec["vdim"])


def attention(w: Dict[str, Tensor], spec: dict, h: Tensor, keys: Tensor, values: Tensor, eps: float) -> Tensor:
    tokens, heads = h.shape[0], spec["heads"]
    q = rms_norm(h @ w["q"].T + w["q.b"], w["q.norm"], eps).view(tokens, heads, spec["dim"])
    rot, mask = spec.get("rot"), spec.get("mask")
    if rot is not None:
        q = rotate_half(q, rot["base"], rot["dims"])
    o = chunk_attention(q, keys, values, spec["scale"], None if mask is None else mask["size"])
    return o.reshape(tokens, heads * spec["vdim"]) @ w["o"].T + w["o.b"]


def head_delta(w: Dict[str, Tensor], spec: dict, h: Tensor, eps: float) -> Tensor:
    """The gated delta rule with one decay per head and a silu gate on the normed read-out."""
    tokens = h.shape[0]
    heads, kv_heads, dim, vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = silu(causal_conv(h @ w["q"].T, w["q.conv"])).view(tokens, kv_heads, dim)
    k = silu(causal_conv(h @ w["k"].T, w["k.conv"])).view(tokens, kv_heads, dim)
    v = silu(causal_conv(h @ w["v"].T, w["v.conv"])).view(tokens, heads, vdim)
    shared = heads // kv_heads
    q = (unit(q) * dim ** -0.5).repeat_interleave(shared, dim=1)
    k = unit(k).repeat_interleave(shared, dim=1)
    beta = sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = rms_norm(delta_scan(q, k, v, g[:, :, None].expand(tokens, heads, dim), beta), w["norm"], eps)
    gate = silu(h @ w["g"].T).view(tokens, heads, vdim)
    return (o * gate).reshape(tokens, heads * vdim) @ w["o"].T


def route(router: Tensor, h: Tensor, top: int):
    """The `top` experts of every token with the largest sigmoid scores, and the scores themselves."""
    scores = sigmoid(h @ router.T)
    return torch.topk(scores, top, dim=-1)


def expert_mlp(w: Dict[str, Tensor], spec: dict, h: Tensor) -> Tensor:
    """Every token's chosen experts run on the token scaled by the expert's score; their results are added
    to the shared expert's."""
    scores, chosen = route(w["router"], h, spec["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for score, expert in zip(scores[t], chosen[t].tolist()):
            out[t] += dense_mlp(_under(w, f"e{expert}."), (score * h[t])[None])[0]
    return out if spec.get("shared") is None else out + dense_mlp(_under(w, "shared."), h)


def lozanex_forward(config: dict, weights: Dict[str, Tensor], tokens: List[int], *,
                    streams: Optional[list] = None, dtype: torch.dtype = torch.float64) -> Tensor:
    """Logits [T, vocab] of one sequence from the start; `streams` receives the residual stream
    after every layer."""
    w = {name: value.to(dtype) for name, value in weights.items()}
    eps = config["norm"]["eps"]
    x = rms_norm(w["embed"][torch.tensor(tokens, dtype=torch.int64)], w["embed.norm"], eps)
    cached: Dict[int, tuple] = {}
    for i, layer in enumerate(config["layers"]):
        p, spec = f"l{i}.", layer["mixer"]
        mix = _under(w, p + "mix.")
        if layer["type"] == "delta":
            y = head_delta(mix, spec, x, eps)
        elif layer["type"] == "attention":
            source = spec.get("kv_from")
            cached[i] = attention_keys(mix, spec, x, eps) if source is None else cached[source]
            y = attention(mix, spec, x, *cached[i], eps)
        else:
            raise ValueError(f"unknown mixer {layer['type']!r}")
        x = x + rms_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(expert_mlp(_under(w, p + "mlp."), layer["mlp"], x), w[p + "norm2"], eps)
        if streams is not None:
            streams.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
