"""Plain, slow implementation of the Bosenex decoder: one function per mechanism, whole sequences only.

Written from the design's equations with dense tensors on the CPU: no cache, no pages, no portions, no batch.
Nothing here is imported by the product package and nothing of the product is imported here.  Notation: ``h``
[L, width] is a sublayer's input for the L tokens of one sequence, positions are 0 .. L-1, weights are stored
[out, in] and applied as ``h @ W.T``.

A layer is  x = x + mixer(N1(x));  x = x + ff(N2(x))  with N an RMS norm; the mixer is a matrix memory with
exponential gates ("mlstm") or window attention and a state-space mixer side by side ("parallel").
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


def rms_norm(x: torch.Tensor, weight: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def sub(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


# ---------------------------------------------------------------------------------------------- matrix memory
def log_gates(h: torch.Tensor, w: Dict[str, torch.Tensor], cap: float):
    """(log input gate, log forget gate), each [L, heads]: both pre-activations pass cap * tanh(. / cap)."""
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap))
    return i, f


def matrix_memory(q, k, v, i, f, cancellations: Optional[list] = None):
    """q, k [L, H, D], v [L, H, V], log gates [L, H] -> [L, H, V], token by token, with the running maximum m (zero at the
    start) that keeps the exponentials small.  ``cancellations`` receives, per token, how much is left of S^T q after
    cancellation (the least over the heads of rms(S^T q) / rms(|S|^T |q|))."""
    L, H, D = q.shape
    V = v.shape[2]
    S, n, m = q.new_zeros(H, D, V), q.new_zeros(H, D), q.new_zeros(H)
    out, left = q.new_zeros(L, H, V), q.new_zeros(L)
    for t in range(L):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        m = m_new
        read, size = torch.einsum("hdv,hd->hv", S, q[t]), torch.einsum("hd,hd->h", n, q[t]).abs()
        out[t] = read / (torch.maximum(size, torch.exp(-m)) + 1e-6)[:, None]
        spread = torch.einsum("hdv,hd->hv", S.abs(), q[t].abs())
        left[t] = ((read ** 2).mean(-1).sqrt() / (spread ** 2).mean(-1).sqrt().clamp_min(1e-30)).min()
    if cancellations is not None:
        cancellations.append(left)
    return out


def mlstm(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, cancellations: Optional[list] = None) -> torch.Tensor:
    L = h.shape[0]
    H, D, V = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (h @ w["q"].T).view(L, H, D) * D ** -0.5, (h @ w["k"].T).view(L, H, D), (h @ w["v"].T).view(L, H, V)
    i, f = log_gates(h, w, float(m["gate_cap"]))
    heads = rms_norm(matrix_memory(q, k, v, i, f, cancellations), None, eps).reshape(L, H * V)
    return (heads * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ---------------------------------------------------------------------------------------------- window attention
def rotate_halves(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [L, heads, D]: element i pairs with element i + dims/2; elements from ``dims`` on pass unchanged."""
    n = dims // 2
    freqs = torch.tensor([base ** (-2.0 * i / dims) for i in range(n)], dtype=x.dtype)
    angle = (positions.to(x.dtype)[:, None] * freqs[None, :])[:, None, :]
    u, v = x[..., :n], x[..., n:dims]
    out = x.clone()
    out[..., :n] = u * torch.cos(angle) - v * torch.sin(angle)
    out[..., n:dims] = v * torch.cos(angle) + u * torch.sin(angle)
    return out


def softmax_with_sink(scores: torch.Tensor, visible: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """scores [H, L, L], sink [H]: the denominator holds one more term per head, exp(sink[h]), without a value."""
    H, L, _ = scores.shape
    scores = scores.masked_fill(~visible, float("-inf"))
    col = sink.to(scores.dtype).view(H, 1, 1).expand(H, L, 1)
    return torch.softmax(torch.cat([scores, col], dim=-1), dim=-1)[..., :-1]


def window_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict) -> torch.Tensor:
    """Grouped heads, partly rotated queries and keys, capped scores, a window, a sink and a gate per head."""
    L = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(L)
    q, k, v = (h @ w["q"].T).view(L, H, D), (h @ w["k"].T).view(L, G, D), (h @ w["v"].T).view(L, G, V)
    if m.get("rot") is not None:
        base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
        q, k = rotate_halves(q, pos, base, dims), rotate_halves(k, pos, base, dims)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    if m.get("softcap") is not None:
        scores = float(m["softcap"]) * torch.tanh(scores / float(m["softcap"]))
    i, j = torch.arange(L)[:, None], torch.arange(L)[None, :]
    visible = j <= i
    if m.get("mask") is not None:
        visible = visible & (i - j < int(m["mask"]["size"]))
    p = softmax_with_sink(scores, visible[None], w["sink"])
    heads = torch.einsum("hij,jhv->ihv", p, v) * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return heads.reshape(L, H * V) @ w["o"].T


# ---------------------------------------------------------------------------------------------- state space
def causal_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [L, C], taps [C, T]: per channel, zeros before the start, the last tap weighs the current token."""
    L, T = x.shape[0], taps.shape[1]
    padded = torch.cat([x.new_zeros(T - 1, x.shape[1]), x])
    return sum(padded[t:t + L] * taps[:, t] for t in range(T)) + bias


def scalar_decay_scan(x, B, C, dt, rate, skip):
    """x [L, H, V], B and C [L, H, N], dt [L, H], rate and skip [H] -> (y [L, H, V], spread [L, H, V]), token by token: a head's
    state decays by exp(-rate * dt) as a whole.  ``spread`` is y with the magnitude of every term in its place."""
    L, H, V = x.shape
    S = x.new_zeros(H, B.shape[2], V)
    out, spread = x.new_zeros(L, H, V), x.new_zeros(L, H, V)
    for t in range(L):
        S = torch.exp(-rate * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out[t] = torch.einsum("hnv,hn->hv", S, C[t]) + skip[:, None] * x[t]
        spread[t] = torch.einsum("hnv,hn->hv", S.abs(), C[t].abs()) + (skip[:, None] * x[t]).abs()
    return out, spread


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """The gate first, then a norm over each of ``parts`` equal parts of the row."""
    y = y * z * torch.sigmoid(z)
    return rms_norm(y.view(y.shape[0], parts, -1), None, eps).reshape(y.shape) * weight


def mamba2(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, cancellations: Optional[list] = None) -> torch.Tensor:
    """``cancellations`` receives, per token, how much is left of a normed part after cancellation (the least over the parts)."""
    L = h.shape[0]
    H, V, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * V
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    xbc = causal_conv(xbc, w["conv"], w["conv.b"])
    xbc = xbc * torch.sigmoid(xbc)
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    B, C = (t.view(L, G, N).repeat_interleave(H // G, dim=1) for t in (B, C))
    dt = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=1e9)
    y, spread = (t.reshape(L, inner) for t in scalar_decay_scan(x.view(L, H, V), B, C, dt, torch.exp(w["A_log"]), w["D"]))
    parts = int(m["norm_groups"])
    if cancellations is not None:
        size = lambda t: ((t * z * torch.sigmoid(z)).view(L, parts, -1) ** 2).mean(-1).sqrt()
        cancellations.append((size(y) / size(spread).clamp_min(1e-30)).min(dim=-1).values)
    return gated_group_norm(y, z, w["norm"], parts, eps) @ w["o"].T


def side_by_side(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, cancellations: Optional[list] = None) -> torch.Tensor:
    """Half the sum of the two outputs, each normed over the width with a weight of its own."""
    left = rms_norm(window_attention(h, sub(w, "left."), m["left"]), w["left.out"], eps)
    right = rms_norm(mamba2(h, sub(w, "right."), m["right"], eps, cancellations), w["right.out"], eps)
    return 0.5 * (left + right)


# ---------------------------------------------------------------------------------------------- feed-forward
def relu_gated(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return (torch.relu(h @ gate.T) * (h @ up.T)) @ down.T


def clamped_expert(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def routed(h: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, top: int):
    """(chosen experts [L, top], weights [L, top]): the ``top`` largest logits, softmax over those alone."""
    val, idx = torch.topk(h @ router.T + bias, top, dim=-1)
    return idx, torch.softmax(val, dim=-1)


def route_margins(h: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, top: int) -> torch.Tensor:
    """[L]: distance between the last chosen and the first rejected logit, relative to the largest magnitude."""
    z = h @ router.T + bias
    if top >= z.shape[1]:
        return torch.full((h.shape[0],), float("inf"), dtype=h.dtype)
    ordered = torch.sort(z, dim=-1, descending=True).values
    return (ordered[:, top - 1] - ordered[:, top]) / z.abs().max(dim=-1).values.clamp_min(1e-30)


def moe_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], mlp: dict, margins: Optional[list] = None) -> torch.Tensor:
    top, limit = int(mlp["router"]["top"]), float(mlp["expert"]["limit"])
    idx, weight = routed(h, w["router"], w["router.b"], top)
    if margins is not None:
        margins.append(route_margins(h, w["router"], w["router.b"], top))
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=h.dtype)
    for t in range(h.shape[0]):
        for c in range(top):
            x = int(idx[t, c])
            out[t] += weight[t, c] * clamped_expert(h[t:t + 1], w[f"e{x}.gate"], w[f"e{x}.up"], w[f"e{x}.down"], limit)[0]
    if mlp.get("shared") is not None:
        out = out + clamped_expert(h, w["shared.gate"], w["shared.up"], w["shared.down"], float(mlp["shared"]["limit"]))
    return out


# ---------------------------------------------------------------------------------------------- the model
def layer(x: torch.Tensor, w: Dict[str, torch.Tensor], spec: dict, eps: float, margins: Optional[list] = None,
          cancellations: Optional[list] = None) -> torch.Tensor:
    h = rms_norm(x, w["norm1"], eps)
    if spec["type"] == "parallel":
        x = x + side_by_side(h, sub(w, "mix."), spec["mixer"], eps, cancellations)
    else:
        x = x + mlstm(h, sub(w, "mix."), spec["mixer"], eps, cancellations)
    mlp = spec.get("mlp")
    if mlp is not None:
        h, wf = rms_norm(x, w["norm2"], eps), sub(w, "mlp.")
        x = x + (relu_gated(h, wf["gate"], wf["up"], wf["down"]) if mlp["kind"] == "dense" else moe_ff(h, wf, mlp, margins))
    return x


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            streams: Optional[list] = None, margins: Optional[list] = None, cancellations: Optional[list] = None) -> torch.Tensor:
    """Logits [L, vocab] of one whole sequence.  ``streams`` receives the stream after every layer; ``margins`` receives
    per-token margins of every routed layer (``route_margins``: a small one marks a token at which rounding to 16 bits may choose
    other experts), ``cancellations`` what cancellation leaves of every recurrence's output before it is normed (``matrix_memory``,
    ``mamba2``: a small one marks a token at which rounding is magnified)."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(list(tokens))] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, sub(w, f"l{i}."), spec, eps, margins, cancellations)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T * float(cfg.get("logit_scale", 1.0))
