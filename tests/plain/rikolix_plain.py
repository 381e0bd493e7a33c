"""Plain, slow implementation of the Rikolix decoder: one function per mechanism, whole sequences only.

Written from the design's equations with dense tensors on the CPU: no cache, no pages, no portions, no batch.
Nothing here is imported by the product package and nothing of the product is imported here.  Notation: ``h``
[L, width] is a sublayer's input for the L tokens of one sequence, positions are 0 .. L-1, weights are stored
[out, in] and applied as ``h @ W.T``.

A layer is  x = x + N1b(mixer(N1(x)));  x = x + N2b(ff(N2(x)))  with N an RMS norm whose weight is stored as its
distance from one.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch


# ---------------------------------------------------------------------------------------------- norms, rotation
def rms_norm(x: torch.Tensor, weight: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def rms_norm_about_one(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_norm(x, None, eps) * (1.0 + weight)


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int, sign: float = 1.0) -> torch.Tensor:
    """x [L, heads, D]: the pair (2i, 2i + 1) turns by sign * position * base^(-2i/dims); elements from ``dims`` on pass."""
    out = x.clone()
    for i in range(dims // 2):
        angle = sign * positions.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def causal(L: int) -> torch.Tensor:
    return torch.arange(L)[None, :] <= torch.arange(L)[:, None]


# ---------------------------------------------------------------------------------------------- mixers
def latent_rows(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """(latent c [L, rank], rotated key part [L, rot_dim]): what a token leaves for its own layer and for borrowers."""
    C = int(m["kv_rank"])
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :C], w["dkv.norm"], eps)
    k_rot = rotate_neighbours(down[:, None, C:], torch.arange(h.shape[0]), float(m["rot"]["base"]), int(m["rot_dim"]))[:, 0]
    return c, k_rot


def latent_queries(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """(plain part [L, H, dim], rotated part [L, H, rot_dim]) from the queries' own normed latent."""
    H, D, R = int(m["heads"]), int(m["dim"]), int(m["rot_dim"])
    c_q = rms_norm(h @ w["dq"].T, w["dq.norm"], eps)
    q = (c_q @ w["uq"].T).view(-1, H, D + R)
    return q[..., :D], rotate_neighbours(q[..., D:], torch.arange(h.shape[0]), float(m["rot"]["base"]), R)


def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, rows) -> torch.Tensor:
    """``rows``: (c, k_rot) of this layer or of the layer it borrows from; expansions and queries are its own."""
    L, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    c, k_rot = rows
    q_plain, q_rot = latent_queries(h, w, m, eps)
    k_plain = (c @ w["uk"].T).view(L, H, D)
    value = (c @ w["uv"].T).view(L, H, V)
    scores = torch.einsum("ihd,jhd->hij", q_plain, k_plain) + torch.einsum("ihr,jr->hij", q_rot, k_rot)
    scores = (scores * float(m["scale"])).masked_fill(~causal(L)[None], float("-inf"))
    heads = torch.einsum("hij,jhv->ihv", torch.softmax(scores, dim=-1), value)
    return heads.reshape(L, H * V) @ w["o"].T


def sigmoid_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    """Grouped heads; q and k normed over the whole projection; weights sigmoid(score + bias[head]), not normalised; values
    turned by their position over all their dimensions, outputs turned back by the query's."""
    L, H, G, D, V = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(L)
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).view(L, H, D)
    k = rms_norm(h @ w["k"].T, w["k.norm"], eps).view(L, G, D)
    v = (h @ w["v"].T).view(L, G, V)
    q, k = rotate_neighbours(q, pos, base, dims), rotate_neighbours(k, pos, base, dims)
    v = rotate_neighbours(v, pos, base, V)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"]) + w["pb"][:, None, None]
    weights = torch.sigmoid(scores) * causal(L)[None]
    heads = rotate_neighbours(torch.einsum("hij,jhv->ihv", weights, v), pos, base, V, sign=-1.0)
    return heads.reshape(L, H * V) @ w["o"].T


# ---------------------------------------------------------------------------------------------- feed-forwards
def squared_relu(x: torch.Tensor) -> torch.Tensor:
    return torch.relu(x) ** 2


def dense(h: torch.Tensor, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    return squared_relu(h @ w["up"].T) @ w["down"].T


def choose(scores: torch.Tensor, correction: torch.Tensor, top: int, groups: Optional[dict]) -> List[List[int]]:
    """Per token the ``top`` outputs with the largest score + correction, from the ``groups.keep`` groups of neighbours with
    the largest best member (ties: the lower index)."""
    choice = (scores + correction).tolist()
    out = []
    for row in choice:
        E = len(row)
        allowed = list(range(E))
        if groups is not None:
            size = E // int(groups["count"])
            best = [max(row[g * size:(g + 1) * size]) for g in range(int(groups["count"]))]
            kept = sorted(range(len(best)), key=lambda g: (-best[g], g))[:int(groups["keep"])]
            allowed = [e for e in allowed if e // size in kept]
        out.append(sorted(allowed, key=lambda e: (-row[e], e))[:top])
    return out


def choice_margin(row: List[float], chosen: List[int], groups: Optional[dict]) -> float:
    """How far the choice score of the last output chosen lies above the best one passed over, and that of the worst group
    kept above the best group left out (the smaller of the two): what a rounding of the scores must stay below."""
    E = len(row)
    allowed, margin = list(range(E)), float("inf")
    if groups is not None:
        size = E // int(groups["count"])
        best = sorted((max(row[g * size:(g + 1) * size]), g) for g in range(int(groups["count"])))[::-1]
        keep = int(groups["keep"])
        if keep < len(best):
            margin = best[keep - 1][0] - best[keep][0]
        kept = [g for _, g in best[:keep]]
        allowed = [e for e in allowed if e // size in kept]
    rest = [row[e] for e in allowed if e not in chosen]
    return min(margin, min(row[e] for e in chosen) - max(rest)) if rest else margin


def mixture(h: torch.Tensor, w: Dict[str, torch.Tensor], mlp: dict, log: Optional[list] = None) -> torch.Tensor:
    """Weighted sum of the chosen experts; outputs of the router behind the experts stand for the input itself."""
    router = mlp["router"]
    E = int(router["experts"])
    scores = torch.softmax(h @ w["router"].T, dim=-1)
    ids = choose(scores, w["correction"], int(router["top"]), router.get("groups"))
    if log is not None:
        choice = (scores + w["correction"]).tolist()
        log.append(torch.tensor([choice_margin(choice[t], ids[t], router.get("groups")) / max(scores[t].tolist()) for t in range(len(ids))]))
    out = torch.zeros_like(h)
    for t, chosen in enumerate(ids):
        for e in chosen:
            y = h[t] if e >= E else squared_relu(h[t] @ w[f"e{e}.up"].T) @ w[f"e{e}.down"].T
            out[t] += scores[t, e] * y
    return out


# ---------------------------------------------------------------------------------------------- the model
def _under(weights: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(raw: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, streams: Optional[list] = None,
            log: Optional[list] = None) -> torch.Tensor:
    """Logits [L, vocab].  ``streams`` receives the residual stream behind every layer, ``log`` every router's margins
    (``choice_margin`` over the largest score, per token)."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = float(raw["norm"]["eps"])
    x = W["embed"][torch.tensor(tokens)] * float(raw["embedding"]["scale"])
    rows = {}
    for i, layer in enumerate(raw["layers"]):
        p = f"l{i}."
        m, w = layer["mixer"], _under(W, p + "mix.")
        h = rms_norm_about_one(x, W[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                src = i
                rows[i] = latent_rows(h, w, m, eps)
            y = latent_attention(h, w, m, eps, rows[src])
        else:
            y = sigmoid_attention(h, w, m, eps)
        x = x + rms_norm_about_one(y, W[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_norm_about_one(x, W[p + "norm2"], eps)
            w = _under(W, p + "mlp.")
            y = dense(h, w) if mlp["kind"] == "dense" else mixture(h, w, mlp, log)
            x = x + rms_norm_about_one(y, W[p + "norm2b"], eps)
        if streams is not None:
            streams.append(x)
    return rms_norm_about_one(x, W["final.norm"], eps) @ W["head"].T
