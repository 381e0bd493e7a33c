"""Matrix memory with exponential gates: a float32 matrix, a normaliser and a running maximum per head and sequence."""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import ops
from ..cache.manager import CacheNeed
from ..config.registry import MIXERS
from ..config.specs import MixerSpec
from .base import CacheView, Mixer, StepContext, WeightSpec


@MIXERS.register("matrix_memory")
class MatrixMemory(Mixer):
    """q = W_q h * ``q_scale`` and k = W_k h have ``n_heads`` heads of ``head_dim``, v = W_v h heads of ``value_dim``.  Per head a log
    input gate i = cap tanh((W_i h + b_i) / cap) and a log forget gate f = logsigmoid(cap tanh((W_f h + b_f) / cap)), cap =
    ``gate_cap``.  With the running maximum m_t = max(f + m_(t-1), i), zero before the first token,
    S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T, n_t likewise with k alone, and the head's output is
    o = S_t^T q / (max(|n_t . q|, exp(-m_t)) + ``denom_eps``).  Each head's o is divided by its root mean square (``norm_eps`` inside the
    root); the concatenated heads are multiplied by a weight and by sigmoid(W_g h), and projected by W_o.

    The state of a sequence (all heads' S, n and m, float32) lives in the sequence's slot of the cache manager's state arena; it
    starts at zero and is carried from step to step.  The six projections of h are one product with float32 rows
    (q | k | v | g | i | f); the gates, the recurrence, the norm and the output gate follow in ``ops.matrix_memory``: token by token for
    steps of single tokens, short portions and the float32 engine, in chunks that run side by side on the tensor cores for longer
    portions in bfloat16.  The kernels take what they need to know about the step from the step's device arrays, so a step of
    single tokens can be replayed from a CUDA graph.

    Options (``spec.extra``): ``gate_cap``, ``q_scale`` (default ``head_dim`` ** -0.5), ``denom_eps`` (default 1e-6).
    Tensor names by role "q", "k", "v", "g", "i", "f", "i_bias", "f_bias", "norm", "o".
    """

    def __init__(self, spec: MixerSpec, prefix: str, dtype: torch.dtype):
        if spec.n_heads <= 0 or spec.head_dim <= 0 or spec.value_dim <= 0:
            raise ValueError("matrix memory: heads and head sizes must be positive")
        self.cap = float(spec.option("gate_cap", 0.0))
        if not (self.cap > 0.0):
            raise ValueError("matrix memory: the cap on the gates must be positive")
        self.spec, self.prefix, self.dtype = spec, prefix, dtype
        self.q_scale = float(spec.option("q_scale", spec.head_dim ** -0.5))
        self.denom_eps = float(spec.option("denom_eps", 1e-6))
        name = spec.tensor_name
        self.names = {r: name(r, d) for r, d in (("q", "q_proj.weight"), ("k", "k_proj.weight"), ("v", "v_proj.weight"), ("g", "g_proj.weight"),
                                                 ("i", "i_gate.weight"), ("f", "f_gate.weight"), ("i_bias", "i_gate.bias"),
                                                 ("f_bias", "f_gate.bias"), ("norm", "norm.weight"), ("o", "o_proj.weight"))}
        self.w_in = self.w_o = self.b_i = self.b_f = self.norm = None

    def weight_specs(self) -> List[WeightSpec]:
        s, p, nm = self.spec, self.prefix, self.names
        qk, v = s.n_heads * s.head_dim, s.n_heads * s.value_dim
        return [WeightSpec(p + nm["q"], (qk, s.hidden)), WeightSpec(p + nm["k"], (qk, s.hidden)), WeightSpec(p + nm["v"], (v, s.hidden)),
                WeightSpec(p + nm["g"], (v, s.hidden)), WeightSpec(p + nm["i"], (s.n_heads, s.hidden)),
                WeightSpec(p + nm["f"], (s.n_heads, s.hidden)), WeightSpec(p + nm["i_bias"], (s.n_heads,), role="vector", init="small"),
                WeightSpec(p + nm["f_bias"], (s.n_heads,), role="vector", init="forget_bias"),
                WeightSpec(p + nm["norm"], (v,), role="vector", init="ones_normal"), WeightSpec(p + nm["o"], (s.hidden, v))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        p, nm = self.prefix, self.names
        parts = [tensors[p + nm[r]] for r in ("q", "k", "v", "g", "i", "f")]
        # rows: q | k | v | g | i | f, filled up to whole tiles of sixteen for the products (the padding's columns go unread)
        parts.append(parts[0].new_zeros(-sum(t.shape[0] for t in parts) % 16, self.spec.hidden))
        self.w_in = torch.cat(parts, dim=0).contiguous()
        self.w_o = tensors[p + nm["o"]]
        self.b_i, self.b_f, self.norm = tensors[p + nm["i_bias"]], tensors[p + nm["f_bias"]], tensors[p + nm["norm"]]

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_o, self.b_i, self.b_f, self.norm))

    def cache_need(self) -> CacheNeed:
        s = self.spec
        return CacheNeed.state((s.n_heads * (s.head_dim * s.value_dim + s.head_dim + 1),), torch.float32)

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: CacheView) -> torch.Tensor:
        s, n = self.spec, ctx.n_tokens
        rows = ctx.scratch("memory.rows", (n, self.w_in.shape[0]), torch.float32)
        ops.linear(h, self.w_in, rows)
        y = ctx.scratch("memory.y", (n, s.n_heads * s.value_dim))
        ops.matrix_memory(ctx, rows, self.b_i, self.b_f, self.cap, self.norm, s.norm_eps, cache.state, y, s.n_heads, s.head_dim, s.value_dim,
                          self.q_scale, self.denom_eps)
        out = ctx.scratch("memory.out", (n, s.hidden), torch.float32 if self.output_float32 else None)
        ops.linear(y, self.w_o, out)
        return out
