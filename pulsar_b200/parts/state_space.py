"""The state-space mixer with one decay per head (the dual form of linear attention): convolution, recurrence, gated norm."""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import ops
from ..cache.manager import CacheNeed
from ..config.registry import MIXERS
from ..config.specs import MixerSpec
from .base import CacheView, Mixer, StepContext, WeightSpec


@MIXERS.register("state_space_dual")
class StateSpaceDual(Mixer):
    """W_in h = [z: inner | x: inner | B: groups * state | C: groups * state | dt: heads], inner = ``n_heads`` * ``value_dim``.  x, B and C
    pass a causal convolution of ``conv`` taps per channel with a bias, and silu.  dt = softplus(dt + dt_bias) per head; head h reads
    B and C of group floor(h / (heads / groups)); S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T (a matrix [state, value_dim]),
    y_t = S_t^T C_t + D_h x_t.  The concatenated heads are multiplied by silu(z), normed in ``norm_groups`` equal parts (each by its own
    root mean square, ``norm_eps`` inside the root), multiplied by a weight and projected by W_o.

    The state of a sequence (all heads' matrices and the convolution's last ``conv - 1`` inputs per channel, float32) lives in the
    sequence's slot of the cache manager's state arena; it starts at zero and is carried from step to step.  The input
    projection has float32 rows; everything behind it is ``ops.state_space``: token by token (the convolution in the same kernel)
    for steps of single tokens, short portions and the float32 engine, in chunks that run side by side on the tensor cores for
    longer portions in bfloat16.  The kernels take what they need to know about the step from the step's device arrays, so a
    step of single tokens can be replayed from a CUDA graph.

    Options (``spec.extra``): ``state``, ``groups``, ``conv``, ``norm_groups``.
    Tensor names by role "in", "conv", "conv_bias", "dt_bias", "a_log", "d", "norm", "o".
    """

    def __init__(self, spec: MixerSpec, prefix: str, dtype: torch.dtype):
        self.n_state, self.n_groups = int(spec.option("state", 0)), int(spec.option("groups", 1))
        self.taps, self.norm_groups = int(spec.option("conv", 0)), int(spec.option("norm_groups", 1))
        if min(spec.n_heads, spec.value_dim, self.n_state, self.n_groups, self.taps, self.norm_groups) <= 0:
            raise ValueError("state space: heads, head size, state, groups, conv and norm_groups must be positive")
        self.inner = spec.n_heads * spec.value_dim
        if spec.n_heads % self.n_groups or self.inner % self.norm_groups:
            raise ValueError(f"state space: {spec.n_heads} heads in {self.n_groups} groups and {self.inner} channels in {self.norm_groups} "
                             "normed parts do not divide evenly")
        self.channels = self.inner + 2 * self.n_groups * self.n_state        # those that pass the convolution
        self.spec, self.prefix, self.dtype = spec, prefix, dtype
        name = spec.tensor_name
        self.names = {r: name(r, d) for r, d in (("in", "in_proj.weight"), ("conv", "conv1d.weight"), ("conv_bias", "conv1d.bias"),
                                                 ("dt_bias", "dt_bias"), ("a_log", "A_log"), ("d", "D"), ("norm", "norm.weight"),
                                                 ("o", "out_proj.weight"))}
        self.w: Dict[str, torch.Tensor] = {}

    def weight_specs(self) -> List[WeightSpec]:
        s, p, nm = self.spec, self.prefix, self.names
        return [WeightSpec(p + nm["in"], (self.inner + self.channels + s.n_heads, s.hidden)),
                WeightSpec(p + nm["conv"], (self.channels, self.taps), role="vector", init="taps"),
                WeightSpec(p + nm["conv_bias"], (self.channels,), role="vector", init="small"),
                WeightSpec(p + nm["dt_bias"], (s.n_heads,), role="vector", init="step_bias"),
                WeightSpec(p + nm["a_log"], (s.n_heads,), role="vector", init="decay_log"),
                WeightSpec(p + nm["d"], (s.n_heads,), role="vector", init="ones_normal"),
                WeightSpec(p + nm["norm"], (self.inner,), role="vector", init="ones_normal"),
                WeightSpec(p + nm["o"], (s.hidden, self.inner))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w = {role: tensors[self.prefix + n] for role, n in self.names.items()}
        w_in = self.w["in"]
        if w_in.shape[0] % 16:               # whole tiles of sixteen rows for the products (the padding's columns go unread)
            self.w["in"] = torch.cat([w_in, w_in.new_zeros(-w_in.shape[0] % 16, w_in.shape[1])], dim=0).contiguous()

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.w.values())

    def cache_need(self) -> CacheNeed:
        return CacheNeed.state((self.inner * self.n_state + self.channels * (self.taps - 1),), torch.float32)

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: CacheView) -> torch.Tensor:
        s, n, w = self.spec, ctx.n_tokens, self.w
        rows = ctx.scratch("space.rows", (n, w["in"].shape[0]), torch.float32)
        ops.linear(h, w["in"], rows)
        y = ctx.scratch("space.y", (n, self.inner))
        ops.state_space(ctx, rows, w["conv"], w["conv_bias"], w["dt_bias"], w["a_log"], w["d"], w["norm"], self.norm_groups, s.norm_eps,
                        cache.state, y, s.n_heads, self.n_state, s.value_dim, self.n_groups)
        out = ctx.scratch("space.out", (n, s.hidden), torch.float32 if self.output_float32 else None)
        ops.linear(y, w["o"], out)
        return out
