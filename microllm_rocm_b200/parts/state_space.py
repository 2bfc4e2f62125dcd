"""Selective state space: a recurrent mixer whose state is one matrix per head, with one step size per token and head.

  [z | x | B | C | dt] = Win u      z, x: heads x vdim;  B, C: groups x state (head h reads group h // (heads / groups));  dt: heads
  x, B, C through a short causal convolution over time per channel (`conv` taps, with a bias) and silu
  dt = softplus(dt + dt_bias)
  per head, S [state, vdim] from zero:  S <- exp(-exp(A_log) dt) S + dt B x^T;   y = S^T C + D x
  y * silu(z), divided by the root mean square of each of `norm_groups` equal parts of the row, times a weight;  then Wo

B and C are the k and q of `recurrent.head_scan` (one decay per token and head, a weight dt on what is added), shared by the
heads of a group.  The state (S, fp32) and the convolution's last taps - 1 inputs live in the request's state slot.
Everything between the projection and the last product is fp32.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..kernels import gemm_bf16, recurrent, state_space
from ..kernels.linear import linear
from .base import CompositeNeed, FixedStateNeed, Mixer, PositionEncoding, Runtime, StepContext, WeightSpec, register_mixer


@register_mixer("selective_state_space")
class SelectiveStateSpace(Mixer):
    graph_safe = True

    def __init__(self, params: dict, rt: Runtime, position: Optional[PositionEncoding] = None):
        self.prefix = params.get("prefix", "")
        self.hidden = int(params["hidden_size"])
        self.nh, self.dv = int(params["num_heads"]), int(params["vdim"])
        self.groups, self.state = int(params["groups"]), int(params["state"])
        self.taps = int(params.get("conv", 1))
        self.norm_groups = int(params.get("norm_groups", 1))
        self.eps = float(params.get("eps", 1e-6))
        self.inner = self.nh * self.dv
        if self.nh % self.groups or self.inner % self.norm_groups:
            raise ValueError("selective_state_space: groups divide the heads, norm_groups the heads' columns")
        if not (0 < self.state <= recurrent.MAX_WIDTH and self.dv > 0):
            raise ValueError(f"selective_state_space: a state of {self.state} x {self.dv} per head (at most {recurrent.MAX_WIDTH} rows)")
        if not 1 <= self.taps <= recurrent.MAX_TAPS:
            raise ValueError(f"selective_state_space: {self.taps} taps (1..{recurrent.MAX_TAPS})")
        names = {"in": "in_proj.weight", "conv": "conv.weight", "conv_bias": "conv.bias", "dt_bias": "dt_bias", "a_log": "A_log", "d": "D",
                 "norm": "norm.weight", "o": "out_proj.weight"}
        names.update(params.get("names", {}))
        self.names = names
        self.rt = rt
        # columns of the projection: z | x | B | C | dt, rows padded to a multiple of 8, which the products like
        self.bc_cols = self.groups * self.state
        self.conv_cols = self.inner + 2 * self.bc_cols
        self.dt_col = self.inner + self.conv_cols
        self.used_rows = self.dt_col + self.nh
        self.in_rows = -(-self.used_rows // 8) * 8
        self.w_in = self.w_o = self.w_conv = self.b_conv = self.dt_bias = self.a_log = self.d = self.norm_w = None

    # --- declarations -----------------------------------------------------------------
    def cache_need(self):
        items = [("state", FixedStateNeed((self.nh, self.state, self.dv), torch.float32))]
        if self.taps > 1:
            items.append(("conv", FixedStateNeed((self.taps - 1, self.conv_cols), torch.float32)))
        return CompositeNeed(tuple(items))

    def weight_specs(self) -> Dict[str, WeightSpec]:
        n, vector = self.names, lambda shape, init: WeightSpec(shape, role="vector", init=init)
        return {n["in"]: WeightSpec((self.used_rows, self.hidden)), n["o"]: WeightSpec((self.hidden, self.inner)),
                n["conv"]: vector((self.conv_cols, self.taps), ("normal", 0.5)), n["conv_bias"]: vector((self.conv_cols,), ("normal", 0.1)),
                n["dt_bias"]: vector((self.nh,), ("normal", 1.0)), n["a_log"]: vector((self.nh,), ("normal", 0.5)),
                n["d"]: vector((self.nh,), ("one_plus_normal", 0.1)), n["norm"]: vector((self.inner,), ("one_plus_normal", 0.1))}

    def fused_tensors(self):
        # (one piece: the padding rows behind it are what the fused tensor adds)
        return {"in_proj.padded": (WeightSpec((self.in_rows, self.hidden)), [(self.names["in"], 0)])}

    def kernel_sources(self):
        own = state_space.sources()
        return own if self.rt.is_fp32 else own + gemm_bf16.sources(engine_only=True)

    def bind(self, tensors):
        n = self.names
        if "in_proj.padded" in tensors:
            self.w_in = tensors["in_proj.padded"]
            self.w_in[self.used_rows:].zero_()           # the padding rows: their columns of the product are never read
        else:
            w = tensors[n["in"]]
            self.w_in = torch.zeros((self.in_rows, self.hidden), dtype=w.dtype, device=w.device)
            self.w_in[:self.used_rows] = w
        self.w_conv, self.b_conv = tensors[n["conv"]], tensors[n["conv_bias"]]
        self.dt_bias, self.a_log, self.d = tensors[n["dt_bias"]], tensors[n["a_log"]], tensors[n["d"]]
        self.norm_w, self.w_o = tensors[n["norm"]], tensors[n["o"]]

    def replay_key(self):
        if not self.rt.is_fp32 and not gemm_bf16._direct_library(self.rt.device):
            return None                  # the library product would go through the tensor framework
        return ("selective_state_space", self.hidden, self.nh, self.dv, self.groups, self.state, self.taps, self.norm_groups, self.eps)

    def own_tensors(self):
        return [self.w_in, self.w_o, self.w_conv, self.b_conv, self.dt_bias, self.a_log, self.d, self.norm_w]

    # --- compute ------------------------------------------------------------------------
    def forward(self, x: torch.Tensor, ctx: StepContext, cache) -> torch.Tensor:
        T, flag, f32 = x.shape[0], ctx.error_flag, torch.float32
        state, conv = cache["state"], cache.get("conv")
        buf = lambda role, cols, dtype=f32: ctx.buffer("state_space." + role, (T, cols), dtype)
        proj = linear(x, self.w_in, None, f32, partials_ok=True, error_flag=flag,
                      alloc=lambda shape, dtype: ctx.buffer("state_space.proj", shape, dtype))
        u = buf("u", self.conv_cols)
        recurrent.short_conv(proj, self.inner, self.w_conv, conv.storage if conv is not None else None, state.slots, ctx, u, silu=True,
                             update_state=False, bias=self.b_conv)
        dt, decay = buf("dt", self.nh), buf("decay", self.nh)
        move = conv is not None and conv.writable
        state_space.steps(proj, self.dt_col, self.dt_bias, self.a_log, dt, decay, ctx, conv_col=self.inner,
                          conv_state=conv.storage if move else None, slots=conv.slots if move else None)
        xs, b, c = u[:, :self.inner], u[:, self.inner:self.inner + self.bc_cols], u[:, self.inner + self.bc_cols:]
        o = buf("o", self.inner)
        recurrent.head_scan(c, b, decay, xs, o, state.storage, state.slots, ctx, self.nh, self.state, self.dv, weight=dt, kv_heads=self.groups)
        gated = buf("gated", self.inner, self.rt.dtype)
        state_space.gated_group_norm(o, xs, self.d, proj, 0, self.norm_w, gated, self.nh, self.dv, self.norm_groups, self.eps)
        return linear(gated, self.w_o, None, f32, partials_ok=True, error_flag=flag,
                      alloc=lambda shape, dtype: ctx.buffer("state_space.out", shape, dtype))
