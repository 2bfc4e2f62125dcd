"""Kernels around a selective state-space recurrence (`csrc/state_space.cu`): its step sizes and decays, and the skip, gate and
grouped norm of its result.  The recurrence itself is `recurrent.head_scan`, the convolution in front `recurrent.short_conv`."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from typing import Optional

import torch

from . import build, ops
from .attention_kv import _columns
from .build import KernelError

SOURCE = "state_space.cu"
ops.register_signatures(SOURCE, {
    "mlb_ssm_steps": [c_void_p, c_longlong, c_int, c_longlong, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                      c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p],
    "mlb_gated_group_norm": [c_void_p, c_void_p, c_longlong, c_void_p, c_void_p, c_longlong, c_int, c_longlong, c_int, c_void_p, c_void_p,
                             c_int, c_int, c_int, c_int, c_int, c_float, c_void_p],
})


def sources():
    return [(SOURCE, {}), ("delta_rule.cu", {}), ("short_conv.cu", {})]


def steps(proj: torch.Tensor, dt_col: int, dt_bias: torch.Tensor, a_log: torch.Tensor, dt: torch.Tensor, decay: torch.Tensor, ctx,
          conv_col: int = 0, conv_state: Optional[torch.Tensor] = None, slots: Optional[torch.Tensor] = None) -> None:
    """dt [T, heads] = softplus(proj[:, dt_col + h] + dt_bias[h]), decay = exp(-exp(a_log[h]) * dt); `proj` fp32 rows or their
    partial results.  With `conv_state` [slots, taps - 1, C] the state of a convolution over the columns from conv_col moves on to
    the step's last inputs (call this behind `recurrent.short_conv(..., update_state=False)`)."""
    _, ld, n, stride = _columns(proj, "proj")
    T, H = dt.shape
    for name, t, shape in (("dt", dt, (proj.shape[-2], H)), ("decay", decay, (T, H)), ("dt_bias", dt_bias, (H,)), ("a_log", a_log, (H,))):
        ops._need(t, name, torch.float32)
        if tuple(t.shape) != shape:
            raise KernelError(f"state_space.steps: {name} must be {shape}, got {tuple(t.shape)}")
    if dt_col + H > ld:
        raise KernelError("state_space.steps: the projection has no such columns")
    hist = channels = num_slots = 0
    if conv_state is not None:
        ops._need(conv_state, "conv_state", torch.float32, 3)
        num_slots, hist, channels = conv_state.shape
        if conv_col + channels > ld:
            raise KernelError("state_space.steps: the projection has no such columns")
    L = ops.lib(SOURCE)
    build.check(L, L.mlb_ssm_steps(proj.data_ptr(), ld, n, stride, int(dt_col), dt_bias.data_ptr(), a_log.data_ptr(), dt.data_ptr(),
                                   decay.data_ptr(), T, H, int(conv_col), channels, hist, ops._ptr(conv_state), ops._ptr(slots), num_slots,
                                   ctx.seq_starts.data_ptr(), ctx.num_seqs, ops._stream()))


def gated_group_norm(o: torch.Tensor, x: torch.Tensor, d: torch.Tensor, z: torch.Tensor, z_col: int, weight: torch.Tensor, out: torch.Tensor,
                     heads: int, dv: int, groups: int, eps: float) -> None:
    """out = n((o + d[h] * x) * silu(z columns from z_col)) * weight in out's dtype, n dividing each of `groups` equal parts of
    the row by its own root mean square.  `x`: a column view [T, heads * dv] of fp32 rows; `z`: fp32 rows or partial results."""
    ops._need(o, "o", torch.float32, 2); ops._need(out, "out", dims=2); ops._need(d, "d", torch.float32, 1)
    ops._need(weight, "weight", torch.float32, 1)
    _, ld, n, stride = _columns(z, "z")
    T, width = o.shape
    if (width != heads * dv or tuple(out.shape) != (T, width) or tuple(x.shape) != (T, width) or x.dtype != torch.float32 or x.stride(1) != 1
            or d.shape[0] != heads or weight.shape[0] != width or z_col + width > ld or z.shape[-2] != T or groups <= 0 or width % groups):
        raise KernelError("state_space.gated_group_norm: shapes do not agree")
    L = ops.lib(SOURCE)
    build.check(L, L.mlb_gated_group_norm(o.data_ptr(), x.data_ptr(), x.stride(0), d.data_ptr(), z.data_ptr(), ld, n, stride, int(z_col),
                                          weight.data_ptr(), out.data_ptr(), ops.dtype_tag(out), T, heads, dv, groups, float(eps), ops._stream()))
