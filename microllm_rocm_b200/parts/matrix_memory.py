"""Two mixers whose state is one matrix per head with ONE decay per head (beside the mixers with a decay per key channel in
`linear_attention.py`):

`retention`
  q, k = Wq x, Wk x  (heads x dim),  v = Wv x  (heads x vdim);  q and k rotated by the position encoding's table (split halves),
  k then times k_scale (dim^-1/2)
  per head, S [dim, vdim] from zero:  S <- d_h S + k_t v_t^T;  o_t = S^T q_t  with a FIXED decay d_h per head
  o / rms(o) per head (no weight) * silu(Wg x),  then Wo

`mlstm`
  q = Wq x * dim^-1/2,  k = Wk x  (heads x dim),  v = Wv x  (heads x vdim)
  per head  i = c tanh((Wi x + bi) / c),  f = log sigmoid(c tanh((Wf x + bf) / c))  (logs of the gates, capped at c)
  m_t = max(f + m_(t-1), i) from 0;  S <- e^(f + m_(t-1) - m_t) S + e^(i - m_t) k_t v_t^T,  n likewise with k_t alone
  o_t = S^T q_t / (max(|n . q_t|, e^(-m_t)) + 1e-6)
  o / rms(o) per head * weight (heads x vdim) * sigmoid(Wg x),  then Wo

All projections that read x are one fused product.  Everything between it and the output projection is fp32: the rotation,
the gates and their exponentials, the recurrence and its states (matrix, vector, running maximum), the per-head norm.
The vector n is one more column of the matrix's recurrence (a value of 1), so one scan makes numerator and denominator."""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..kernels import gemm_bf16, linear_attention, ops, recurrent
from ..kernels.linear import linear
from .base import CompositeNeed, FixedStateNeed, Mixer, PositionEncoding, Runtime, StepContext, WeightSpec, register_mixer
from .linear_attention import _check_widths

DENOMINATOR_EPS = 1e-6


class HeadDecayMixer(Mixer):
    """What the two share: the fused projection q | k | v | gate | (more rows), its padding, the output projection."""
    graph_safe = True
    kind = ""

    def __init__(self, params: dict, rt: Runtime, names: dict, extra: Tuple[str, ...] = ()):
        self.prefix = params.get("prefix", "")
        self.hidden = int(params["hidden_size"])
        self.nh = int(params["num_heads"])
        self.dk, self.dv = int(params["dim"]), int(params["vdim"])
        self.eps = float(params.get("eps", 1e-6))
        _check_widths(self.kind, self.dk, self.dv)
        self.names = dict(q="q_proj.weight", k="k_proj.weight", v="v_proj.weight", gate="g_proj.weight", o="o_proj.weight", **names)
        self.names.update(params.get("names", {}))
        self.rt = rt
        self.qk_cols, self.v_cols = self.nh * self.dk, self.nh * self.dv
        self.k_col, self.v_col = self.qk_cols, 2 * self.qk_cols
        self.g_col = self.v_col + self.v_cols
        self.extra_cols = {}                       # name of an extra projection with one row per head -> its first column
        at = self.g_col + self.v_cols
        for name in extra:
            self.extra_cols[name] = at
            at += self.nh
        self.used_rows = at
        self.in_rows = -(-at // 8) * 8             # padded to a multiple of 8 rows, which the products like
        self.w_in = self.w_o = None

    def _pieces(self) -> List[Tuple[str, int]]:
        n = self.names
        return [(n["q"], 0), (n["k"], self.k_col), (n["v"], self.v_col), (n["gate"], self.g_col)] + \
            [(n[name], col) for name, col in self.extra_cols.items()]

    def weight_specs(self) -> Dict[str, WeightSpec]:
        n, W = self.names, self.hidden
        specs = {n["q"]: WeightSpec((self.qk_cols, W)), n["k"]: WeightSpec((self.qk_cols, W)), n["v"]: WeightSpec((self.v_cols, W)),
                 n["gate"]: WeightSpec((self.v_cols, W)), n["o"]: WeightSpec((W, self.v_cols))}
        specs.update({n[name]: WeightSpec((self.nh, W)) for name in self.extra_cols})
        return specs

    def fused_tensors(self):
        return {"in_proj.weight": (WeightSpec((self.in_rows, self.hidden)), self._pieces())}

    def kernel_sources(self):
        own = linear_attention.sources()
        return own if self.rt.is_fp32 else own + gemm_bf16.sources(engine_only=True)

    def bind(self, tensors):
        if "in_proj.weight" in tensors:
            self.w_in = tensors["in_proj.weight"]
            self.w_in[self.used_rows:].zero_()           # the padding rows: their columns of the product are never read
        else:
            pieces = [tensors[name] for name, _ in self._pieces()]
            if self.in_rows > self.used_rows:
                pieces.append(torch.zeros((self.in_rows - self.used_rows, self.hidden), dtype=pieces[0].dtype, device=pieces[0].device))
            self.w_in = torch.cat(pieces, 0).contiguous()
        self.w_o = tensors[self.names["o"]]

    def _replayable(self) -> bool:
        return self.rt.is_fp32 or gemm_bf16._direct_library(self.rt.device)

    def _project(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        return linear(x, self.w_in, None, torch.float32, partials_ok=True, error_flag=ctx.error_flag,
                      alloc=lambda shape, dtype: ctx.buffer("head_decay.proj", shape, dtype))

    def _out(self, gated: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        return linear(gated, self.w_o, None, torch.float32, partials_ok=True, error_flag=ctx.error_flag,
                      alloc=lambda shape, dtype: ctx.buffer("head_decay.out", shape, dtype))

    def _buffers(self, T: int, ctx: StepContext):
        buf = lambda role, cols: ctx.buffer("head_decay." + role, (T, cols), torch.float32)
        return buf("q", self.qk_cols), buf("k", self.qk_cols), buf("v", self.v_cols), buf("o", self.v_cols)


@register_mixer("retention")
class Retention(HeadDecayMixer):
    kind = "retention"

    def __init__(self, params: dict, rt: Runtime, position: Optional[PositionEncoding] = None):
        super().__init__(params, rt, {})
        self.decay_values = tuple(float(d) for d in params["decay"])
        if len(self.decay_values) != self.nh:
            raise ValueError("retention: one decay per head")
        self.k_scale = float(params.get("k_scale", self.dk ** -0.5))
        self.rotary = position.rotary_table(self.dk) if position is not None else None
        if self.rotary is not None and (self.rotary.interleaved or self.rotary.magnitude != 1.0):
            raise ValueError("retention turns split halves with plain cosines and sines")
        # layers with the same rotation share a step's table of cosines and sines
        rot = params.get("position")
        self.rotation_key = ("retention.rotation", tuple(sorted(rot.params.items()))) if self.rotary is not None else None
        self.head_decay = torch.tensor(self.decay_values, dtype=torch.float32, device=rt.device)     # a constant of the design, not a weight

    def kernel_sources(self):
        return super().kernel_sources() + ([("rope_kv.cu", {})] if self.rotary is not None else [])

    def cache_need(self):
        return CompositeNeed((("state", FixedStateNeed((self.nh, self.dk, self.dv), torch.float32)),))

    def replay_key(self):
        if not self._replayable():
            return None
        return ("retention", self.hidden, self.nh, self.dk, self.dv, self.eps, self.k_scale, self.rotation_key)

    def own_tensors(self):
        return [self.w_in, self.w_o, self.head_decay]

    def _cos_sin(self, ctx: StepContext, T: int) -> Optional[torch.Tensor]:
        if self.rotary is None:
            return None
        table = ctx.step_values.get(self.rotation_key)
        if table is None:
            out = ctx.buffer(self.rotation_key, (T, self.rotary.rotary_dim // 2, 2), torch.float32)
            table = ctx.step_values[self.rotation_key] = ops.rope_table(ctx.positions, self.rotary.inv_freq, out=out)
        return table

    def forward(self, x: torch.Tensor, ctx: StepContext, cache) -> torch.Tensor:
        T, state = x.shape[0], cache["state"]
        proj = self._project(x, ctx)
        q, k, v, o = self._buffers(T, ctx)
        linear_attention.head_decay_prepare(proj, 0, self.k_col, self.v_col, q, k, v, self.nh, self.dk, self.dv, ctx, k_scale=self.k_scale,
                                            cos_sin=self._cos_sin(ctx, T))
        recurrent.head_scan(q, k, self.head_decay, v, o, state.storage, state.slots, ctx, self.nh, self.dk, self.dv)
        gated = ctx.buffer("head_decay.gated", (T, self.v_cols), self.rt.dtype)
        linear_attention.head_norm_gate(o, None, proj, self.g_col, "silu", gated, self.nh, self.dv, self.eps)
        return self._out(gated, ctx)


@register_mixer("mlstm")
class MatrixLSTM(HeadDecayMixer):
    kind = "mlstm"

    def __init__(self, params: dict, rt: Runtime, position: Optional[PositionEncoding] = None):
        super().__init__(params, rt, dict(i="i_proj.weight", f="f_proj.weight", i_bias="i_proj.bias", f_bias="f_proj.bias", norm="o_norm.weight"),
                         extra=("i", "f"))
        self.cap = float(params["gate_cap"])
        if not self.cap > 0:
            raise ValueError("mlstm: gate_cap must be positive")
        self.q_scale = float(params.get("q_scale", self.dk ** -0.5))
        self.i_bias = self.f_bias = self.norm_w = None

    def cache_need(self):
        f32 = torch.float32
        return CompositeNeed((("state", FixedStateNeed((self.nh, self.dk, self.dv), f32)), ("n", FixedStateNeed((self.nh, self.dk), f32)),
                              ("m", FixedStateNeed((self.nh,), f32))))

    def weight_specs(self) -> Dict[str, WeightSpec]:
        n, specs = self.names, super().weight_specs()
        specs[n["i_bias"]] = WeightSpec((self.nh,), role="vector", init=("normal", 1.0))
        specs[n["f_bias"]] = WeightSpec((self.nh,), role="vector", init=("normal", 2.0))
        specs[n["norm"]] = WeightSpec((self.v_cols,), role="vector", init=("one_plus_normal", 0.1))
        return specs

    def bind(self, tensors):
        super().bind(tensors)
        n = self.names
        self.i_bias, self.f_bias, self.norm_w = tensors[n["i_bias"]], tensors[n["f_bias"]], tensors[n["norm"]]

    def replay_key(self):
        if not self._replayable():
            return None
        return ("mlstm", self.hidden, self.nh, self.dk, self.dv, self.eps, self.cap, self.q_scale)

    def own_tensors(self):
        return [self.w_in, self.w_o, self.i_bias, self.f_bias, self.norm_w]

    def forward(self, x: torch.Tensor, ctx: StepContext, cache) -> torch.Tensor:
        T, state = x.shape[0], cache["state"]
        proj = self._project(x, ctx)
        q, k, v, o = self._buffers(T, ctx)
        gates = ctx.buffer("head_decay.gates", (3, T, self.nh), torch.float32)          # what is kept, what is taken, e^-m
        linear_attention.head_decay_prepare(proj, 0, self.k_col, self.v_col, q, k, v, self.nh, self.dk, self.dv, ctx, q_scale=self.q_scale,
                                            gates=gates, i_col=self.extra_cols["i"], f_col=self.extra_cols["f"], i_bias=self.i_bias,
                                            f_bias=self.f_bias, cap=self.cap, m_state=cache["m"].storage, slots=cache["m"].slots)
        den = ctx.buffer("head_decay.den", (T, self.nh), torch.float32)
        recurrent.head_scan(q, k, gates[0], v, o, state.storage, state.slots, ctx, self.nh, self.dk, self.dv, weight=gates[1],
                            n_state=cache["n"].storage, den=den)
        gated = ctx.buffer("head_decay.gated", (T, self.v_cols), self.rt.dtype)
        linear_attention.head_norm_gate(o, self.norm_w, proj, self.g_col, "sigmoid", gated, self.nh, self.dv, self.eps, den=den, floor=gates[2],
                                        den_eps=DENOMINATOR_EPS)
        return self._out(gated, ctx)
