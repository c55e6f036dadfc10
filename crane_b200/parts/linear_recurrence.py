"""A mixer whose memory is one number per channel (Griffin's recurrent block with a real-gated linear
recurrent unit).  Two branches of C channels, y = gelu_tanh(W_y x + b_y) and u = conv(W_x x + b_x) + c with a
causal convolution over time per channel; u in equal parts b, each through two square matrices of its own:

    r = sigmoid(R_b u_b + rb),  i = sigmoid(I_b u_b + ib),  a = exp(-8 r softplus(lam))
    S <- a S + sqrt(1 - a^2) i u;   out = W_o (S y)

The state, the convolution and everything between u and S are 32-bit.  Prompts and portions: one kernel forms a and
the addend of every token, a second one walks them; single tokens: the first kernel does both.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from ..kernels import step_of_single_tokens
from ..weights.loader import TensorSpec
from .base import CacheNeed, Part, register_part


@register_part("mixer", "gated_linear_recurrence")
class GatedLinearRecurrence(Part):
    """params: ``hidden_size``, ``channels``, ``blocks`` (the equal parts), ``conv`` (taps), ``names``.  Tensors: y, x
    [C, hidden], o [hidden, C], gate_r, gate_i [blocks, C / blocks, C / blocks] ([out, in] each), and in 32-bit y_bias,
    x_bias, conv_bias, lam [C], conv [C, taps], gate_r_bias, gate_i_bias [blocks, C / blocks].  The request's slot
    holds the states and the convolution's last inputs."""
    kind = "mixer"
    state_graph_safe = True
    decode_bucket_safe = True
    NAMES = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "gate_r": "ra",
             "gate_r_bias": "ra.b", "gate_i": "ri", "gate_i_bias": "ri.b", "lam": "lam", "o": "o"}
    MAX_TAPS = 16

    @classmethod
    def manifest(cls, spec):
        a, p = spec.params, spec.prefix
        w, C, B, T = (int(a[k]) for k in ("hidden_size", "channels", "blocks", "conv"))
        nm = {k: p + v for k, v in dict(cls.NAMES, **(a.get("names") or {})).items()}
        c = C // B
        return {nm["y"]: TensorSpec((C, w)), nm["x"]: TensorSpec((C, w)), nm["o"]: TensorSpec((w, C)),
                nm["gate_r"]: TensorSpec((B, c, c)), nm["gate_i"]: TensorSpec((B, c, c)),
                nm["y_bias"]: TensorSpec((C,), "float32", "offset"), nm["x_bias"]: TensorSpec((C,), "float32", "offset"),
                nm["conv"]: TensorSpec((C, T), "float32", "unit"), nm["conv_bias"]: TensorSpec((C,), "float32", "offset"),
                nm["gate_r_bias"]: TensorSpec((B, c), "float32", "offset"),
                nm["gate_i_bias"]: TensorSpec((B, c), "float32", "offset"), nm["lam"]: TensorSpec((C,), "float32", "slow")}

    def load(self, weights, rt):
        a, p = self.params, self.prefix
        self.C, blocks, taps = (int(a[k]) for k in ("channels", "blocks", "conv"))
        if blocks <= 0 or self.C % blocks or not 1 <= taps <= self.MAX_TAPS:
            raise ValueError(f"{p}: {self.C} channels in {blocks} equal parts with {taps} taps (1 .. {self.MAX_TAPS})")
        w = {k: weights.pop(p + v) for k, v in dict(self.NAMES, **(a.get("names") or {})).items()}
        self.w_in = torch.cat([w["y"], w["x"]], dim=0).contiguous()                   # one product: [y | x]
        self.b_in = torch.cat([w["y_bias"], w["x_bias"]]).contiguous()
        self.o_w = w["o"]
        gates, mma = rt.kernels.pack_gates(w["gate_r"], w["gate_i"], rt.exact)
        self.scan = rt.kernels.GateScan(
            y_off=0, x_off=self.C, s_off=0, ring_off=self.C, conv_w=w["conv"].t().contiguous(), conv_b=w["conv_bias"],
            gates=gates, mma=mma, rb=w["gate_r_bias"].reshape(-1).contiguous(), ib=w["gate_i_bias"].reshape(-1).contiguous(),
            sp=F.softplus(w["lam"].double(), threshold=60.0).float().contiguous(), parts=blocks)
        self.floats = self.C * (1 + taps)

    def cache_need(self) -> CacheNeed:
        return CacheNeed("state", state_shape=(self.floats,), state_dtype=torch.float32)

    def forward(self, h, ctx, cache, rt, hold: bool = False):
        n, k = h.shape[0], rt.kernels
        proj = rt.linear(h, self.w_in, self.b_in, "lin_proj")
        aux = rt.ws.get("lin_aux", n, 2 * self.C, torch.float32)
        o = rt.ws.get("lin_o", n, self.C, rt.dtype)
        k.gate_scan_prep(proj, 2 * self.C, ctx, cache.state, self.scan, aux, o, rt.err, rt.dtype)
        if step_of_single_tokens(ctx):
            rt.launches += 1
        else:
            k.channel_scan(aux, proj, 2 * self.C, ctx, cache.state, self.scan, o, rt.err)
            rt.launches += 2
        return rt.linear(o, self.o_w, None, "lin_out", hold=hold)
