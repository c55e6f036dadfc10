"""Mixers whose memory is one matrix S [dim, vdim] per head and request, walked token by token:

    S <- diag(w_t) S;   u = beta_t (v_t - S^T k_t)  or  u = v_t;   S <- S + k_t u^T;   o_t = S^T q_t

``gated_linear_attention``: no correction (u = v), a decay per key channel
w = sigmoid(W_a2 (W_a1 x) + b)^(1 / tau), q scaled by dim^(-1/2).

``gated_delta``: the delta rule's correction with beta = sigmoid(W_b x) and one decay per head,
w = exp(-exp(A_log) softplus(W_a x + dt_bias)); q, k and v first pass a short causal convolution
over time and silu, q and k are scaled to unit length per head (q also by dim^(-1/2)); head h reads
q/k head h // (heads / kv_heads).  The convolutions' last taps - 1 inputs are state too.

Both norm each head's read-out over vdim (a plain weight shared by the heads), multiply by
silu(W_g x) and project.  ``gated_delta`` has two options: one decay per head AND key channel,
w = exp(-exp(A_log_h) softplus(W_a2 (W_a1 x) + dt_bias)), and a gate sigmoid(W_g2 (W_g1 x)).

``wkv_time_mix``: every projection reads a mix of its own of the token's row and the one before,
x + (x' - x) mu; r, k, v from three of them, a gate silu(W_g .), a decay per key channel
w = exp(-exp(W_w2 tanh(W_w1 .) + w0)); the read-out sees the state before the token's write and, of the
token itself, its write scaled per key channel by u:

    o_t = (S + diag(u) k_t v_t^T)^T r_t;   S <- diag(w_t) S + k_t v_t^T

``exponential_gates`` (the matrix memory of xLSTM): no correction, gates i and exp(f) per head whose
logarithms are capped, f = log sigmoid(.), kept in range by a running maximum M, which starts at 0:

    M' = max(f + M, i);  S <- exp(f + M - M') S + exp(i - M') k v^T;  N likewise with k alone
    o = S^T q / (max(|N . q|, exp(-M')) + eps)

State and everything between the projections and the output projection are 32-bit.  One kernel walks
the recurrence for all of them (``matrix_state_scan``), prompts, portions and single tokens alike, so a
state does not depend on how the tokens were cut.  (``exponential_gates`` has a second one, for portions of a
few tokens or more of large bfloat16 steps: ``memory_chunks``, 64 tokens at a time on the tensor cores, equal to
the walk but for 32-bit rounding.)
"""
from __future__ import annotations

from dataclasses import replace

import torch

from ..kernels import step_of_single_tokens
from ..weights.loader import TensorSpec
from .base import CacheNeed, Part, register_part


def _state_floats(rt, heads: int, dim: int, vdim: int, where: str) -> int:
    """Floats of a slot's states of ``heads`` heads with ``vdim`` columns each."""
    rows, lanes = rt.kernels.matrix_state_plan(dim)
    if rows == 0:
        raise ValueError(f"{where}: keys of {dim} elements are wider than the recurrence kernel takes")
    return heads * rows * lanes * vdim


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttention(Part):
    """params: ``hidden_size``, ``heads``, ``dim``, ``vdim``, ``tau``, ``norm_eps`` (of the head norm),
    ``decay_rank`` (inner size of the decay's two products; None: read from the stored tensor),
    ``names``.  Tensors: q, k [H dim, hidden], v, g [H vdim, hidden], o [hidden, H vdim],
    a1 [rank, hidden], a2 [H dim, rank], and in 32-bit a2_bias [H dim], norm [vdim]."""
    kind = "mixer"
    state_graph_safe = True      # the kernels read the step's metadata on the device, skip rows of no
                                 # entry and touch no slot for an entry without rows
    NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "a1": "a1", "a2": "a2", "a2_bias": "a2.b", "norm": "norm"}

    @classmethod
    def manifest(cls, spec):
        a, p = spec.params, spec.prefix
        w, H, d, m = int(a["hidden_size"]), int(a["heads"]), int(a["dim"]), int(a["vdim"])
        nm = dict(cls.NAMES, **(a.get("names") or {}))
        rank = a.get("decay_rank")
        rank, free = (-1, 16) if rank is None else (int(rank), 0)
        return {p + nm["q"]: TensorSpec((H * d, w)), p + nm["k"]: TensorSpec((H * d, w)),
                p + nm["v"]: TensorSpec((H * m, w)), p + nm["g"]: TensorSpec((H * m, w)),
                p + nm["o"]: TensorSpec((w, H * m)), p + nm["a1"]: TensorSpec((rank, w), free=free),
                p + nm["a2"]: TensorSpec((H * d, rank), "float32", "unit", free=free),
                p + nm["a2_bias"]: TensorSpec((H * d,), "float32", "unit"),
                p + nm["norm"]: TensorSpec((m,), "float32", "scale")}

    def load(self, weights, rt):
        a, p = self.params, self.prefix
        self.H, self.d, self.m = int(a["heads"]), int(a["dim"]), int(a["vdim"])
        nm = dict(self.NAMES, **(a.get("names") or {}))
        self.tau = float(a["tau"])
        self.eps = float(a.get("norm_eps") or 0.0)
        # one product for everything that reads the block's input: [q | k | v | g | a1]
        self.w_in = torch.cat([weights.pop(p + nm[n]) for n in ("q", "k", "v", "g", "a1")], dim=0).contiguous()
        self.cols = self.w_in.shape[0]
        self.a2t = weights.pop(p + nm["a2"]).t().contiguous()          # [rank, H dim]: channels side by side
        if self.a2t.shape[0] != self.cols - 2 * self.H * (self.d + self.m):
            raise ValueError(f"{p}: the decay's two matrices do not share their inner size")
        self.bias, self.norm_w, self.o_w = weights[p + nm["a2_bias"]], weights[p + nm["norm"]], weights[p + nm["o"]]
        self.floats = _state_floats(rt, self.H, self.d, self.m, p)

    def cache_need(self) -> CacheNeed:
        return CacheNeed("state", state_shape=(self.floats,), state_dtype=torch.float32)

    def forward(self, h, ctx, cache, rt, hold: bool = False):
        n, k = h.shape[0], rt.kernels
        hd, hv = self.H * self.d, self.H * self.m
        proj = rt.linear(h, self.w_in, None, "gla_proj")
        aux = rt.ws.get("gla_aux", n, 3 * hd + hv, torch.float32)
        k.decay_gate_prep(proj, self.cols, ctx.tok_entry, self.a2t, self.bias, 1.0 / self.tau, self.d ** -0.5, aux,
                          self.H, self.d, self.m, rt.dtype)
        o_raw = rt.ws.get("gla_o_raw", n, hv, torch.float32)
        k.matrix_state_scan(aux, (0, hd, 2 * hd, 2 * hd + hv, 0), True, False, 1, ctx, cache.state, o_raw,
                            self.H, self.d, self.m, rt.err)
        o = rt.ws.get("gla_o", n, hv, rt.dtype)
        k.head_norm_gate(o_raw, proj, self.cols, 2 * hd + hv, ctx.tok_entry, self.norm_w, self.eps, o, self.H, self.m)
        rt.launches += 3
        return rt.linear(o, self.o_w, None, "gla_out", hold=hold)


@register_part("mixer", "gated_delta")
class GatedDelta(Part):
    """params: ``hidden_size``, ``heads``, ``kv_heads`` (q/k heads), ``dim``, ``vdim``, ``conv`` (taps),
    ``norm_eps`` (of the head norm), ``key_eps`` (under the root of the unit vectors; default 1e-6),
    ``decay`` ("head", or "channel": one per head and key channel from a low-rank product), ``gate``
    ("full", or "low_rank": W_g = W_g2 W_g1), ``gate_act`` ("silu", "sigmoid"), ``decay_rank`` /
    ``gate_rank`` (the low-rank products' inner sizes; None: read from the stored tensors), ``names``.
    Tensors: q, k [G dim, hidden], v [H vdim, hidden], b [H, hidden], o [hidden, H vdim]; g [H vdim, hidden]
    or g1 [rank, hidden], g2 [H vdim, rank]; a [H, hidden] or a1 [rank, hidden], a2 [H dim, rank]; and in
    32-bit q_conv, k_conv [G dim, taps], v_conv [H vdim, taps], A_log [H], dt_bias [H] or [H dim],
    norm [vdim]."""
    kind = "mixer"
    state_graph_safe = True
    decode_bucket_safe = True
    NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "b": "b", "a": "a", "o": "o", "q_conv": "q.conv",
             "k_conv": "k.conv", "v_conv": "v.conv", "A_log": "A_log", "dt_bias": "dt_bias", "norm": "norm",
             "a1": "a1", "a2": "a2", "g1": "g1", "g2": "g2"}

    @classmethod
    def _options(cls, a, where):
        decay, gate, act = (str(a.get(k) or v) for k, v in (("decay", "head"), ("gate", "full"), ("gate_act", "silu")))
        if decay not in ("head", "channel") or gate not in ("full", "low_rank") or act not in ("silu", "sigmoid"):
            raise ValueError(f"{where}: no decay '{decay}', gate '{gate}' or gate activation '{act}'")
        return decay == "channel", gate == "low_rank", act == "sigmoid"

    @classmethod
    def manifest(cls, spec):
        a, p = spec.params, spec.prefix
        w, H, G, d, m, T = (int(a[k]) for k in ("hidden_size", "heads", "kv_heads", "dim", "vdim", "conv"))
        nm = dict(cls.NAMES, **(a.get("names") or {}))
        channel, low_gate, _ = cls._options(a, p)
        out = {p + nm["q"]: TensorSpec((G * d, w)), p + nm["k"]: TensorSpec((G * d, w)),
               p + nm["v"]: TensorSpec((H * m, w)), p + nm["b"]: TensorSpec((H, w)),
               p + nm["o"]: TensorSpec((w, H * m)),
               p + nm["q_conv"]: TensorSpec((G * d, T), "float32", "unit"),
               p + nm["k_conv"]: TensorSpec((G * d, T), "float32", "unit"),
               p + nm["v_conv"]: TensorSpec((H * m, T), "float32", "unit"),
               p + nm["A_log"]: TensorSpec((H,), "float32", "slow" if channel else "offset"),
               p + nm["dt_bias"]: TensorSpec((H * d if channel else H,), "float32", "offset"),
               p + nm["norm"]: TensorSpec((m,), "float32", "scale")}
        for wanted, one, two, rows, rank in ((channel, "a1", "a2", H * d, a.get("decay_rank")),
                                             (low_gate, "g1", "g2", H * m, a.get("gate_rank"))):
            rank, free = (-1, 16) if rank is None else (int(rank), 0)
            if wanted:
                out[p + nm[one]] = TensorSpec((rank, w), free=free)
                out[p + nm[two]] = TensorSpec((rows, rank), free=free)
        if not channel:
            out[p + nm["a"]] = TensorSpec((H, w))
        if not low_gate:
            out[p + nm["g"]] = TensorSpec((H * m, w))
        return out

    def load(self, weights, rt):
        a, p = self.params, self.prefix
        self.H, self.G, self.d, self.m, self.taps = (int(a[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        if self.H % self.G:
            raise ValueError(f"{p}: {self.H} heads are not a multiple of {self.G} query/key heads")
        nm = dict(self.NAMES, **(a.get("names") or {}))
        self.eps = float(a.get("norm_eps") or 0.0)
        self.key_eps = float(a["key_eps"]) if a.get("key_eps") is not None else 1e-6
        self.channel, low_gate, self.sigmoid_gate = self._options(a, p)
        # one product for everything that reads the block's input: [q | k | v | g | b | a], or of a low-rank
        # decay or gate the first matrix in the place of a or g
        order = ("q", "k", "v", "g1" if low_gate else "g", "b", "a1" if self.channel else "a")
        mats = [weights.pop(p + nm[n]) for n in order]
        at = [0]
        for m in mats:
            at.append(at[-1] + m.shape[0])
        self.gate_off, self.b_off, self.a_off = at[3], at[4], at[5]
        self.w_in = torch.cat(mats, dim=0).contiguous()
        self.cols = self.w_in.shape[0]
        L = rt.kernels.LowRank
        self.a2 = self.g2 = None
        for name, first, wanted in (("a2", mats[5], self.channel), ("g2", mats[3], low_gate)):
            if not wanted:
                continue
            second = weights.pop(p + nm[name])
            rank = first.shape[0]
            if second.shape[1] != rank:
                raise ValueError(f"{p}: the two matrices of {name[0]} do not share their inner size")
            packed, mma = rt.kernels.pack_low_rank(second, rt.exact)
            setattr(self, name, L(packed, rank, self.a_off if name == "a2" else self.gate_off, second.shape[0], mma=mma))
        self.conv_w = torch.cat([weights.pop(p + nm[n]) for n in ("q_conv", "k_conv", "v_conv")], dim=0).contiguous()
        self.a_log, self.dt_bias = weights[p + nm["A_log"]], weights[p + nm["dt_bias"]]
        self.norm_w, self.o_w = weights[p + nm["norm"]], weights[p + nm["o"]]
        self.channels = C = 2 * self.G * self.d + self.H * self.m
        # rows of the recurrence's inputs: [q | k | v | w | beta], or with a decay per channel [q | k | v | beta | w]
        # with the decays on a multiple of 16 bytes
        if self.channel:
            self.beta_at, self.w_at = C, -(-(C + self.H) // 4) * 4
            self.aux_cols = -(-(self.w_at + self.H * self.d) // 4) * 4
        else:
            self.w_at, self.beta_at, self.aux_cols = C, C + self.H, C + 2 * self.H
        self.conv_off = _state_floats(rt, self.H, self.d, self.m, p)
        self.floats = self.conv_off + (self.taps - 1) * self.channels

    def cache_need(self) -> CacheNeed:
        return CacheNeed("state", state_shape=(self.floats,), state_dtype=torch.float32)

    def forward(self, h, ctx, cache, rt):
        n, k = h.shape[0], rt.kernels
        gd, hv, H = self.G * self.d, self.H * self.m, self.H
        proj = rt.linear(h, self.w_in, None, "delta_proj")
        aux = rt.ws.get("gated_delta_aux", n, self.aux_cols, torch.float32)
        k.conv_delta_prep(proj, self.cols, ctx, cache.state, self.conv_off, self.conv_w, self.taps, self.a_log,
                          self.dt_bias, aux, H, self.G, self.d, self.m, self.key_eps, self.d ** -0.5, rt.err, rt.dtype,
                          b_off=self.b_off, a_off=-1 if self.channel else self.a_off, w_off=self.w_at,
                          beta_off=self.beta_at)
        second = []
        if self.a2 is not None:
            second.append(replace(self.a2, out=aux[:, self.w_at:], kind="soft_decay", bias=self.dt_bias,
                                  rate=self.a_log, per_rate=self.d))
        gate, gate_cols, gate_off = proj, self.cols, self.gate_off
        if self.g2 is not None:
            gate, gate_cols, gate_off = rt.ws.get("gated_delta_gate", n, hv, rt.dtype), hv, 0
            second.append(replace(self.g2, out=gate))
        rt.launches += low_rank_products(k, proj, self.cols, ctx.tok_entry, n, rt.dtype, second)
        o_raw = rt.ws.get("gated_delta_o_raw", n, hv, torch.float32)
        k.matrix_state_scan(aux, (0, gd, 2 * gd, self.w_at, self.beta_at), self.channel, "delta", H // self.G, ctx,
                            cache.state, o_raw, H, self.d, self.m, rt.err)
        o = rt.ws.get("gated_delta_o", n, hv, rt.dtype)
        k.head_norm_gate(o_raw, gate, gate_cols, gate_off, ctx.tok_entry, self.norm_w, self.eps, o, H, self.m,
                         sigmoid=self.sigmoid_gate)
        rt.launches += 4 if self.taps > 1 and not step_of_single_tokens(ctx) else 3
        return rt.linear(o, self.o_w, None, "delta_out")


def low_rank_products(k, low, cols, tok_entry, n, dtype, parts) -> int:
    """The second matrices of a mixer's low-rank products, in one launch where one kernel takes both.  Returns
    the launches."""
    if not parts:
        return 0
    if len(parts) == 2 and parts[0].mma == parts[1].mma:
        k.low_rank_expand(low, cols, tok_entry, n, dtype, parts[0], parts[1])
        return 1
    for p in parts:
        k.low_rank_expand(low, cols, tok_entry, n, dtype, p)
    return len(parts)


@register_part("mixer", "wkv_time_mix")
class WkvTimeMix(Part):
    """params: ``hidden_size``, ``heads``, ``dim`` (of keys and values), ``norm_eps`` (of the head norm),
    ``decay_rank`` (inner size of the decay's two products; None: read from the stored tensor), ``names``.
    Tensors: r, k, v, g [H dim, hidden], o [hidden, H dim], w1 [rank, hidden], w2 [H dim, rank], and in
    32-bit mu_r, mu_k, mu_v, mu_g, mu_w [hidden], w0, norm [H dim], u [H, dim].  The request's slot holds the
    states and, behind them, the row of the token before the next one."""
    kind = "mixer"
    state_graph_safe = True
    decode_bucket_safe = True
    MIXES = ("r", "k", "v", "g", "w")
    NAMES = {"r": "r", "k": "k", "v": "v", "g": "g", "o": "o", "w1": "w1", "w2": "w2", "w0": "w0", "u": "u",
             "norm": "norm", "mu_r": "mu.r", "mu_k": "mu.k", "mu_v": "mu.v", "mu_g": "mu.g", "mu_w": "mu.w"}

    @classmethod
    def manifest(cls, spec):
        a, p = spec.params, spec.prefix
        w, H, d = int(a["hidden_size"]), int(a["heads"]), int(a["dim"])
        nm = dict(cls.NAMES, **(a.get("names") or {}))
        rank = a.get("decay_rank")
        rank, free = (-1, 16) if rank is None else (int(rank), 0)
        out = {p + nm[n]: TensorSpec((H * d, w)) for n in ("r", "k", "v", "g")}
        out.update({p + nm["mu_" + s]: TensorSpec((w,), "float32", "unit") for s in cls.MIXES})
        out.update({p + nm["o"]: TensorSpec((w, H * d)), p + nm["w1"]: TensorSpec((rank, w), free=free),
                    p + nm["w2"]: TensorSpec((H * d, rank), free=free),
                    p + nm["w0"]: TensorSpec((H * d,), "float32", "slow"),
                    p + nm["u"]: TensorSpec((H, d), "float32", "unit"),
                    p + nm["norm"]: TensorSpec((H * d,), "float32", "scale")})
        return out

    def load(self, weights, rt):
        a, p = self.params, self.prefix
        self.w, self.H, self.d = int(a["hidden_size"]), int(a["heads"]), int(a["dim"])
        nm = dict(self.NAMES, **(a.get("names") or {}))
        self.eps = float(a.get("norm_eps") or 0.0)
        # the projections, each of a mix of its own, as one grouped product: [r | k | v | g | w1]; w1 is a product
        # of its own where it is wider than the heads together (the last group can only be narrower)
        mats = [weights.pop(p + nm[n]) for n in ("r", "k", "v", "g", "w1")]
        self.rank, hd = mats[4].shape[0], self.H * self.d
        self.w1 = mats.pop() if self.rank > hd else None
        self.w_in = torch.cat(mats, dim=0).contiguous()
        self.cols = self.w_in.shape[0]
        self.mu = torch.stack([weights[p + nm["mu_" + s]] for s in self.MIXES]).contiguous()
        second = weights.pop(p + nm["w2"])
        if second.shape[1] != self.rank:
            raise ValueError(f"{p}: the decay's two matrices do not share their inner size")
        packed, mma = rt.kernels.pack_low_rank(second, rt.exact)
        self.w2 = rt.kernels.LowRank(packed, self.rank, 4 * hd if self.w1 is None else 0, hd, kind="exp_decay", bias=weights[p + nm["w0"]],
                                     tanh=True, mma=mma)
        self.u, self.norm_w, self.o_w = weights[p + nm["u"]], weights[p + nm["norm"]], weights[p + nm["o"]]
        # rows of the recurrence's inputs: [r | k | v | w | b]
        self.aux_cols = -(-(4 * hd + self.H) // 4) * 4
        self.row_off = _state_floats(rt, self.H, self.d, self.d, p)
        self.floats = self.row_off + self.w

    def cache_need(self) -> CacheNeed:
        return CacheNeed("state", state_shape=(self.floats,), state_dtype=torch.float32)

    def forward(self, h, ctx, cache, rt):
        n, k, H, d = h.shape[0], rt.kernels, self.H, self.d
        hd = H * d
        mixes = len(self.MIXES)
        xs = rt.ws.get("time_mixes", mixes * n, self.w, rt.dtype, cap=mixes * rt.ws.max_rows).view(mixes, n, self.w)
        k.token_shift_mix(h, self.mu, ctx, cache.state, self.row_off, xs, rt.err)
        proj = rt.linear_grouped(xs, self.w_in, hd, "time_mix_proj")
        aux = rt.ws.get("time_mix_aux", n, self.aux_cols, torch.float32)
        w2 = replace(self.w2, out=aux[:, 3 * hd:])
        if self.w1 is None:
            k.low_rank_expand(proj, self.cols, ctx.tok_entry, n, rt.dtype, w2, bonus=k.Bonus(self.u, aux, 4 * hd, H, d, d))
        else:
            k.bonus_prep(proj, self.cols, ctx.tok_entry, self.u, aux, 4 * hd, H, d, d, rt.dtype)
            low = rt.linear(xs[4], self.w1, None, "time_mix_low", hold=True)
            k.low_rank_expand(low, self.rank, ctx.tok_entry, n, rt.dtype, w2)
            rt.launches += 1
        o_raw = rt.ws.get("time_mix_o_raw", n, hd, torch.float32)
        k.matrix_state_scan(aux, (0, hd, 2 * hd, 3 * hd, 4 * hd), True, "bonus", 1, ctx, cache.state, o_raw, H, d, d,
                            rt.err)
        o = rt.ws.get("time_mix_o", n, hd, rt.dtype)
        k.head_norm_gate(o_raw, proj, self.cols, 3 * hd, ctx.tok_entry, self.norm_w, self.eps, o, H, d)
        rt.launches += 4
        return rt.linear(o, self.o_w, None, "time_mix_out")


@register_part("mixer", "exponential_gates")
class ExponentialGates(Part):
    """params: ``hidden_size``, ``heads``, ``dim``, ``vdim``, ``gate_cap``, ``norm_eps`` (of the head norm), ``den_eps``
    (what is added to the normaliser), ``names``.  Tensors: q, k [H dim, hidden], v, g [H vdim, hidden],
    o [hidden, H vdim], i, f [H, hidden], and in 32-bit i_bias, f_bias [H], norm [H vdim].  The read-out is normed
    per head, times ``norm``, times sigmoid(g).  The request's slot holds per head the state with the normaliser
    as one more column, and behind the states the running maxima."""
    kind = "mixer"
    state_graph_safe = True
    decode_bucket_safe = True
    CHUNK_MIN = 24               # from this many tokens on an entry walks in chunks
    NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "i": "i", "f": "f", "i_bias": "i.b", "f_bias": "f.b",
             "norm": "norm"}

    @classmethod
    def manifest(cls, spec):
        a, p = spec.params, spec.prefix
        w, H, d, m = (int(a[k]) for k in ("hidden_size", "heads", "dim", "vdim"))
        nm = dict(cls.NAMES, **(a.get("names") or {}))
        out = {p + nm["q"]: TensorSpec((H * d, w)), p + nm["k"]: TensorSpec((H * d, w)),
               p + nm["v"]: TensorSpec((H * m, w)), p + nm["g"]: TensorSpec((H * m, w)),
               p + nm["o"]: TensorSpec((w, H * m)), p + nm["norm"]: TensorSpec((H * m,), "float32", "scale")}
        for gate in ("i", "f"):
            out[p + nm[gate]] = TensorSpec((H, w))
            out[p + nm[gate + "_bias"]] = TensorSpec((H,), "float32", "unit")
        return out

    def load(self, weights, rt):
        a, p = self.params, self.prefix
        self.H, self.d, self.m = (int(a[k]) for k in ("heads", "dim", "vdim"))
        nm = dict(self.NAMES, **(a.get("names") or {}))
        self.cap, self.eps, self.den_eps = float(a["gate_cap"]), float(a["norm_eps"]), float(a["den_eps"])
        # one product for everything that reads the block's input: [q | k | v | g | i | f]
        self.w_in = torch.cat([weights.pop(p + nm[n]) for n in ("q", "k", "v", "g", "i", "f")], dim=0).contiguous()
        if self.w_in.shape[0] % 8:                    # rows of whole 16-byte pieces
            self.w_in = torch.cat([self.w_in, self.w_in.new_zeros(-self.w_in.shape[0] % 8, self.w_in.shape[1])])
        self.cols = self.w_in.shape[0]
        self.bias_i, self.bias_f = weights[p + nm["i_bias"]], weights[p + nm["f_bias"]]
        self.norm_w, self.o_w = weights[p + nm["norm"]], weights[p + nm["o"]]
        # rows of the recurrence's inputs: [q | k | v | kept share | new share | floor]
        self.w_at = 2 * self.H * self.d + self.H * self.m
        self.aux_cols = -(-(self.w_at + 3 * self.H) // 4) * 4
        self.max_off = _state_floats(rt, self.H, self.d, self.m + 1, p)
        self.floats = self.max_off + self.H

    def cache_need(self) -> CacheNeed:
        return CacheNeed("state", state_shape=(self.floats,), state_dtype=torch.float32)

    def forward(self, h, ctx, cache, rt, hold: bool = False):
        n, k, H, d, m = h.shape[0], rt.kernels, self.H, self.d, self.m
        hd, hv = H * d, H * m
        proj = rt.linear(h, self.w_in, None, "exp_gates_proj")
        aux = rt.ws.get("exp_gates_aux", n, self.aux_cols, torch.float32)
        gates = 2 * hd + 2 * hv
        chunked = not rt.exact and not step_of_single_tokens(ctx) and k.memory_chunks_takes(proj, self.cols, d, m)
        logs = rt.ws.get("exp_gates_logs", n, 2 * H, torch.float32) if chunked else None
        k.exp_gate_prep(proj, self.cols, ctx, cache.state, self.max_off, self.bias_i, self.bias_f, self.cap, d ** -0.5,
                        aux, H, d, m, gates, gates + H, self.w_at, rt.err, rt.dtype, logs=logs, logs_min=self.CHUNK_MIN)
        o_raw = rt.ws.get("exp_gates_o_raw", n, hv, torch.float32)
        den = rt.ws.get("exp_gates_den", n, H, torch.float32)
        if chunked:
            k.memory_chunks(proj, self.cols, (0, hd, 2 * hd), logs, ctx, cache.state, o_raw, den, H, d, m, d ** -0.5,
                            self.CHUNK_MIN, rt.err)
            rt.launches += 1
        # (one entry of a step that is padded by less than 64 rows walks in chunks whole)
        if not chunked or ctx.kv_len.shape[0] > 1 or n < self.CHUNK_MIN + 64:
            k.matrix_state_scan(aux, (0, hd, 2 * hd, self.w_at, self.w_at + H), False, "gated", 1, ctx, cache.state, o_raw,
                                H, d, m, rt.err, den=den, max_len=self.CHUNK_MIN if chunked else 0)
            rt.launches += 1
        o = rt.ws.get("exp_gates_o", n, hv, rt.dtype)
        k.head_norm_gate(o_raw, proj, self.cols, 2 * hd + hv, ctx.tok_entry, self.norm_w, self.eps, o, H, m, sigmoid=True,
                         den=den, floor=aux[:, self.w_at + 2 * H:], den_eps=self.den_eps)
        rt.launches += 2
        return rt.linear(o, self.o_w, None, "exp_gates_out", hold=hold)
