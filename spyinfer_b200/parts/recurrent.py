"""Mixers that carry a matrix state per request and head from token to token, in 32-bit.

``matrix_memory`` (the matrix memory of the xLSTM family, mLSTM): per head ``q, k [dk]``, ``v [dv]`` and two log gates
``i = cap * tanh((W_i h + b_i) / cap)``, ``f = logsigmoid(cap * tanh((W_f h + b_f) / cap))``; with the running maximum
``m' = max(f + m, i)`` (``m`` starts at 0): ``S = exp(f + m - m') S + exp(i - m') k v^T``, ``n`` likewise with ``k``,
``o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)``, ``q`` scaled by ``dk^(-1/2)``.

``delta_rule`` (the generalised delta rule): per head ``r, k, v [d]``, a decay per key channel
``w = exp(-exp(-1/2) * sigmoid(W_w2 tanh(W_w1 h) + w0))`` and a removal rate ``a = sigmoid(W_a h + b_a)``; with the unit key
``u = k / sqrt(sum k^2 + 1e-6)``: ``S = diag(w) S - (a * u)(u^T S) + k v^T`` (both terms read the old ``S``), ``o = S^T r``.

``gated_linear_attention`` (gated linear attention with a decay per key channel): per head ``q, k [dk]``, ``v [dv]`` and the
decay ``a = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)``: ``S = diag(a) S + k v^T``, ``o = S^T q``, ``q`` scaled by ``dk^(-1/2)``; its
gate is ``silu(W_g h)`` and its norm weight has one head's size and is shared by the heads.

``gated_delta_rule`` (the delta rule with one decay a head): q, k and v each pass a short causal convolution over time and silu, q and k
become unit vectors a head (``x / sqrt(sum x^2 + 1e-6)``, q also times ``dk^(-1/2)``) and are shared by groups of heads; with
``g = exp(-exp(A_log) softplus(W_a h + dt_bias))`` and ``beta = sigmoid(W_b h)``, one number a head: ``S = g S``, ``u = beta (v - S^T k)``,
``S = S + k u^T``, ``o = S^T q``; its gate is ``silu(W_g h)`` and its norm weight is shared by the heads.

``state_space_dual`` (the scan of Mamba-2): ``W_in h = [z | x | B | C | dt]``; x, B and C together pass a convolution with a bias and
silu; per head ``dt = softplus(dt + dt_bias)``, ``S = exp(-exp(A_log) dt) S + dt B x^T``, ``y = S^T C + D x`` with B and C shared by groups of
heads; ``y * silu(z)`` is RMS-normed in equal parts of the row (the gate comes first), then the output projection.

The others end alike: each head's ``o`` divided by its root mean square, times a weight over all heads, times
a gate of ``W_g h`` (a sigmoid unless said otherwise), then the output projection.  All projections of the input are one fused product with a 32-bit result
(what enters the recurrence is never rounded to 16 bits); the state lives in the request's slot of the cache manager.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..config.spec import CompositeCacheNeed, PartSpec, StateCacheNeed
from ..weights.loader import WeightDecl
from .base import Mixer
from .linear import Linear
from .registry import build_part, register_part

_TILE = 8     # value columns of the narrowest tile of the scan kernel, each of which keeps its own n and m (csrc/recurrence.cu)


class _Recurrent(Mixer):
    graph_safe = True
    gate = "sigmoid"       # the output gate's activation

    #: (relative tensor name, rows as a function of the sizes) of the projections that are fused, in column order
    def _fused_names(self):
        raise NotImplementedError

    def _bind_common(self, tensors, fused_names, out_name):
        p = self.prefix
        ws = [tensors[p + n] for n in fused_names]
        if len({t.dtype for t in ws}) > 1:
            ws = [t.float() for t in ws]
        self.fused = Linear(torch.cat(ws, dim=0).contiguous(), self.ctx.dtype)
        self.o = Linear(tensors[p + out_name], self.ctx.dtype)
        self.norm_weight = tensors[p + "norm"].float().contiguous()

    def _finish(self, o, proj, gate_offset, heads, dv):
        y = torch.empty(o.shape, dtype=self.ctx.dtype, device=o.device)
        kernels.gated_head_norm(o, proj, gate_offset, self.norm_weight, y, heads, dv, self.eps, gate=self.gate)
        return self.o(y, defer=self.defer_output, out_dtype=self.output_dtype)


@register_part("matrix_memory")
class MatrixMemory(_Recurrent):
    """params: ``hidden_size``, ``heads``, ``dim`` (q/k size a head), ``vdim`` (value size a head), ``gate_cap``, ``eps``
    (of the per-head norm), ``prefix``.  Tensors: ``q, k [heads dim, hidden]``, ``v, g [heads vdim, hidden]``,
    ``i, f [heads, hidden]`` with biases ``i.b, f.b [heads]``, ``norm [heads vdim]``, ``o [hidden, heads vdim]``."""

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.heads = int(params["hidden_size"]), int(params["heads"])
        self.dk, self.dv = int(params["dim"]), int(params["vdim"])
        self.cap, self.eps = float(params["gate_cap"]), float(params["eps"])
        if not self.cap > 0.0 or min(self.hidden, self.heads, self.dk, self.dv) <= 0:
            raise ValueError("matrix_memory: sizes and the gates' cap must be positive")
        self.prefix = params.get("prefix", "")
        H, dk, dv = self.heads, self.dk, self.dv
        self.offsets = (0, H * dk, 2 * H * dk, 2 * H * dk + 2 * H * dv, 2 * H * dk + 2 * H * dv + H)      # q, k, v, i, f
        self.gate_offset = 2 * H * dk + H * dv
        self.record = (dk * dv + -(-dv // _TILE) * (dk + 1) + 3) // 4 * 4
        self.fused = self.o = self.norm_weight = self.bias_i = self.bias_f = None

    def weight_decls(self):
        p, H, dk, dv, W = self.prefix, self.heads, self.dk, self.dv, self.hidden
        return [WeightDecl(p + "q", (H * dk, W)), WeightDecl(p + "k", (H * dk, W)), WeightDecl(p + "v", (H * dv, W)), WeightDecl(p + "g", (H * dv, W)),
                WeightDecl(p + "o", (W, H * dv)), WeightDecl(p + "norm", (H * dv,), init="one_plus_normal"), WeightDecl(p + "i", (H, W)),
                WeightDecl(p + "i.b", (H,)), WeightDecl(p + "f", (H, W)), WeightDecl(p + "f.b", (H,))]

    def bind(self, tensors):
        self._bind_common(tensors, ("q", "k", "v", "g", "i", "f"), "o")
        self.bias_i = tensors[self.prefix + "i.b"].float().contiguous()
        self.bias_f = tensors[self.prefix + "f.b"].float().contiguous()

    def modules(self):
        return ["recurrence", "gated_norm"] + self.fused.modules() + self.o.modules()

    def linears(self):
        return [self.fused, self.o]

    def cache_need(self):
        return StateCacheNeed((self.heads * self.record,), "float32")

    def forward(self, x, batch, cache):
        proj = self.fused(x, out_dtype=torch.float32)
        o = torch.empty((x.shape[0], self.heads * self.dv), dtype=torch.float32, device=x.device)
        kernels.mlstm_scan(proj, self.offsets, self.bias_i, self.bias_f, cache.state, batch.q_start, batch.state_slot, batch.num_seqs, o,
                           self.heads, self.dk, self.dv, self.dk ** -0.5, self.cap, status=batch.status,
                           longest=1 if batch.one_token_each else batch.num_tokens)
        return self._finish(o, proj, self.gate_offset, self.heads, self.dv)


@register_part("delta_rule")
class DeltaRule(_Recurrent):
    """params: ``hidden_size``, ``heads``, ``dim`` (key, value and receptance size a head), ``decay_rank`` (inner size of
    the decay's two-step projection), ``eps``, ``prefix``.  Tensors: ``r, k, v, g, a [heads dim, hidden]``, ``a.b``,
    ``w1 [rank, hidden]``, ``w2 [heads dim, rank]``, ``w0``, ``norm [heads dim]``, ``o [hidden, heads dim]``."""

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.heads, self.d = int(params["hidden_size"]), int(params["heads"]), int(params["dim"])
        self.rank, self.eps = int(params["decay_rank"]), float(params["eps"])
        if min(self.hidden, self.heads, self.d, self.rank) <= 0:
            raise ValueError("delta_rule: sizes must be positive")
        self.prefix = params.get("prefix", "")
        n = self.heads * self.d
        self.offsets = (0, n, 2 * n, 4 * n)       # r, k, v, a
        self.gate_offset, self.rank_offset = 3 * n, 5 * n
        self.fused = self.w2 = self.o = self.norm_weight = self.bias_a = self.decay_offset = None

    def weight_decls(self):
        p, n, W, R = self.prefix, self.heads * self.d, self.hidden, self.rank
        return ([WeightDecl(p + name, (n, W)) for name in ("k", "v", "g", "a")]
                + [WeightDecl(p + "a.b", (n,)), WeightDecl(p + "w1", (R, W)), WeightDecl(p + "w2", (n, R)), WeightDecl(p + "w0", (n,)),
                   WeightDecl(p + "norm", (n,), init="one_plus_normal"), WeightDecl(p + "o", (W, n)), WeightDecl(p + "r", (n, W))])

    def bind(self, tensors):
        self._bind_common(tensors, ("r", "k", "v", "g", "a", "w1"), "o")
        self.w2 = Linear(tensors[self.prefix + "w2"], self.ctx.dtype)
        self.bias_a = tensors[self.prefix + "a.b"].float().contiguous()
        self.decay_offset = tensors[self.prefix + "w0"].float().contiguous()

    def modules(self):
        return ["recurrence", "gated_norm"] + self.fused.modules() + self.w2.modules() + self.o.modules()

    def linears(self):
        return [self.fused, self.w2, self.o]

    def cache_need(self):
        return StateCacheNeed((self.heads * self.d * self.d,), "float32")

    def forward(self, x, batch, cache):
        proj = self.fused(x, out_dtype=torch.float32)
        inner = torch.empty((x.shape[0], self.rank), dtype=self.ctx.dtype, device=x.device)
        kernels.tanh_cols(proj, self.rank_offset, self.rank, inner)
        decay_pre = self.w2(inner, out_dtype=torch.float32)
        o = torch.empty((x.shape[0], self.heads * self.d), dtype=torch.float32, device=x.device)
        kernels.delta_scan(proj, self.offsets, decay_pre, self.bias_a, self.decay_offset, cache.state, batch.q_start, batch.state_slot,
                           batch.num_seqs, o, self.heads, self.d, status=batch.status, longest=1 if batch.one_token_each else batch.num_tokens)
        return self._finish(o, proj, self.gate_offset, self.heads, self.d)


@register_part("gated_linear_attention")
class GatedLinearAttention(_Recurrent):
    """params: ``hidden_size``, ``heads``, ``dim`` (q/k size a head), ``vdim`` (value size a head), ``tau`` (the decay's
    temperature), ``decay_rank`` (inner size of the decay's two-step projection), ``eps`` (of the per-head norm), ``prefix``.
    Tensors: ``q, k [heads dim, hidden]``, ``v, g [heads vdim, hidden]``, ``a1 [rank, hidden]``, ``a2 [heads dim, rank]``,
    ``a2.b [heads dim]``, ``norm [vdim]`` (one head's, shared), ``o [hidden, heads vdim]``."""

    gate = "silu"

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.heads = int(params["hidden_size"]), int(params["heads"])
        self.dk, self.dv, self.rank = int(params["dim"]), int(params["vdim"]), int(params["decay_rank"])
        self.tau, self.eps = float(params["tau"]), float(params["eps"])
        if not self.tau > 0.0 or min(self.hidden, self.heads, self.dk, self.dv, self.rank) <= 0:
            raise ValueError("gated_linear_attention: sizes and tau must be positive")
        self.prefix = params.get("prefix", "")
        H, dk, dv = self.heads, self.dk, self.dv
        self.offsets = (0, H * dk, 2 * H * dk)                       # q, k, v
        self.gate_offset, self.rank_offset = 2 * H * dk + H * dv, 2 * H * dk + 2 * H * dv
        self.fused = self.a2 = self.o = self.norm_weight = self.decay_bias = None

    def weight_decls(self):
        p, H, dk, dv, W, R = self.prefix, self.heads, self.dk, self.dv, self.hidden, self.rank
        return [WeightDecl(p + "q", (H * dk, W)), WeightDecl(p + "k", (H * dk, W)), WeightDecl(p + "v", (H * dv, W)), WeightDecl(p + "g", (H * dv, W)),
                WeightDecl(p + "o", (W, H * dv)), WeightDecl(p + "norm", (dv,), init="one_plus_normal"), WeightDecl(p + "a1", (R, W)),
                WeightDecl(p + "a2", (H * dk, R)), WeightDecl(p + "a2.b", (H * dk,))]

    def bind(self, tensors):
        self._bind_common(tensors, ("q", "k", "v", "g", "a1"), "o")
        self.norm_weight = self.norm_weight.repeat(self.heads).contiguous()      # one head's weight, for every head
        self.a2 = Linear(tensors[self.prefix + "a2"], self.ctx.dtype)
        self.decay_bias = tensors[self.prefix + "a2.b"].float().contiguous()

    def modules(self):
        return ["recurrence", "gated_norm"] + self.fused.modules() + self.a2.modules() + self.o.modules()

    def linears(self):
        return [self.fused, self.a2, self.o]

    def cache_need(self):
        return StateCacheNeed((self.heads * self.dk * self.dv,), "float32")

    def forward(self, x, batch, cache):
        proj = self.fused(x, out_dtype=torch.float32)
        inner = torch.empty((x.shape[0], self.rank), dtype=self.ctx.dtype, device=x.device)
        kernels.tanh_cols(proj, self.rank_offset, self.rank, inner, activation="none")
        decay_pre = self.a2(inner, out_dtype=torch.float32)
        o = torch.empty((x.shape[0], self.heads * self.dv), dtype=torch.float32, device=x.device)
        kernels.gla_scan(proj, self.offsets, decay_pre, self.decay_bias, self.tau, cache.state, batch.q_start, batch.state_slot, batch.num_seqs, o,
                         self.heads, self.dk, self.dv, self.dk ** -0.5, status=batch.status, longest=1 if batch.one_token_each else batch.num_tokens)
        return self._finish(o, proj, self.gate_offset, self.heads, self.dv)


class _ConvRecurrent(_Recurrent):
    """A recurrence behind a short convolution: what it keeps is its matrix states and the convolution's last inputs."""

    conv = None

    def cache_need(self):
        states, past = StateCacheNeed((self.heads * self.dk * self.dv,), "float32"), self.conv.cache_need()
        return CompositeCacheNeed((states, past)) if past is not None else states

    @staticmethod
    def _views(cache):
        return (cache.parts[0], cache.parts[1]) if cache.kind == "composite" else (cache, None)

    def linears(self):
        return [self.fused, self.o]

    def modules(self):
        return ["head_scan", "gated_norm"] + self.conv.modules() + self.fused.modules() + self.o.modules()


@register_part("gated_delta_rule")
class GatedDeltaRule(_ConvRecurrent):
    """params: ``hidden_size``, ``heads`` (of values and states), ``kv_heads`` (of queries and keys, a divisor), ``dim`` (q/k size a
    head), ``vdim``, ``taps`` (of the convolutions), ``eps`` (of the per-head norm), ``prefix``.  Tensors: ``q, k [kv_heads dim, hidden]``,
    ``v, g [heads vdim, hidden]``, ``q.conv, k.conv, v.conv [rows, taps]``, ``b, a [heads, hidden]``, ``A_log, dt_bias [heads]``,
    ``norm [vdim]`` (shared by the heads), ``o [hidden, heads vdim]``."""

    gate = "silu"

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.heads, self.groups = int(params["hidden_size"]), int(params["heads"]), int(params["kv_heads"])
        self.dk, self.dv, self.taps, self.eps = int(params["dim"]), int(params["vdim"]), int(params["taps"]), float(params["eps"])
        if min(self.hidden, self.heads, self.groups, self.dk, self.dv) <= 0 or self.heads % self.groups:
            raise ValueError(f"gated_delta_rule: {self.heads} heads over {self.groups} key heads of {self.dk} x {self.dv} are not served")
        self.prefix = params.get("prefix", "")
        n_k, n_v = self.groups * self.dk, self.heads * self.dv
        self.rows = (("q", n_k), ("k", n_k), ("v", n_v))
        self.offsets = (0, n_k, 2 * n_k)                              # q, k, v in the convolution's channels
        self.channels = 2 * n_k + n_v
        self.gate_offset = self.channels                              # in the fused projection: q, k, v, g, b, a
        self.rate_col, self.decay_col = self.gate_offset + n_v, self.gate_offset + n_v + self.heads
        self.conv = build_part(PartSpec("causal_conv", {"channels": self.channels, "taps": self.taps, "weight": "conv", "activation": "silu"}), ctx)
        self.fused = self.o = self.norm_weight = self.a_log = self.dt_bias = None

    def weight_decls(self):
        p, W, H = self.prefix, self.hidden, self.heads
        decls = []
        for name, rows in self.rows:
            decls += [WeightDecl(p + name, (rows, W)), WeightDecl(p + name + ".conv", (rows, self.taps))]
        return decls + [WeightDecl(p + "g", (H * self.dv, W)), WeightDecl(p + "b", (H, W)), WeightDecl(p + "a", (H, W)), WeightDecl(p + "A_log", (H,)),
                        WeightDecl(p + "dt_bias", (H,)), WeightDecl(p + "norm", (self.dv,), init="one_plus_normal"), WeightDecl(p + "o", (W, H * self.dv))]

    def bind(self, tensors):
        p = self.prefix
        self._bind_common(tensors, ("q", "k", "v", "g", "b", "a"), "o")
        self.norm_weight = self.norm_weight.repeat(self.heads).contiguous()      # one head's weight, for every head
        convs = [tensors[p + n + ".conv"] for n, _ in self.rows]
        if len({t.dtype for t in convs}) > 1:
            convs = [t.float() for t in convs]
        self.conv.bind({"conv": torch.cat(convs, dim=0)})
        self.a_log, self.dt_bias = tensors[p + "A_log"].float().contiguous(), tensors[p + "dt_bias"].float().contiguous()

    def forward(self, x, batch, cache):
        states, past = self._views(cache)
        proj = self.fused(x, out_dtype=torch.float32)
        qkv = self.conv.forward(proj, batch, past, out_dtype=torch.float32)
        o = torch.empty((x.shape[0], self.heads * self.dv), dtype=torch.float32, device=x.device)
        kernels.gated_delta_scan(qkv, self.offsets, proj, self.rate_col, self.decay_col, self.a_log, self.dt_bias, states.state, batch.q_start,
                                 batch.state_slot, batch.num_seqs, o, self.heads, self.heads // self.groups, self.dk, self.dv, self.dk ** -0.5,
                                 status=batch.status, longest=1 if batch.one_token_each else batch.num_tokens)
        return self._finish(o, proj, self.gate_offset, self.heads, self.dv)


@register_part("state_space_dual")
class StateSpaceDual(_ConvRecurrent):
    """params: ``hidden_size``, ``heads``, ``vdim`` (channels a head), ``state`` (states a channel), ``groups`` (of B and C, a divisor of
    the heads), ``taps`` (of the convolution), ``norm_groups`` (parts of the output norm), ``eps``, ``prefix``.  With ``inner = heads
    vdim``: tensors ``in [2 inner + 2 groups state + heads, hidden]`` (rows ``[z | x | B | C | dt]``), ``conv [inner + 2 groups state, taps]``,
    ``conv.b``, ``dt_bias, A_log, D [heads]``, ``norm [inner]``, ``o [hidden, inner]``."""

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.heads, self.groups = int(params["hidden_size"]), int(params["heads"]), int(params["groups"])
        self.dk, self.dv, self.taps, self.eps = int(params["state"]), int(params["vdim"]), int(params["taps"]), float(params["eps"])
        self.parts_of_norm = int(params.get("norm_groups", 1))
        self.inner = self.heads * self.dv
        if min(self.hidden, self.heads, self.groups, self.dk, self.dv, self.parts_of_norm) <= 0 or self.heads % self.groups or self.inner % self.parts_of_norm:
            raise ValueError(f"state_space_dual: {self.heads} heads of {self.dv}, {self.groups} groups of {self.dk} states, {self.parts_of_norm} norm parts are not served")
        self.prefix = p = params.get("prefix", "")
        n = self.groups * self.dk
        self.channels = self.inner + 2 * n
        self.offsets = (0, self.inner, self.inner + n)                # x, B, C in the convolution's channels
        # the fused projection's rows in another order than stored: [x | B | C | z | dt], so that the convolution's channels come first
        self.gate_offset, self.dt_col = self.channels, self.channels + self.inner
        self.conv = build_part(PartSpec("causal_conv", {"channels": self.channels, "taps": self.taps, "weight": p + "conv", "bias": p + "conv.b",
                                                        "activation": "silu"}), ctx)
        self.fused = self.o = self.norm_weight = self.dt_bias = self.a_log = self.d_skip = None

    def weight_decls(self):
        p, W, H = self.prefix, self.hidden, self.heads
        return ([WeightDecl(p + "in", (self.inner + self.channels + H, W))] + self.conv.weight_decls()
                + [WeightDecl(p + "dt_bias", (H,)), WeightDecl(p + "A_log", (H,)), WeightDecl(p + "D", (H,), init="one_plus_normal"),
                   WeightDecl(p + "norm", (self.inner,), init="one_plus_normal"), WeightDecl(p + "o", (W, self.inner))])

    def bind(self, tensors):
        p = self.prefix
        w, inner = tensors[p + "in"], self.inner
        self.fused = Linear(torch.cat([w[inner:inner + self.channels], w[:inner], w[inner + self.channels:]], dim=0).contiguous(), self.ctx.dtype)
        self.o = Linear(tensors[p + "o"], self.ctx.dtype)
        self.conv.bind({d.name: tensors[d.name] for d in self.conv.weight_decls()})
        self.norm_weight, self.dt_bias, self.a_log, self.d_skip = (tensors[p + n].float().contiguous() for n in ("norm", "dt_bias", "A_log", "D"))

    def forward(self, x, batch, cache):
        states, past = self._views(cache)
        proj = self.fused(x, out_dtype=torch.float32)
        xbc = self.conv.forward(proj, batch, past, out_dtype=torch.float32)
        o = torch.empty((x.shape[0], self.inner), dtype=torch.float32, device=x.device)
        kernels.ssd_scan(xbc, self.offsets, proj, self.dt_col, self.a_log, self.dt_bias, self.d_skip, states.state, batch.q_start, batch.state_slot,
                         batch.num_seqs, o, self.heads, self.heads // self.groups, self.dk, self.dv, status=batch.status,
                         longest=1 if batch.one_token_each else batch.num_tokens)
        y = torch.empty(o.shape, dtype=self.ctx.dtype, device=o.device)
        kernels.gate_group_norm(o, proj, self.gate_offset, self.norm_weight, y, self.parts_of_norm, self.eps)
        return self.o(y, defer=self.defer_output, out_dtype=self.output_dtype)
