"""A mixture of small gated feed-forward experts, of which every token uses the few with the largest router scores.

Router: ``s = softmax(W_router h)`` over all experts, in 32-bit; the ``top`` largest scores are the chosen experts' weights
as they are (no renormalising).  An expert: ``g = min(W_gate h, limit)``, ``u = clamp(W_up h, -limit, limit)``,
``W_down (g * sigmoid(slope * g) * (u + 1))``, no biases.  An optional shared expert of the same form (sizes and limit of its
own) runs for every token, weighted by ``sigmoid(W_sg h)``, one number a token.

All experts' gate and up projections are one product, their down projections one product over the activations side by
side; the kernel between the two multiplies each expert's activation by the token's weight for it, which is exactly zero
for an expert that the token did not choose.  A token's result therefore does not depend on what else is in the batch.

A step of many tokens (``routed_from`` or more; ``SPYINFER_MOE_ROUTED_FROM`` in the environment sets the number, 0 turns the form
off; never inside a captured graph) takes the routed form instead: the (token, chosen expert) pairs are sorted by expert on the
device, the tokens' rows gathered in that order, each expert's two products run on its own run of rows (views of the same
fused weights, nothing stored twice), and every token's ``top`` results and the shared expert's are added in a fixed order in
32-bit.  On the bfloat16 path the products of all experts are one launch each (``gemm_grouped``: the runs are padded to whole tiles, a
tile finds its expert on the device, nothing is read back); with sizes that launch does not take, and in 32-bit, the experts' row
counts are read back once a layer to size a product for each.  Weights and arithmetic are the same, so the two forms differ by the
order of sums only.  The router may be absent: with a table of experts by token id a token's choice is fixed and its experts weigh the
same, so nothing is scored.  Both forms serve the options of the choice (a correction for the choice only, groups
of router outputs, identity experts, whose pairs take no rows) and both activations.
"""
from __future__ import annotations

import os

import torch

from .. import kernels
from ..weights.loader import WeightDecl
from .base import FeedForward
from .linear import Linear
from .registry import register_part


@register_part("expert_mixture")
class ExpertMixture(FeedForward):
    """params: ``hidden_size``, ``experts``, ``top``, ``ff`` (an expert's inner size), ``limit``, ``shared_ff`` (0: no shared
    expert), ``shared_limit``, ``slope`` (default 1.702), ``prefix``; ``activation`` (``clamped_swish``, the default, or ``silu``:
    ``W_down (silu(W_gate h) * W_up h)`` without clamps, ``limit`` then unused); and the options of the choice: ``identity``
    (default 0: so many further router outputs, behind the experts', stand for experts without tensors that return their
    input), ``correction`` (default false: a tensor ``correction [experts + identity]`` is added to the scores for the choice
    only), ``groups`` (None or ``(count, keep)``: the router's outputs form ``count`` equal groups of neighbours, a group counts
    by its best choice score, and only the ``keep`` best groups' outputs can be chosen), ``scoring`` (``softmax`` over all outputs, the
    default, or ``sigmoid`` of each output's logit) and ``group_score`` (``best``, the default, or ``best_two``: the sum of a group's two
    largest choice scores); or ``scoring="table"`` with ``vocab_size``: no router, the integer tensor ``table [vocab_size, top]`` gives every
    token id its experts, each with the weight ``1 / top`` (none of the other options of the choice then).  ``shared_gate`` (default
    true): the shared expert's result is weighted by the sigmoid of ``shared.sg``'s logit; false: it is added as it is.  Tensors: ``router [experts +
    identity, hidden]``, ``e<i>.{gate,up} [ff, hidden]``, ``e<i>.down [hidden, ff]``, and with a shared expert
    ``shared.{gate,up,down}`` and ``shared.sg [1, hidden]``."""

    graph_safe = True

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.experts, self.top, self.ff = int(params["hidden_size"]), int(params["experts"]), int(params["top"]), int(params["ff"])
        self.slope = float(params.get("slope", 1.702))
        self.shared_ff, self.shared_limit = int(params.get("shared_ff") or 0), float(params.get("shared_limit") or 0.0)
        self.limit = float(params.get("limit") or 0.0)
        self.activation = params.get("activation", "clamped_swish")
        self.identity, self.has_correction = int(params.get("identity") or 0), bool(params.get("correction", False))
        self.groups = tuple(int(v) for v in params["groups"]) if params.get("groups") else None
        self.outputs = self.experts + self.identity                 # the router's outputs
        self.scoring, self.group_score = params.get("scoring", "softmax"), params.get("group_score", "best")
        self.shared_gate = bool(params.get("shared_gate", True))
        self.by_table = self.scoring == "table"
        if self.by_table and (self.identity or self.has_correction or self.groups is not None or int(params.get("vocab_size") or 0) <= 0
                              or (self.shared_ff and self.shared_gate)):
            raise ValueError("expert_mixture: a table of experts needs vocab_size, takes no options of the choice and no gate on the shared expert")
        if not self.by_table and self.shared_ff and not self.shared_gate:
            raise ValueError("expert_mixture: a shared expert beside a router has a gate")
        self.vocab = int(params.get("vocab_size") or 0)
        self.takes_batch = self.by_table
        self.table = None
        if self.scoring not in ("softmax", "sigmoid", "table") or self.group_score not in ("best", "best_two"):
            raise ValueError(f"expert_mixture: scoring {self.scoring!r} (softmax, sigmoid, table), group score {self.group_score!r} (best, best_two)")
        if min(self.hidden, self.experts, self.top, self.ff) <= 0 or self.top > self.outputs or self.shared_ff < 0 or self.identity < 0:
            raise ValueError(f"expert_mixture: {self.experts} experts of {self.ff}, top {self.top}, shared {self.shared_ff} are not served")
        if self.activation not in ("clamped_swish", "silu") or (self.activation == "clamped_swish" and not self.limit > 0.0):
            raise ValueError(f"expert_mixture: activation {self.activation!r} (clamped_swish with a positive limit, or silu)")
        if self.groups is not None:
            count, keep = self.groups
            if count <= 0 or self.outputs % count or not 0 < keep <= count or keep * (self.outputs // count) < self.top:
                raise ValueError(f"expert_mixture: {count} groups of which {keep} are kept do not fit {self.outputs} router outputs and top {self.top}")
        self.plain_choice = not self.identity and not self.has_correction and self.groups is None and self.activation == "clamped_swish" and self.scoring == "softmax"
        self.correction = None
        self.prefix = params.get("prefix", "")
        self.cols = self.experts * self.ff + self.shared_ff
        self.router = self.gate_up = self.down = None
        # the products' rows: tokens * experts in the dense form; tokens * top in the routed one, and for every expert half a tile of padding
        # (one launch) or, with a product for each expert, so many that it fills the GPU
        self.grouped = ctx.dtype == torch.bfloat16 and self.ff % 8 == 0 and self.hidden % 8 == 0
        default = self._grouped_from() if self.grouped else -(-1024 * self.experts // self.top)
        try:
            self.routed_from = int(os.environ.get("SPYINFER_MOE_ROUTED_FROM", params.get("routed_from", default)))
        except ValueError:
            self.routed_from = default

    def _grouped_from(self) -> int:
        spare = 2 * self.experts - 3 * self.top                    # half the dense form's rows must be enough and some over
        return max(1024, -(-3 * 128 * self.experts // spare)) if spare > 0 else 0     # fewer tokens: the form's further launches cost what it saves

    def weight_decls(self):
        p, W = self.prefix, self.hidden
        if self.by_table:
            decls = [WeightDecl(p + "table", (self.vocab, self.top), init=f"choice:{self.experts}", integer=True)]
        else:
            decls = [WeightDecl(p + "router", (self.outputs, W))] + ([WeightDecl(p + "correction", (self.outputs,))] if self.has_correction else [])
        for e in range(self.experts):
            decls += [WeightDecl(f"{p}e{e}.gate", (self.ff, W)), WeightDecl(f"{p}e{e}.up", (self.ff, W)), WeightDecl(f"{p}e{e}.down", (W, self.ff))]
        if self.shared_ff:
            decls += [WeightDecl(p + "shared.gate", (self.shared_ff, W)), WeightDecl(p + "shared.up", (self.shared_ff, W)),
                      WeightDecl(p + "shared.down", (W, self.shared_ff))] + ([WeightDecl(p + "shared.sg", (1, W))] if self.shared_gate else [])
        return decls

    def bind(self, tensors):
        p = self.prefix
        names = [f"e{e}." for e in range(self.experts)] + (["shared."] if self.shared_ff else [])
        rows = [tensors[p + n + half] for n in names for half in ("gate", "up")]
        downs = [tensors[p + n + "down"] for n in names]
        if len({t.dtype for t in rows + downs}) > 1:
            rows, downs = [t.float() for t in rows], [t.float() for t in downs]
        self.gate_up = Linear(torch.cat(rows, dim=0).contiguous(), self.ctx.dtype)
        self.down = Linear(torch.cat(downs, dim=1).contiguous(), self.ctx.dtype)
        if self.by_table:
            self.table = tensors[p + "table"].contiguous()
            if int(self.table.min()) < 0 or int(self.table.max()) >= self.experts:
                raise ValueError(f"expert_mixture: the table {p + 'table'!r} names experts outside 0 .. {self.experts - 1}")
            return
        # the router (and the shared expert's gate behind it) in 32-bit
        routes = [tensors[p + "router"].float()] + ([tensors[p + "shared.sg"].float()] if self.shared_ff else [])
        self.router = Linear(torch.cat(routes, dim=0).contiguous(), self.ctx.dtype)
        if self.has_correction:
            self.correction = tensors[p + "correction"].float().contiguous()

    def modules(self):
        return ["moe"] + (["gemm_grouped"] if self._one_launch() else []) + (self.router.modules() if self.router is not None else []) + self.gate_up.modules() + self.down.modules()

    def linears(self):
        return ([self.router] if self.router is not None else []) + [self.gate_up, self.down]

    def _one_launch(self) -> bool:
        return self.grouped and self.gate_up is not None and self.gate_up.fast and self.down.fast

    def forward(self, x, batch=None):
        if 0 < self.routed_from <= x.shape[0] and self.top < self.outputs and not torch.cuda.is_current_stream_capturing():
            return self._routed(x, batch)
        logits = self.router(x, out_dtype=torch.float32) if not self.by_table else None
        gu = self.gate_up(x)
        y = torch.empty((x.shape[0], self.cols), dtype=self.ctx.dtype, device=x.device)
        if self.by_table:
            kernels.moe_activation_table(gu, self.table, batch.token_ids, y, self.experts, self.ff, self.limit, self.shared_ff, self.shared_limit, self.slope,
                                         activation=self.activation)
            return self.down(y, defer=self.defer_output)
        if self.plain_choice:
            kernels.moe_activation(gu, logits, y, self.experts, self.top, self.ff, self.limit, self.shared_ff, self.shared_limit, self.slope)
            return self.down(y, defer=self.defer_output)
        idw = torch.empty((x.shape[0],), dtype=torch.float32, device=x.device) if self.identity else None
        kernels.moe_activation(gu, logits, y, self.experts, self.top, self.ff, self.limit, self.shared_ff, self.shared_limit, self.slope,
                               identity=self.identity, correction=self.correction, groups=self.groups, activation=self.activation, id_weight=idw,
                               scoring=self.scoring, group_score=self.group_score)
        if not self.identity:
            return self.down(y, defer=self.defer_output)
        # the identity experts' share, weight * input, joins the experts' sum in 32-bit: in the consumer's kernel where it offers that
        # (the block arrangement said so), else here
        if self.leave_output_bias:
            self.output_rows = (x, idw)
            return self.down(y, defer=self.defer_output)
        return kernels.add_scaled_rows(self.down(y, out_dtype=torch.float32), x, idw)

    def _products_one_by_one(self, x, offsets, row_token, row_w):
        T, E, top, ff, dev = x.shape[0], self.experts, self.top, self.ff, x.device
        starts = offsets.cpu().tolist()                      # the layer's one read-back: the experts' row counts size their products
        n = starts[E]                                        # n rows are in use: a token may have chosen fewer real experts than `top`
        results = torch.empty((T * top, self.hidden), dtype=torch.float32, device=dev)
        if n:
            rows = kernels.gather_rows(x, row_token[:n], torch.empty((n, self.hidden), dtype=x.dtype, device=dev))
            gu = torch.empty((n, 2 * ff), dtype=self.ctx.dtype, device=dev)
            for e in range(E):
                a, b = starts[e], starts[e + 1]
                if b > a:
                    self.gate_up.part(rows[a:b], rows=(2 * ff * e, 2 * ff * (e + 1)), out=gu[a:b])
            y = kernels.expert_activation(gu, row_w, torch.empty((n, ff), dtype=self.ctx.dtype, device=dev), self.limit, self.slope, activation=self.activation)
            for e in range(E):
                a, b = starts[e], starts[e + 1]
                if b > a:
                    self.down.part(y[a:b], cols=(ff * e, ff * (e + 1)), out=results[a:b])
        return results

    def _routed(self, x, batch):
        T, E, top, ff, sff, dev = x.shape[0], self.experts, self.top, self.ff, self.shared_ff, x.device
        logits = self.router(x, out_dtype=torch.float32) if not self.by_table else None
        idw = shared_w = None
        grouped = self._one_launch()
        pad = kernels.grouped_tile_rows() if grouped else 1
        if self.by_table:
            offsets, slot, row_token, row_w, *tiles = kernels.moe_route_table(self.table, batch.token_ids, E, pad=pad)
        elif self.plain_choice:
            offsets, slot, row_token, row_w, shared_w, *tiles = kernels.moe_route(logits, E, top, bool(sff), pad=pad)
        else:
            offsets, slot, row_token, row_w, shared_w, idw, *tiles = kernels.moe_route_general(
                logits, E, top, self.identity, self.correction, self.groups, bool(sff), scoring=self.scoring, group_score=self.group_score, pad=pad)
        if grouped:
            rows = kernels.gather_rows(x, row_token, torch.empty((row_token.shape[0], self.hidden), dtype=x.dtype, device=dev))
            gu = kernels.gemm_grouped(rows, self.gate_up.weight, tiles[0], E, 2 * ff, row_step=2 * ff)
            y = kernels.expert_activation(gu, row_w, torch.empty((rows.shape[0], ff), dtype=self.ctx.dtype, device=dev), self.limit, self.slope,
                                          activation=self.activation)
            results = kernels.gemm_grouped(y, self.down.weight, tiles[0], E, self.hidden, col_step=ff, out_dtype=torch.float32)
        else:
            results = self._products_one_by_one(x, offsets, row_token, row_w)
        shared = None
        if sff:
            sgu = self.gate_up.part(x, rows=(2 * ff * E, 2 * ff * E + 2 * sff), out_dtype=self.ctx.dtype)
            sy = kernels.expert_activation(sgu, shared_w, torch.empty((T, sff), dtype=self.ctx.dtype, device=dev), self.shared_limit, self.slope,
                                           activation=self.activation)
            shared = self.down.part(sy, cols=(ff * E, ff * E + sff), out_dtype=torch.float32)
        out = kernels.moe_combine(results, slot, shared, torch.empty((T, self.hidden), dtype=torch.float32, device=dev))
        if idw is None:
            return out
        if self.leave_output_bias:                           # the identity experts' share is the consumer's to add
            self.output_rows = (x, idw)
            return out
        return kernels.add_scaled_rows(out, x, idw)
