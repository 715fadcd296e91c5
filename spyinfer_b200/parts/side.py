"""A layer's own input for each token, let through by a gate on the residual stream.

A table ``[vocabulary, slices * dim]`` that a model's layers share holds, for every token id, a vector of ``dim`` for each of them.
With ``e`` the layer's vector of a token and ``x`` the stream: ``y = W_proj (gelu_tanh(W_gate x) * e)``; the stream takes
``rms_norm(y) * weight``, which is handed on as a record that the next norm of the stream forms in its own launch.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..weights.loader import WeightDecl
from .base import NormedDelta, Part
from .linear import Linear
from .registry import register_part


@register_part("token_input")
class TokenInput(Part):
    """params: ``hidden_size``, ``vocab_size``, ``dim``, ``slices`` (how many layers share the table), ``index`` (this layer's slice), ``table``
    (the table's full name), ``prefix``.  Tensors: ``gate [dim, hidden]``, ``proj [hidden, dim]``, ``norm [hidden]`` (a plain weight; its eps
    is that of the norm which forms the record)."""

    graph_safe = True
    kernel_modules = ("embedding",)

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.vocab, self.dim = int(params["hidden_size"]), int(params["vocab_size"]), int(params["dim"])
        self.slices, self.index, self.table_name, self.prefix = int(params["slices"]), int(params["index"]), params["table"], params.get("prefix", "")
        if min(self.hidden, self.vocab, self.dim) <= 0 or not 0 <= self.index < self.slices:
            raise ValueError(f"token_input: slice {self.index} of {self.slices}, {self.dim} wide, is not served")
        self.gate = self.proj = self.norm_w = self.table = None

    def weight_decls(self):
        p = self.prefix
        return [WeightDecl(p + "gate", (self.dim, self.hidden)), WeightDecl(p + "proj", (self.hidden, self.dim)),
                WeightDecl(p + "norm", (self.hidden,), init="one_plus_normal")]

    def shared_decls(self):
        return [WeightDecl(self.table_name, (self.vocab, self.slices * self.dim))]

    def bind(self, tensors):
        p = self.prefix
        self.gate, self.proj = Linear(tensors[p + "gate"], self.ctx.dtype), Linear(tensors[p + "proj"], self.ctx.dtype)
        self.norm_w = tensors[p + "norm"].float().contiguous()

    def bind_shared(self, tensors):
        self.table = tensors[self.table_name]

    def modules(self):
        return list(self.kernel_modules) + self.gate.modules() + self.proj.modules()

    def linears(self):
        return [self.gate, self.proj]

    def forward(self, stream, batch):
        """``stream [T, hidden]`` in the activations' type -> ``y``, possibly a stack of split-K partial products."""
        g = self.gate(stream, defer=True)
        z = torch.empty((stream.shape[0], self.dim), dtype=stream.dtype, device=stream.device)
        kernels.token_gate(g, self.table, self.index * self.dim, batch.token_ids, z, status=batch.status)
        return self.proj(z, defer=True)

    def defer(self, y):
        return NormedDelta(y, self.norm_w, 1.0)
