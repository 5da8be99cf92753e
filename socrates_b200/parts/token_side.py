"""A per-layer token input: after its sublayers a layer adds its own slice of a row looked up by token id.

    e = table[token][index * dim : (index + 1) * dim]
    y = W_proj (gelu(W_gate x) * e)                     x the residual stream itself, gelu in its tanh form
    x <- x + y / sqrt(mean(y^2) + eps) * w

The table holds the slices of all layers side by side and is one tensor of the model.  The stream is folded and
rounded by the kernel that norms it elsewhere; the gate's product, the activation with the lookup (one kernel)
and the projection follow; the norm rides with the pending branch and costs no pass of its own.
Tensors: the table under the name the spec gives; `<name>gate`, `proj`, `norm`.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..kernels import ops
from .base import Branch, ParamSpec, Part, ResidualStream, register_part
from .block import stream_rows
from .linear import Linear


class TokenSide(Part):
    def __init__(self, spec, name):
        super().__init__(spec, name)
        p = spec.params
        self.hidden, self.vocab = int(p["hidden_size"]), int(p["vocab_size"])
        self.dim, self.index, self.slices = int(p["dim"]), int(p["index"]), int(p["slices"])
        self.table_name, self.eps = str(p["table"]), float(p["norm_eps"])
        if self.dim < 1 or not 0 <= self.index < self.slices:
            raise ValueError(f"slice {self.index} of {self.slices} with {self.dim} values")
        self.gate: Optional[Linear] = None
        self.proj: Optional[Linear] = None
        self.table = self.gain = None

    def parameters(self) -> Dict[str, ParamSpec]:
        n = self.name
        return {self.table_name: ParamSpec((self.vocab, self.slices * self.dim)),
                n + "gate": ParamSpec((self.dim, self.hidden)), n + "proj": ParamSpec((self.hidden, self.dim)),
                n + "norm": ParamSpec((self.hidden,), role="gain", init="gain")}

    def bind(self, tensors: Mapping[str, torch.Tensor], dtype) -> None:
        n = self.name
        self.table = tensors[self.table_name]
        self.gate, self.proj = Linear(tensors[n + "gate"]), Linear(tensors[n + "proj"])
        self.gain = tensors[n + "norm"]

    def streamed_weights(self):
        return [self.gate.weight, self.proj.weight]

    def apply(self, ctx, stream: ResidualStream) -> None:
        x = stream_rows(ctx, stream)
        z = self.gate(ctx, x, "side_gate", out="model_or_partial")
        act = ctx.buffers.take("side_act", x.shape[0], (self.dim,), ctx.dtype)
        ops.gelu_lookup(act, z, self.table, self.index * self.dim, ctx.token_ids, ctx.token_feedback)
        stream.pending = Branch(self.proj(ctx, act, "branch", out="partial"), post_gain=self.gain, post_eps=self.eps)


register_part("stream_op", "token_side", TokenSide)
