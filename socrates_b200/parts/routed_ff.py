"""Mixture of experts: every token runs through a few of many small gated feed-forwards.

    z = W_router x (float32) ,  s = softmax(z) over ALL router outputs
    chosen: the `top` largest of s + correction, taken only inside the `keep` best of `groups` equal groups
            of neighbouring outputs (a group's score is its largest s + correction)
    out = sum over chosen e of s_e * expert_e(x) ,  expert_e(x) = W_down_e (silu(W_gate_e x) * (W_up_e x))
    the last `identity` router outputs have no weights: their "expert" returns x itself

The weights are the plain scores (without the correction, not renormalized).  The router's product
and the choice are float32 in both engines.

With `router: "table"` there is no router product at all: an integer table [vocab, top] names the experts of
every token ID (no expert twice in a row), and each of them counts 1 / top.

With `weighting: "chosen"` the experts are chosen by the logits themselves (plus `router.b` with `router_bias`)
and weighed by the softmax over the chosen logits only.

With `weighting: "sigmoid"` scores are s = sigmoid(z): a group counts with the sum of its two largest s, the `top`
largest s of the open groups are chosen and weigh s / (their sum + 1e-20) * `scale`.

With `unit: "relu_squared"` an expert has no gate: W_down relu(W_up x)^2.

With `clamp` (`limit`, `alpha`, `offset`) an expert is the clamped gated unit instead:
    g = min(W_gate x, limit) ,  u = clamp(W_up x, -limit, limit) ,  W_down (g * sigmoid(alpha g) * (u + offset))
and `shared` (`intermediate_size`, `limit`) names one more such expert that runs for every token with weight one:
its rows stand behind the experts' in both products.

How it runs: all experts' gate/up matrices are one matrix [E * 2F, d] (rows interleaved as in the dense
gated feed-forward, so the product's epilogue applies silu(gate) * up) and all down matrices one matrix
[d, E * F].  The routing kernel leaves a dense float32 weight per (token, expert), zero where the expert
was not chosen; the activations are scaled by it, and the ONE down product then sums the chosen experts'
outputs by itself.  The identity experts' share, x times the sum of their weights, is one more slab of
the branch's partial sums.  Nothing is read back and no shape depends on the choice, so decode steps are
recorded into graphs like any other; the price is that every expert is computed for every token, which
costs nothing while a step streams the weights anyway (decoding) and E / top times the needed products
for long prompt portions.
For clamped experts gates and values are two halves of the first product and one kernel clamps, gates and
scales all experts' units; experts without a gate have half the first product and one such kernel.
Tensors: `<name>router`, `router.b`, `correction` (or `table`), `e<i>.gate`, `e<i>.up`, `e<i>.down`, `shared.gate`,
`shared.up`, `shared.down`.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..kernels import ops
from .base import Branch, ParamSpec, Part, register_part
from .linear import Linear


class RoutedFeedForward(Part):
    # Steps of a model with this part launch their kernels strictly one after the other.  With programmatic
    # dependent launch a 2,048-token FIRST step of a process at real widths (eight experts of 2,048 x 1,024)
    # never came back in about one run in five; it always did with the attribute off, and so did the same
    # model with dense feed-forwards.  Every wait in the kernels involved is bounded, and which of them stalls
    # was not found, so the overlap between consecutive kernels is given up for these models.
    serial_launches = True

    def __init__(self, spec, name):
        super().__init__(spec, name)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.inter = int(p["intermediate_size"])             # of one expert
        self.experts = int(p["num_experts"])
        self.identity = int(p.get("num_identity", 0))
        self.top = int(p["top"])
        self.groups = int(p.get("groups", 1))
        self.keep = int(p.get("keep_groups", self.groups))
        self.correction_tensor = bool(p.get("correction", True))
        self.routing = str(p.get("router", "scores"))         # "scores": a router product; "table": by token id
        if self.routing not in ("scores", "table"):
            raise ValueError(f"router {self.routing!r} is neither 'scores' nor 'table'")
        self.vocab = int(p.get("vocab_size", 0))
        if self.routing == "table" and (self.identity or self.vocab < 1):
            raise ValueError("a routing table needs the vocabulary's size and takes no identity experts")
        self.E = self.experts + self.identity
        if self.experts < 1 or self.identity < 0:
            raise ValueError(f"{self.experts} experts and {self.identity} identity experts")
        if self.E % self.groups or not 1 <= self.keep <= self.groups:
            raise ValueError(f"{self.E} router outputs in {self.groups} groups of which {self.keep} stay")
        if not 1 <= self.top <= self.keep * (self.E // self.groups):
            raise ValueError(f"{self.top} choices among {self.keep * (self.E // self.groups)} open experts")
        self.weighting = str(p.get("weighting", "all"))       # softmax over "all" outputs or the "chosen" ones, or "sigmoid"
        if self.weighting not in ("all", "chosen", "sigmoid"):
            raise ValueError(f"weighting {self.weighting!r} is none of 'all', 'chosen' and 'sigmoid'")
        if self.weighting == "sigmoid" and (self.routing == "table" or self.correction_tensor):
            raise ValueError("weights from sigmoid scores take no table and no correction")
        self.scale = float(p.get("scale", 1.0))
        if self.scale != 1.0 and self.weighting != "sigmoid":
            raise ValueError("a scale on the weights is served with sigmoid scores only")
        self.unit = str(p.get("unit", "gated"))
        if self.unit not in ("gated", "relu_squared"):
            raise ValueError(f"an expert's unit {self.unit!r} is neither 'gated' nor 'relu_squared'")
        if self.unit != "gated" and (p.get("clamp") is not None or p.get("shared")):
            raise ValueError("experts without a gate take no clamp and no shared expert")
        if self.weighting == "chosen" and (self.routing == "table" or self.groups > 1 or self.correction_tensor):
            raise ValueError("weights from the chosen logits take no table, groups or correction")
        self.router_bias = bool(p.get("router_bias", False))
        if self.router_bias and self.weighting != "chosen":
            raise ValueError("a router bias is served with weights from the chosen logits only")
        self.clamp = p.get("clamp")
        self.shared = p.get("shared")
        self.shared_inter = int(self.shared["intermediate_size"]) if self.shared else 0
        if self.clamp is None and self.shared:
            raise ValueError("a shared expert is served beside clamped experts only")
        if self.clamp is not None and not (float(self.clamp["limit"]) > 0
                                           and (not self.shared or float(self.shared["limit"]) > 0)):
            raise ValueError("a clamp must be positive")
        self.width = self.experts * self.inter + self.shared_inter      # columns of the activations
        self.router = self.correction = self.table = self.bias = None
        self.gate_up: Optional[Linear] = None
        self.down: Optional[Linear] = None

    def parameters(self) -> Dict[str, ParamSpec]:
        n = self.name
        if self.routing == "table":
            out = {n + "table": ParamSpec((self.vocab, self.top), role="int", init="distinct", bounds=(0, self.experts))}
        else:
            out = {n + "router": ParamSpec((self.E, self.hidden), role="gain", init="normal")}
        if self.correction_tensor and self.routing == "scores":
            out[n + "correction"] = ParamSpec((self.E,), role="gain", init="normal")
        if self.router_bias:
            out[n + "router.b"] = ParamSpec((self.E,), role="gain", init="normal")
        if self.shared_inter:
            out[n + "shared.gate"] = ParamSpec((self.shared_inter, self.hidden))
            out[n + "shared.up"] = ParamSpec((self.shared_inter, self.hidden))
            out[n + "shared.down"] = ParamSpec((self.hidden, self.shared_inter))
        for e in range(self.experts):
            if self.unit == "gated":
                out[f"{n}e{e}.gate"] = ParamSpec((self.inter, self.hidden))
            out[f"{n}e{e}.up"] = ParamSpec((self.inter, self.hidden))
            out[f"{n}e{e}.down"] = ParamSpec((self.hidden, self.inter))
        return out

    def bind(self, tensors: Mapping[str, torch.Tensor], dtype) -> None:
        n, F, d = self.name, self.inter, self.hidden
        if self.routing == "table":
            self.table = tensors[n + "table"]
            lo, hi = int(self.table.min()), int(self.table.max())
            if lo < 0 or hi >= self.experts:
                raise ValueError(f"{n}table names experts {lo}..{hi}; there are {self.experts}")
        else:
            self.router = tensors[n + "router"]              # float32: the router's product is never rounded
            self.correction = tensors[n + "correction"] if self.correction_tensor else None
            self.bias = tensors[n + "router.b"] if self.router_bias else None
        if self.clamp is not None:
            names = [f"{n}e{e}." for e in range(self.experts)] + ([n + "shared."] if self.shared_inter else [])
            self.gate_up = Linear(torch.cat([tensors[x + "gate"] for x in names] + [tensors[x + "up"] for x in names], dim=0))
            self.down = Linear(torch.cat([tensors[x + "down"] for x in names], dim=1))
            return
        if self.unit != "gated":
            self.gate_up = Linear(torch.cat([tensors[f"{n}e{e}.up"] for e in range(self.experts)], dim=0))
            self.down = Linear(torch.cat([tensors[f"{n}e{e}.down"] for e in range(self.experts)], dim=1))
            return
        rows = [torch.stack([tensors[f"{n}e{e}.gate"], tensors[f"{n}e{e}.up"]], dim=1).reshape(2 * F, d)
                for e in range(self.experts)]
        self.gate_up = Linear(torch.cat(rows, dim=0))
        self.down = Linear(torch.cat([tensors[f"{n}e{e}.down"] for e in range(self.experts)], dim=1))

    def streamed_weights(self):
        return [self.gate_up.weight, self.down.weight]

    def route(self, ctx, x: torch.Tensor):
        """float32 weights [N, E] (zero where an output was not chosen), ids int32 and weights float32 [N, top]."""
        N = x.shape[0]
        take = ctx.buffers.take
        if self.routing == "table":
            weights = take("moe_weights", N, (self.E,), torch.float32)
            ops.moe_table(weights, ctx.token_ids, self.table, ctx.token_feedback)
            return weights, None, None
        weights = take("moe_weights", N, (self.E,), torch.float32)
        ids = take("moe_ids", N, (self.top,), torch.int32)
        picked = take("moe_picked", N, (self.top,), torch.float32)
        if self.weighting == "chosen":
            ops.moe_router(x, self.router, self.bias, weights, ids, picked, self.top)
            return weights, ids, picked
        if self.weighting == "sigmoid":
            ops.moe_router(x, self.router, None, weights, ids, picked, self.top, sigmoid=True, groups=self.groups,
                           keep=self.keep, scale=self.scale)
            return weights, ids, picked
        logits = take("moe_logits", N, (self.E,), torch.float32)
        ops.moe_logits(logits, x, self.router)
        ops.moe_route(logits, self.correction, weights, ids, picked, self.groups, self.keep, self.top)
        return weights, ids, picked

    def forward(self, ctx, x: torch.Tensor) -> Branch:
        N, d, width = x.shape[0], self.hidden, self.width
        weights, _, _ = self.route(ctx, x)
        if self.clamp is not None:
            gu = self.gate_up(ctx, x, "moe_gate_up", out="model_or_partial")
            act = ctx.buffers.take("moe_act", N, (width,), ctx.dtype)
            limit = float(self.clamp["limit"])
            ops.moe_glu_clamp(act, gu, weights, self.experts, self.inter, limit,
                              float(self.shared["limit"]) if self.shared else limit, float(self.clamp["alpha"]),
                              float(self.clamp["offset"]))
        elif self.unit != "gated":
            up = self.gate_up(ctx, x, "moe_gate_up", out="model_or_partial")
            act = ctx.buffers.take("moe_act", N, (width,), ctx.dtype)
            ops.moe_act(act, up, weights, self.experts, self.inter)
        elif ctx.can_fuse_silu_mul(N, self.gate_up.weight, x.dtype):
            act = self.gate_up(ctx, x, "moe_act", epilogue=1)
        else:
            gu = self.gate_up(ctx, x, "moe_gate_up")
            act = ctx.buffers.take("moe_act", N, (width,), ctx.dtype)
            ops.silu_mul(act, gu, interleaved=True)
        if self.clamp is None and self.unit == "gated":
            ops.moe_scale(act, weights, self.experts)
        S = ctx.gemm_splits(N, self.down.weight, act.dtype)
        slabs = S + (1 if self.identity else 0)
        partial = ctx.buffers.take_flat("branch", slabs * N * d, torch.float32).view(slabs, N, d)
        ctx.gemm(partial[:S], act, self.down.weight)
        if self.identity:
            ops.moe_passthrough(partial[S], x, weights, self.experts)
        return Branch(partial)


register_part("feed_forward", "routed_experts", RoutedFeedForward)
