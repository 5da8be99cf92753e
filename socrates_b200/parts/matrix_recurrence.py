"""Recurrent mixers with a matrix state per head.

"decayed_linear_attention": one constant decay per head, no denominator, no rotation:
    q = silu(W_q x) ,  k = silu(W_k x) ,  v = silu(W_v x)           (heads of `key_dim` and `value_dim`)
    S_t = decay_h S_(t-1) + k_t v_t^T ,   o_t = S_t^T q_t
    out = W_o (rms(all heads' o together) * w * sigmoid(W_g x))
Tensors: `<name>q`, `k`, `v`, `g`, `norm`, `o`.

"token_shift_mixing": every projection reads its own blend of this token's input and the one before, and the
token decides the decay of every key channel:
    m_s = x + (x' - x) mu_s   for s in r, k, v, g, w                  (x' the previous token's x, zero at first)
    r = W_r m_r ,  k = W_k m_k ,  v = W_v m_v ,  gate = silu(W_g m_g)
    d_t = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))
    o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t ;  S_t = diag(d_t) S_(t-1) + k_t v_t^T
    out = W_o (rms(each head's o) * w * gate)
Tensors: `<name>mu.r` (k, v, g, w), `r`, `k`, `v`, `g`, `w1`, `w2`, `w0`, `u`, `norm`, `o`; the rank of the decay
is w1's number of rows.

The states (and the previous token's x) are float32 and live in the request's state slot, so prompts may arrive in
portions and requests decode side by side.  Activations, decays, the recurrence, the norms and the gates are
float32 in both engines.  One kernel walks a request's tokens with the state in registers (long portions as
segments side by side, joined in order); the norm and the gate are a second one.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..cache.manager import CacheNeeds, StateSpec
from ..kernels import ops
from .base import Branch, ParamSpec, Part, register_part
from .linear import Linear


class MatrixRecurrence(Part):
    """What the two share: sizes, the kernel's scratch, the norm with its gate."""
    out_buffer = "branch"
    # These mixers have been run with kernels launched strictly one after the other only (every model measured with
    # them has routed experts, which ask for that): a model without such experts keeps to it.
    serial_launches = True

    def _sizes(self, H: int, dk: int, dv: int, eps: float) -> None:
        self.H, self.dk, self.dv, self.eps = H, dk, dv, eps
        if not (H >= 1 and 1 <= dk <= 256 and dv >= 1):
            raise ValueError(f"{H} heads of {dk} (keys, at most 256) and {dv} (values) dims")
        self.Ck, self.Cv = H * dk, H * dv
        self.o: Optional[Linear] = None
        self.norm_w: Optional[torch.Tensor] = None

    def _walk(self, ctx, N: int, q, k, v, state, **kw) -> torch.Tensor:
        """float32 rows [N, Cv] of the recurrence's raw outputs."""
        raw = ctx.buffers.take("rec_raw", N, (self.Cv,), torch.float32)
        n_state, n_prod = ops.linear_recurrence_scratch(N, ctx.num_seqs, self.H, self.dk, self.dv)
        take = ctx.buffers.take_flat
        ops.linear_recurrence(raw, q, k, v, state, ctx.seq_starts, ctx.seq_rows, ctx.dtype,
                              seg_state=take("rec_segments", n_state, torch.float32) if n_state else None,
                              seg_prod=take("rec_products", n_prod, torch.float32) if n_prod else None, **kw)
        return raw

    def _finish(self, ctx, raw: torch.Tensor, gate, groups: int, act: str) -> Branch:
        y = ctx.buffers.take("rec_y", raw.shape[0], (self.Cv,), ctx.dtype)
        ops.norm_gate(y, raw, self.norm_w, gate, groups, self.eps, act)
        return Branch(self.o(ctx, y, self.out_buffer, out="partial"))


class DecayedLinearAttention(MatrixRecurrence):
    def __init__(self, spec, name):
        super().__init__(spec, name)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self._sizes(int(p["num_heads"]), int(p["key_dim"]), int(p["value_dim"]), float(p["norm_eps"]))
        self.decay = [float(x) for x in p["decay"]]
        if len(self.decay) != self.H:
            raise ValueError(f"{len(self.decay)} decays for {self.H} heads")
        self.proj: Optional[Linear] = None
        self.decay_t: Optional[torch.Tensor] = None

    def parameters(self) -> Dict[str, ParamSpec]:
        n = self.name
        return {n + "q": ParamSpec((self.Ck, self.hidden)), n + "k": ParamSpec((self.Ck, self.hidden)),
                n + "v": ParamSpec((self.Cv, self.hidden)), n + "g": ParamSpec((self.Cv, self.hidden)),
                n + "norm": ParamSpec((self.Cv,), role="gain", init="gain"), n + "o": ParamSpec((self.hidden, self.Cv))}

    def bind(self, tensors: Mapping[str, torch.Tensor], dtype) -> None:
        n = self.name
        self.proj = Linear(torch.cat([tensors[n + x] for x in ("q", "k", "v", "g")], dim=0))
        self.o = Linear(tensors[n + "o"])
        self.norm_w = tensors[n + "norm"]
        self.decay_t = torch.tensor(self.decay, dtype=torch.float32, device=self.o.weight.device)

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state={"S": StateSpec((self.H, self.dk, self.dv), torch.float32)})

    def streamed_weights(self):
        return [self.proj.weight, self.o.weight]

    def forward(self, ctx, x: torch.Tensor, cache) -> Branch:
        Ck, Cv = self.Ck, self.Cv
        proj = self.proj(ctx, x, "rec_proj", out="model_or_partial")
        raw = self._walk(ctx, x.shape[0], (proj, 0), (proj, Ck), (proj, 2 * Ck), cache.state("S"), decay=self.decay_t,
                         silu_qk=True, silu_v=True)
        return self._finish(ctx, raw, (proj, 2 * Ck + Cv), 1, "sigmoid")


register_part("mixer", "decayed_linear_attention", DecayedLinearAttention)


class TokenShiftMixing(MatrixRecurrence):
    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, spec, name):
        super().__init__(spec, name)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        D = int(p["head_dim"])
        self._sizes(int(p["num_heads"]), D, D, float(p["norm_eps"]))
        self.rank_drawn = int(p.get("decay_rank", 64))        # of random weights; a checkpoint's tensors say theirs
        self.rkvg: Optional[Linear] = None
        self.linears: Dict[str, Linear] = {}
        self.mu = self.w0 = self.u = None

    def parameters(self) -> Dict[str, ParamSpec]:
        n, C, d = self.name, self.Ck, self.hidden
        out = {f"{n}mu.{s}": ParamSpec((d,), role="gain", init="uniform") for s in self.MIXES}
        out.update({n + s: ParamSpec((C, d)) for s in ("r", "k", "v", "g")})
        out[n + "w1"] = ParamSpec((-1, d), default_shape=(self.rank_drawn, d))
        out[n + "w2"] = ParamSpec((C, -1), default_shape=(C, self.rank_drawn))
        out[n + "w0"] = ParamSpec((C,), role="gain", init="uniform", bounds=(-6.0, 0.5))
        out[n + "u"] = ParamSpec((self.H, self.dk), role="gain", init="uniform")
        out[n + "norm"] = ParamSpec((C,), role="gain", init="gain")
        out[n + "o"] = ParamSpec((d, C))
        return out

    def bind(self, tensors: Mapping[str, torch.Tensor], dtype) -> None:
        n = self.name
        self.mu = torch.stack([tensors[f"{n}mu.{s}"] for s in self.MIXES]).contiguous()
        # r, k, v and g side by side: one product for a few tokens, four (of slices of the same tensor) for many
        self.rkvg = Linear(torch.cat([tensors[n + s] for s in "rkvg"], dim=0))
        self.linears = {s: Linear(self.rkvg.weight[i * self.Ck:(i + 1) * self.Ck]) for i, s in enumerate("rkvg")}
        self.linears.update({s: Linear(tensors[n + s]) for s in ("w1", "w2")})
        if self.linears["w1"].out_features != self.linears["w2"].in_features:
            raise ValueError(f"{n}w1 has {self.linears['w1'].out_features} rows and {n}w2 "
                             f"{self.linears['w2'].in_features} columns; they are the decay's rank and must agree")
        self.o = Linear(tensors[n + "o"])
        self.w0, self.u, self.norm_w = tensors[n + "w0"], tensors[n + "u"], tensors[n + "norm"]

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(state={"S": StateSpec((self.H, self.dk, self.dv), torch.float32),
                                 "x": StateSpec((1, self.hidden), torch.float32)})

    def streamed_weights(self):
        return [self.rkvg.weight, self.linears["w1"].weight, self.linears["w2"].weight, self.o.weight]

    def forward(self, ctx, x: torch.Tensor, cache) -> Branch:
        N, d = x.shape
        last = cache.state("x")
        mixed = ctx.buffers.take_flat("rec_mixes", len(self.MIXES) * N * d, ctx.dtype).view(len(self.MIXES), N, d)
        ops.token_shift_mix(mixed, x, self.mu, last, ctx.token_rows)
        ops.short_conv_tail(last, x, None, 2, ctx.seq_starts, ctx.seq_rows)       # the portion's last x stays
        C = self.Ck
        stacked = mixed[:4].view(4 * N, d)
        if 4 * N <= 64 and ctx.gemm_splits(4 * N, self.rkvg.weight, ctx.dtype) > 1:
            # A few tokens: the product streams the weights whatever it multiplies, so all four blends go through all
            # four matrices at once and every reader takes the block that is its own.
            y = self.rkvg(ctx, stacked, "rec_rkvg", out="partial")                  # [S, 4 N, 4 C]
            (r, r0), (k, k0), (v, v0), (g, g0) = ((y[:, i * N:(i + 1) * N], i * C) for i in range(4))
        else:
            r, k, v, g = (self.linears[s](ctx, mixed[i], f"rec_{s}", out="model_or_partial") for i, s in enumerate("rkvg"))
            r0 = k0 = v0 = g0 = 0
        low = self.linears["w1"](ctx, mixed[4], "rec_w1", out="model_or_partial")
        act = ctx.buffers.take("rec_w1_act", N, (self.linears["w1"].out_features,), ctx.dtype)
        ops.bias_act(act, low, None, "tanh")
        raw_decay = self.linears["w2"](ctx, act, "rec_decay", out="float32")
        raw = self._walk(ctx, N, (r, r0), (k, k0), (v, v0), cache.state("S"), raw_decay=(raw_decay, 0), decay_base=self.w0,
                         bonus=self.u)
        return self._finish(ctx, raw, (g, g0), self.H, "silu")


register_part("mixer", "token_shift_mixing", TokenShiftMixing)
