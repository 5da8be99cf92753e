"""Grouped-query softmax attention with unit-normed queries and keys whose layers share values.

    q, k, v = W_q x (+ b_q), W_k x (+ b_k), W_v x (+ b_v)      H query heads and G key/value heads; q, k of `key_dim`,
                                                               v of `value_dim`
    q, k = unit_rms(rotate(q)), unit_rms(rotate(k))            per head, no gain (a rotation keeps a head's norm, so
                                                               the kernel norms first)
    v = (1 - lambda) v + lambda v_first                        ("blend"; v_first: the same token's values in the layer
                                                               whose role is "keep"; the blended v is cached)
    s_ij = (q_i . k_j) * scale ;  s_ij = cap * tanh(s_ij / cap) ;  s_ij -= slope_h * (i - j)
    o_i = softmax_j(s_ij) v_j over j <= i (with `chunk`: floor(j / chunk) = floor(i / chunk)) ;  out = W_o concat_h(o)

Biases, rotation, the cap, the slopes (`distance_slopes`: 2^(-8 (h + 1) / H) for head h) and the chunks are options of
their own.  The three projections are one matrix product; biases, norms, rotation, blending and the cache write are
one kernel that reads it (its split-K partial sums where it was cut).  v_first is a float32 buffer of the step: it
belongs to the step's tokens, nothing of it outlives the step.  Scores, weights and sums are float32; the
tensor-core kernels (heads of one size of 64 or 128, in decoding also 16 and 32) carry each weight as two bfloat16
terms.  A chunked layer's pages go back when their chunk is over.
Tensors: `<name>q`, `k`, `v` (each with `.b`), `vmix` (a scalar), `o`.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..cache.manager import CacheNeeds, PagedKVSpec
from ..kernels import ops
from .attention import decode_partitions
from .base import Branch, ParamSpec, Part, build_part, register_part
from .linear import Linear


class MixedValueAttention(Part):
    out_buffer = "branch"

    def __init__(self, spec, name):
        super().__init__(spec, name)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.H, self.G = int(p["num_heads"]), int(p["num_kv_heads"])
        self.dk, self.dv = int(p["key_dim"]), int(p["value_dim"])
        self.scale = float(p["scale"])
        self.eps = float(p["norm_eps"])
        self.bias = bool(p.get("bias", False))
        self.softcap = float(p.get("softcap") or 0.0)
        self.with_slopes = bool(p.get("distance_slopes", False))
        self.chunk = int(p.get("chunk") or 0)
        self.values: Optional[str] = p.get("values")             # None, "keep" or "blend"
        self.position = build_part("position", p["position"], "")
        if self.H % self.G:
            raise ValueError(f"{self.H} query heads are no multiple of {self.G} key/value heads")
        if not (1 <= self.dk <= 256 and 1 <= self.dv <= 256):
            raise ValueError(f"head sizes {self.dk} (keys) and {self.dv} (values) must be between 1 and 256")
        if self.values not in (None, "keep", "blend"):
            raise ValueError(f"values {self.values!r} is neither 'keep', 'blend' nor None")
        if self.softcap < 0 or self.chunk < 0:
            raise ValueError(f"a cap of {self.softcap}, chunks of {self.chunk}")
        self.Cq, self.Ck, self.Cv = self.H * self.dk, self.G * self.dk, self.G * self.dv
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None
        self.proj_bias = self.slopes = None
        self.blend = 0.0

    def parameters(self) -> Dict[str, ParamSpec]:
        n = self.name
        out: Dict[str, ParamSpec] = {}
        for x, c in (("q", self.Cq), ("k", self.Ck), ("v", self.Cv)):
            out[n + x] = ParamSpec((c, self.hidden))
            if self.bias:
                out[f"{n}{x}.b"] = ParamSpec((c,), role="gain", init="around_zero")
        if self.values is not None:                               # the layer that keeps its values has one too (unused)
            out[n + "vmix"] = ParamSpec((), role="gain", init="uniform", bounds=(0.2, 0.8))
        out[n + "o"] = ParamSpec((self.hidden, self.H * self.dv))
        return out

    def bind(self, tensors: Mapping[str, torch.Tensor], dtype) -> None:
        n = self.name
        self.proj = Linear(torch.cat([tensors[n + x] for x in ("q", "k", "v")], dim=0))
        self.o = Linear(tensors[n + "o"])
        if self.bias:
            self.proj_bias = torch.cat([tensors[f"{n}{x}.b"].float() for x in ("q", "k", "v")]).contiguous()
        if self.values == "blend":
            self.blend = float(tensors[n + "vmix"])
        device = self.o.weight.device
        if self.with_slopes:
            self.slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / self.H) for h in range(self.H)], dtype=torch.float32,
                                       device=device)
        self.position.tables(device)                              # made now: no copy from the host inside a step

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds(paged=PagedKVSpec(self.G, self.dk, None, None if self.dv == self.dk else self.dv,
                                            chunk=self.chunk or None))

    def streamed_weights(self):
        return [self.proj.weight, self.o.weight]

    def partitions(self, ctx, N: int, max_len: int) -> int:
        """Into how many shares each token's visible keys are cut when every token is a block of its own: about
        four blocks an SM, at least 64 keys a share, at most 16 shares.  A function of the token count and of
        limits alone (a recorded graph stays valid); it changes the order of additions, nothing else."""
        span = min(self.chunk or max_len, max_len)
        blocks = max(1, N * self.G)
        return max(1, min(16, (4 * ctx.num_sms) // blocks, -(-span // 64)))

    def forward(self, ctx, x: torch.Tensor, cache) -> Branch:
        N = x.shape[0]
        proj = self.proj(ctx, x, "mv_proj", out="model_or_partial")
        q = ctx.buffers.take("mv_q", N, (self.Cq,), ctx.dtype)
        k_pool, v_pool = cache.pools()
        table = cache.block_table()
        inv_freq, rotary_dim = self.position.tables(x.device)
        v_first = ctx.buffers.take("mv_first_values", N, (self.Cv,), torch.float32) if self.values else None
        ops.qk_norm_rope_kvwrite(
            proj, q, k_pool, v_pool, None, None, inv_freq, rotary_dim, ctx.positions, ctx.token_rows, table, self.eps,
            self.H, self.G, self.dk, value_dim=self.dv, neighbours=self.position.neighbours, bias=self.proj_bias,
            magnitude=self.position.magnitude, unit_norm=True, values=self.values, blend=self.blend, v_first=v_first)
        attn = ctx.buffers.take("mv_attn", N, (self.H * self.dv,), ctx.dtype)
        self.attend(ctx, attn, q, k_pool, v_pool, table, cache.manager.max_len)
        return Branch(self.o(ctx, attn, self.out_buffer, out="partial"))

    def attend(self, ctx, attn, q, k_pool, v_pool, table, max_len: int) -> None:
        """The step's queries over their rows' pages; the choice of kernel."""
        N, page = q.shape[0], k_pool.shape[2]
        scores = dict(softcap=self.softcap, slopes=self.slopes, chunk=self.chunk)
        tensor_cores = ctx.dtype == torch.bfloat16 and self.dk == self.dv
        take = ctx.buffers.take_flat
        if (tensor_cores and not ctx.all_decode and ctx.status is not None
                and ops.attention_tcgen05_supports(self.H, self.G, self.dk, page)):
            # prompt portions (and decoded tokens beside them): the tensor-core tile kernel
            ops.attention_prefill_tcgen05(attn, q, k_pool, v_pool, table, ctx.seq_starts, ctx.seq_rows,
                                          ctx.seq_first_pos, self.H, self.scale, ctx.status, **scores)
        elif tensor_cores and ctx.all_decode and ops.attention_mma_supports(self.H, self.G, self.dk, page, True):
            # decoded tokens: keys cut into as many partitions as stay resident at once
            NP, part_o, part_ml = decode_partitions(ctx, self.G, ops.attention_decode_mma_blocks_per_sm(self.dk), 128), None, None
            if self.chunk:
                NP = max(1, min(NP, -(-self.chunk // 128)))
            if NP > 1:
                part_o = take("attn_part_o", N * self.H * NP * self.dv, torch.float32)
                part_ml = take("attn_part_ml", N * self.H * NP * 2, torch.float32)
            ops.attention_decode_mma(attn, q, k_pool, v_pool, table, ctx.token_rows, ctx.positions, self.H, self.scale,
                                     0, NP, part_o, part_ml, **scores)
        elif (not ctx.all_decode and N >= 4 * ctx.num_seqs
                and ops.attention_bias_tile_supports(self.H, self.G, self.dk, self.dv, ctx.dtype)):
            # prompt portions on the CUDA cores: a tile of a request's consecutive tokens shares the keys it reads
            ops.attention_bias_tile(attn, q, k_pool, v_pool, table, ctx.seq_starts, ctx.seq_rows, ctx.seq_first_pos,
                                    self.H, self.scale, **scores)
        else:
            NP, part_o, part_ml = self.partitions(ctx, N, max_len), None, None
            if NP > 1:
                part_o = take("attn_part_o", N * self.H * NP * self.dv, torch.float32)
                part_ml = take("attn_part_ml", N * self.H * NP * 2, torch.float32)
            ops.attention_bias(attn, q, k_pool, v_pool, table, ctx.token_rows, ctx.positions, self.H, self.scale,
                               num_partitions=NP, part_o=part_o, part_ml=part_ml, **scores)


register_part("mixer", "mixed_value_attention", MixedValueAttention)
