"""A plain float64 statement of the Samovik decoder, one function per mechanism.

It shares nothing with the engine: weights are a mapping name -> tensor, a configuration is the plain
dictionary of config.json, a sequence is processed whole, recurrences walk token by token, every attention
weight is a dense [T, T] matrix and every token runs its experts one by one.  Slow and obvious on purpose.

    x = embed[token]
    per layer i:  x += mixer(dyn_tanh(x)) ;  x += experts(dyn_tanh(x))  (where the layer has them)
                  x += rms(P (gelu(G x) * side[token, i])) * gain
    logits = head(dyn_tanh(x))
"""

from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional

import torch

F64 = torch.float64


def dyn_tanh(x, w: Mapping, name: str):
    """tanh(alpha x) * gain + bias: nothing is averaged."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rms(x, eps: float):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------------------- rotation
def frequencies(rot: Mapping):
    """(frequency per pair, factor on cosines and sines)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=F64), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def at(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(at(float(sc["fast"]))), 0)
    hi = min(math.ceil(at(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, rot: Mapping):
    """x [T, heads, dims]: dim i turns with dim i + dims/2."""
    half = int(rot["dims"]) // 2
    f, m = frequencies(rot)
    a = positions.to(F64)[:, None] * f[None, :]
    c, s = (m * torch.cos(a))[:, None, :], (m * torch.sin(a))[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


# ------------------------------------------------------------------------------------------ mixers
def latent_attention(h, w: Mapping, p: str, m: Mapping, eps: float, positions):
    """Causal attention whose keys and values are made from one latent per token and one rotated key part
    shared by all heads; a sigmoid gate per head."""
    T, H, dn, dr, dv, rank = h.shape[0], *(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    q = (h @ w[p + "q"].T).view(T, H, dn + dr)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :rank], eps) * w[p + "dkv.norm"]
    k = (c @ w[p + "uk"].T).view(T, H, dn)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    score = torch.einsum("ihd,jhd->hij", q[..., :dn], k)
    if dr:
        qr = rotate_halves(q[..., dn:], positions, m["rot"])
        kr = rotate_halves(down[:, None, rank:], positions, m["rot"])[:, 0]
        score = score + torch.einsum("ihd,jd->hij", qr, kr)
    score = score * float(m["scale"])
    seen = torch.ones(T, T, dtype=torch.bool).tril()
    a = torch.softmax(score.masked_fill(~seen, -math.inf), dim=-1)
    o = torch.einsum("hij,jhe->ihe", a, v) * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def lightning(h, w: Mapping, p: str, m: Mapping, eps: float, state: Optional[torch.Tensor] = None):
    """S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t with silu on q, k and v; ONE norm over all heads.
    Returns (out, last state [heads, dim, vdim])."""
    T, H, dk, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k = silu(h @ w[p + "q"].T).view(T, H, dk), silu(h @ w[p + "k"].T).view(T, H, dk)
    v = silu(h @ w[p + "v"].T).view(T, H, dv)
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=h.dtype)[:, None, None]
    S = torch.zeros(H, dk, dv, dtype=h.dtype) if state is None else state.clone()
    rows = []
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hde,hd->he", S, q[t]).reshape(-1))
    y = rms(torch.stack(rows), eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T, S


def wkv(h, w: Mapping, p: str, m: Mapping, eps: float, state: Optional[torch.Tensor] = None,
        before: Optional[torch.Tensor] = None):
    """Time mixing with a decay per key channel that the token decides; the current token counts with the
    bonus u.  Returns (out, last state [heads, dim, dim], last h)."""
    T, H, D = h.shape[0], int(m["heads"]), int(m["dim"])
    first = torch.zeros(1, h.shape[1], dtype=h.dtype) if before is None else before[None]
    prev = torch.cat([first, h[:-1]], dim=0)

    def mix(s):
        return h + (prev - h) * w[p + "mu." + s]

    r, k, v = ((mix(s) @ w[p + s].T).view(T, H, D) for s in "rkv")
    gate = silu(mix("g") @ w[p + "g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix("w") @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(T, H, D)
    u = w[p + "u"].view(H, D)
    S = torch.zeros(H, D, D, dtype=h.dtype) if state is None else state.clone()
    rows = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hde,hd->he", S + u[:, :, None] * kv, r[t]))
        S = decay[t][:, :, None] * S + kv
    o = rms(torch.stack(rows), eps).reshape(T, H * D) * w[p + "norm"] * gate
    return o @ w[p + "o"].T, S, h[-1]


# ------------------------------------------------------------------------------------- feed-forward
def clamped_expert(h, w: Mapping, p: str, limit: float):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(h, w: Mapping, p: str, top: int):
    """(expert ids [T, top], their weights): the largest biased logits, softmax over the chosen ones only."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best, ids = torch.topk(z, top, dim=-1)
    return ids, torch.softmax(best, dim=-1)


def experts(h, w: Mapping, p: str, m: Mapping):
    ids, share = choose(h, w, p, int(m["router"]["top"]))
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros(h.shape[1], dtype=h.dtype)
        for e, s in zip(ids[t].tolist(), share[t]):
            y = y + s * clamped_expert(h[t:t + 1], w, f"{p}e{e}.", float(m["expert"]["limit"]))[0]
        rows.append(y)
    out = torch.stack(rows)
    if m.get("shared"):
        out = out + clamped_expert(h, w, p + "shared.", float(m["shared"]["limit"]))
    return out


def token_side(x, tokens, w: Mapping, i: int, dim: int, eps: float):
    """What layer i's own part of the token's side row adds to the stream."""
    e = w["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[f"l{i}.side.gate"].T) * e) @ w[f"l{i}.side.proj"].T
    return rms(y, eps) * w[f"l{i}.side.norm"]


# -------------------------------------------------------------------------------------- whole model
def forward(cfg: Mapping, w: Mapping, tokens: List[int], trace: Optional[list] = None):
    """Logits [T, vocab] of one sequence; `trace` collects the stream after every layer."""
    w = {k: (v if v.dtype in (torch.int32, torch.int64) else v.to(F64)) for k, v in w.items()}
    ids = torch.tensor(list(tokens))
    positions = torch.arange(len(tokens))
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][ids]
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        h = dyn_tanh(x, w, p + "norm1")
        if l["type"] == "latent_attention":
            x = x + latent_attention(h, w, p + "mix.", m, eps, positions)
        elif l["type"] == "lightning":
            x = x + lightning(h, w, p + "mix.", m, eps)[0]
        else:
            x = x + wkv(h, w, p + "mix.", m, eps)[0]
        if l.get("mlp") is not None:
            x = x + experts(dyn_tanh(x, w, p + "norm2"), w, p + "mlp.", l["mlp"])
        if cfg.get("token_side"):
            x = x + token_side(x, ids, w, i, int(cfg["token_side"]["dim"]), eps)
        if trace is not None:
            trace.append(x.clone())
    return dyn_tanh(x, w, "final.norm") @ w["head"].T
