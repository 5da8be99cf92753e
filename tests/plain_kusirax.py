"""A plain float64 statement of the Kusirax decoder, one function per mechanism.

It shares nothing with the engine: weights are a mapping name -> tensor, a configuration is the plain
dictionary of config.json, a sequence is processed whole, the recurrence walks token by token, every attention
weight is a dense [T, T] matrix and every token runs its experts one by one.  Slow and obvious on purpose.

    x = rms(embed[token])
    per layer:  x = rms(alpha x + mixer(x)) ;  x = rms(alpha x + ff(x))      (the second where the layer has one)
    logits = embed rms(x)
"""

from __future__ import annotations

import math
from typing import List, Mapping, Optional

import torch

F64 = torch.float64


def unit(x, eps: float):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------------------- rotation
def frequencies(rot: Mapping):
    """One frequency per pair; with scaling, by each pair's wavelength: short ones stay, long ones are divided by
    the factor, those between are blended."""
    dims, base = int(rot["dims"]), float(rot["base"])
    sc = rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_halves(x, positions, rot: Optional[Mapping]):
    """x [T, heads, dim]: of the first rot.dims dims, dim i turns with dim i + dims/2."""
    if not rot or not int(rot["dims"]):
        return x
    half = int(rot["dims"]) // 2
    a = positions.to(F64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


# ---------------------------------------------------------------------------------------- attention
def slopes(H: int):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=F64)


def visible(T: int, chunk: Optional[int]):
    """[T, T]: i sees j <= i, and with a chunk only the keys of its own chunk."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & (i // chunk == j // chunk) if chunk else seen


def attention(h, w: Mapping, p: str, m: Mapping, eps: float, positions, v_first=None, distance: bool = False):
    """Grouped heads with unit-normed q and k.  `v_first`: the values of the first mixing layer, which a later
    one blends with its own.  `distance`: biases on the projections and a slope per head on the distance.
    Returns (out, the values this layer computed)."""
    T, H, G, D, E = h.shape[0], *(int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))

    def project(name):
        y = h @ w[p + name].T
        return y + w[p + name + ".b"] if distance else y

    q, k, v = project("q").view(T, H, D), project("k").view(T, G, D), project("v").view(T, G, E)
    own = v
    q, k = (unit(rotate_halves(y, positions, m.get("rot")), eps) for y in (q, k))
    if m.get("v_mix") and v_first is not None:
        lam = w[p + "vmix"]
        v = (1.0 - lam) * v + lam * v_first.view(T, G, E)
    k, v = (y.repeat_interleave(H // G, dim=1) for y in (k, v))
    score = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    if m.get("softcap"):
        score = float(m["softcap"]) * torch.tanh(score / float(m["softcap"]))
    if distance:
        far = (positions[:, None] - positions[None, :]).to(F64)
        score = score - slopes(H)[:, None, None] * far[None]
    seen = visible(T, int(m["mask"]["size"]) if m.get("mask") else None)
    a = torch.softmax(score.masked_fill(~seen, -math.inf), dim=-1)
    return torch.einsum("hij,jhe->ihe", a, v).reshape(T, H * E) @ w[p + "o"].T, own


# ---------------------------------------------------------------------------------------- recurrence
def wkv(h, w: Mapping, p: str, m: Mapping, eps: float, state=None, before=None):
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
    o = unit(torch.stack(rows), eps).reshape(T, H * D) * w[p + "norm"] * gate
    return o @ w[p + "o"].T, S, h[-1]


# ------------------------------------------------------------------------------------- feed-forward
def dense(h, w: Mapping, p: str):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w: Mapping, p: str):
    return torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2 @ w[p + "down"].T


def choose(z, router: Mapping):
    """(expert ids, their weights) of one token's router logits z [experts]."""
    s = sigmoid(z)
    E, top = int(router["experts"]), int(router["top"])
    g = router.get("groups") or {"count": 1, "keep": 1}
    per = E // int(g["count"])
    score = [float(s[i * per:(i + 1) * per].sort(descending=True).values[:2].sum()) for i in range(int(g["count"]))]
    best = sorted(range(len(score)), key=lambda i: -score[i])[:int(g["keep"])]
    open_ = [e for e in range(E) if e // per in best]
    ids = sorted(open_, key=lambda e: -float(s[e]))[:top]
    share = s[ids]
    return ids, share / (share.sum() + 1e-20) * float(router["scale"])


def experts(h, w: Mapping, p: str, m: Mapping):
    rows = []
    for t in range(h.shape[0]):
        ids, share = choose(w[p + "router"] @ h[t], m["router"])
        y = torch.zeros(h.shape[1], dtype=h.dtype)
        for e, c in zip(ids, share):
            y = y + c * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
        rows.append(y)
    return torch.stack(rows)


# -------------------------------------------------------------------------------------- whole model
def forward(cfg: Mapping, w: Mapping, tokens: List[int], trace: Optional[list] = None):
    """Logits [T, vocab] of one sequence; `trace` collects the stream after every layer."""
    w = {k: v.to(F64) for k, v in w.items()}
    positions = torch.arange(len(tokens))
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    x = unit(w["embed"][torch.tensor(list(tokens))], eps) * w["embed.norm"]
    v_first = None
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        if l["type"] == "wkv":
            y = wkv(x, w, p + "mix.", m, eps)[0]
        else:
            y, own = attention(x, w, p + "mix.", m, eps, positions, v_first, distance=l["type"] == "attention_2")
            if m.get("v_mix") and v_first is None:
                v_first = own
        x = unit(alpha * x + y, eps) * w[p + "norm1"]
        if l.get("mlp") is not None:
            y = dense(x, w, p + "mlp.") if l["mlp"]["kind"] == "dense" else experts(x, w, p + "mlp.", l["mlp"])
            x = unit(alpha * x + y, eps) * w[p + "norm2"]
        if trace is not None:
            trace.append(x.clone())
    return (unit(x, eps) * w["final.norm"]) @ w["embed"].T
