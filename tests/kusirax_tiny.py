"""Tiny Kusirax configurations for the tests and their random weights.

The configurations differ from one another in every size and option: keys and values of equal and of different sizes,
heads of 16, 32, 64 and 128 dims (which the bfloat16 engine serves on the tensor cores, in prompts or in decoding) and
of sizes that are no multiple of 8, groups of 1 to 12 query heads; rotation of all dims, of some and of none, scaled and
not; chunks shorter than a page, longer than a tile, and no chunks; with and without a cap; values blended by all
attention layers, by some, by none, with either kind first; one expert a token and all of them, groups of one expert
among others; layers without a feed-forward; a model of recurrences only.

The routers read three code channels of the stream: every token's embedding holds plus or minus six there, no branch
writes into them and their gains are one, so that they keep their signs and one common size, and the routers are drawn
so that no choice is a close call at any size.
"""

from __future__ import annotations

import json
from pathlib import Path

import torch

CODE = 3


def _att(heads, kv_heads, dim, vdim, scale, v_mix, rot=None, base=50.0, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def _cut(heads, kv_heads, dim, vdim, scale, v_mix, size, cap):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if size:
        m["mask"] = {"size": size}
    if cap:
        m["softcap"] = cap
    return m


def _wkv(heads, dim):
    return {"heads": heads, "dim": dim}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, scale, groups=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _model(vocab, width, eps, alpha, *layers):
    return {"architecture": "Kusirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "layers": list(layers)}


TINY = {
    # every mixer and feed-forward, a recurrence first; keys and values of different sizes; a chunk of 20
    "A": (_model(97, 40, 1e-6, 1.5,
                 _layer("wkv", _wkv(3, 8), _dense(56)),
                 _layer("attention", _att(4, 2, 24, 16, 0.3, True, 12, 50.0, (4.0, 1.0, 3.0, 60)), _moe(24, 6, 2, 1.3, (3, 2))),
                 _layer("attention_2", _cut(6, 2, 40, 16, 0.2, True, 20, 6.0), _dense(48)),
                 _layer("attention_2", _cut(4, 2, 16, 16, 0.4, True, 20, 6.0), None),
                 _layer("attention", _att(2, 1, 8, 32, 0.7, True, 8), _moe(24, 6, 3, 0.7, (2, 1)))), 10),
    # attention with chunks keeps the values and plain attention blends them; heads of 64; one expert a token
    "B": (_model(67, 64, 1e-5, 2.5,
                 _layer("attention_2", _cut(4, 1, 64, 64, 0.12, True, 48, 5.0), _moe(16, 7, 1, 2.0)),
                 _layer("attention", _att(2, 1, 64, 64, 0.1, True, 16, 300.0), _dense(72)),
                 _layer("wkv", _wkv(1, 70), None)), 3),
    # heads of 128, one layer that does not blend between two that do; a chunk of 33; groups of one expert
    "C": (_model(300, 64, 1e-5, 1.0,
                 _layer("attention", _att(4, 2, 128, 128, 0.06, True, 128, 1000.0, (8.0, 0.5, 4.0, 128)), _moe(32, 12, 4, 1.5, (4, 2))),
                 _layer("attention_2", _cut(8, 2, 128, 128, 0.07, False, 33, 9.0), _dense(64)),
                 _layer("attention_2", _cut(4, 2, 128, 128, 0.07, True, 100, 4.0), _moe(40, 4, 2, 1.0, (4, 3))),
                 _layer("wkv", _wkv(2, 64), _dense(64))), 40),
    # a width, heads, experts and a vocabulary that are no multiple of 8; a chunk shorter than a page
    "D": (_model(53, 36, 1e-6, 3.0,
                 _layer("attention_2", _cut(3, 3, 6, 5, 1.2, True, 7, 3.0), _moe(10, 5, 2, 1.1)),
                 _layer("wkv", _wkv(3, 5), _dense(22)),
                 _layer("attention", _att(9, 3, 10, 5, 0.8, True, 6, 20.0), _moe(10, 5, 5, 0.9))), 7),
    # heads of 16 and 32 (tensor cores in decoding only), twelve query heads a key head; no cap, no chunk
    "E": (_model(80, 56, 1e-6, 0.8,
                 _layer("attention_2", _cut(12, 1, 16, 16, 0.5, False, None, None), _dense(40)),
                 _layer("attention", _att(5, 5, 32, 32, 0.2, False), _moe(24, 9, 3, 1.0, (3, 1))),
                 _layer("attention_2", _cut(6, 2, 32, 32, 0.25, True, 64, None), _moe(24, 8, 2, 1.0, (2, 2)))), 24),
    # attention and dense feed-forwards only (kernels are launched dependently); heads of 64 in a chunk and without one
    "G": (_model(70, 48, 1e-6, 1.8,
                 _layer("attention", _att(4, 2, 64, 64, 0.1, True, 64, 200.0, (3.0, 1.0, 2.0, 50)), _dense(40)),
                 _layer("attention_2", _cut(6, 2, 64, 64, 0.12, True, 37, 7.0), _dense(56)),
                 _layer("attention_2", _cut(2, 2, 16, 64, 0.4, True, 37, 7.0), None)), 1),
    # recurrences only: no cached rows, no page groups
    "F": (_model(45, 32, 1e-5, 2.0, _layer("wkv", _wkv(4, 16), _dense(40)), _layer("wkv", _wkv(2, 24), None)), 12),
}
# (Model D with seed 5: a recurrent head of 5 dims whose output nearly cancels, so that the norm behind it makes a fifth of
# the row out of a rounding of the input.)
SEEDS = {"D": 8}


def _clear_router(r, width, g):
    """A router over the code channels whose choices are clear for every pattern of signs and every common size."""
    E, top = int(r["experts"]), int(r["top"])
    count, keep = (r["groups"]["count"], r["groups"]["keep"]) if r.get("groups") else (1, 1)
    per = E // count
    signs = torch.tensor([[1.0 if (p >> c) & 1 else -1.0 for c in range(CODE)] for p in range(1 << CODE)])
    sizes = torch.linspace(0.25, 4.5, 24)
    x = (sizes[:, None, None] * signs[None]).reshape(-1, CODE)
    best, best_gap = None, -1.0
    for _ in range(4000):
        w = torch.randn(E, CODE, generator=g) * 0.45
        s = torch.sigmoid(x @ w.T)
        gap, closed = 1.0, torch.zeros(s.shape[0], E, dtype=torch.bool)
        if keep < count:
            gs = s.view(-1, count, per).topk(min(2, per), dim=-1).values.sum(-1)
            o = gs.sort(-1, descending=True)
            gap = float((o.values[:, keep - 1] - o.values[:, keep]).min())
            closed = torch.ones(s.shape[0], count).scatter(1, o.indices[:, :keep], 0.0).bool().repeat_interleave(per, dim=1)
        o = s.masked_fill(closed, -1.0).sort(-1, descending=True).values
        if top < keep * per:
            gap = min(gap, float((o[:, top - 1] - o[:, top]).min()))
        if gap > best_gap:
            best, best_gap = w, gap
        if best_gap > 0.03:
            break
    out = torch.zeros(E, width)
    out[:, :CODE] = best
    return out


def make_weights(cfg: dict, seed: int, rank: int):
    """Random tensors for a configuration, scaled so that every mechanism matters: biases and blends that count, caps
    that bite, decays spread over their range, clear routing."""
    from socrates_b200.config import config_from_dict
    from socrates_b200.engine.model import Model
    from socrates_b200.weights.random_init import random_tensors
    params = Model(config_from_dict(cfg).plan()).parameters()
    w = random_tensors(params, seed)
    g = torch.Generator().manual_seed(seed + 1)
    for name in list(w):
        t = w[name].float()
        if name == "embed":
            t = t * 50.0
            t[:, :CODE] = 6.0 * torch.sign(torch.randn(t.shape[0], CODE, generator=g))
        elif name.endswith(".w1"):
            t = 0.3 * torch.randn(rank, t.shape[1], generator=g)
        elif name.endswith(".w2"):
            t = 0.6 * torch.randn(t.shape[0], rank, generator=g)
        elif name.endswith((".mix.q.b", ".mix.k.b", ".mix.v.b")):
            t = t * 6.0
        elif params[name].role == "matrix":
            t = t * 10.0
        if name.endswith((".mix.o", ".down")):
            t = t * min(1.0, 0.25 * cfg["postln_alpha"])          # branches that do not drown the stream
            t[:CODE] = 0.0
        if name.endswith((".norm1", ".norm2")) or name in ("embed.norm", "final.norm"):
            t[:CODE] = 1.0
        # everything is stored as bfloat16, so both engines and the plain statement read equal values
        w[name] = t.to(torch.bfloat16)
    for i, l in enumerate(cfg["layers"]):
        if l.get("mlp") is not None and l["mlp"]["kind"] == "moe":
            w[f"l{i}.mlp.router"] = _clear_router(l["mlp"]["router"], cfg["width"], g).to(torch.bfloat16)
    return w


def make_folder(tmp_path, name: str, seed: int = None, cfg: dict = None, rank: int = 6):
    """(folder, config dict, weights as float64) of the tiny model `name`."""
    cfg, rank = TINY[name] if cfg is None else (cfg, rank)
    seed = SEEDS.get(name, 5) if seed is None else seed
    w = make_weights(cfg, seed, rank)
    folder = Path(tmp_path) / f"kusirax_{name}"
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_weights(folder, w)
    return folder, cfg, {k: v.double() for k, v in w.items()}


def save_weights(folder, w):
    from safetensors.torch import save_file
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, str(Path(folder) / "model.safetensors"))
