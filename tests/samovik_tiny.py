"""Tiny Samovik configurations for the tests and their random weights.

The configurations differ from one another in every size and option: heads from 1 to 20, key rows of 5 to 130 dims
(multiples of a 16-byte piece and not), value heads smaller and larger than keys, decays of zero and one among
others, ranks of the token's decay from 3 to 40; cached latent rows of exactly 64 and 128 dims (which the bfloat16
engine's prompts read with the tile kernel), of other multiples of 8 (its own latent kernel, with one, two, four and
eight value groups a warp) and of none (the CUDA cores), rotation with and without stretching and none at all;
layers with and without a feed-forward, with and without a shared expert, one expert a token and all of them; token
inputs of several sizes and none; and one model whose sizes are no multiple of 8.

The routers read six code channels of the stream: every token's embedding holds plus or minus six there, the
layers write little into them, and the dynamic tanh makes them plus or minus one, so that no token's choice is a
close call that rounding could turn.
"""

from __future__ import annotations

import json
from pathlib import Path

import torch

CODE = 6


def _lat(heads, dim, rot_dim, vdim, kv_rank, scale, base=100.0, scaling=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return m


def _lin(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def _wkv(heads, dim):
    return {"heads": heads, "dim": dim}


def _moe(ff, limit, experts, top, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


TINY = {
    # every mixer, a recurrent layer first; stretched rotation; a layer without a feed-forward
    "A": ({"architecture": "Samovik", "vocab": 97, "width": 40, "norm": {"eps": 1e-6}, "token_side": {"dim": 12},
           "layers": [_layer("wkv", _wkv(3, 8), _moe(24, 1.2, 6, 2, (16, 0.7))),
                      _layer("latent_attention", _lat(3, 8, 4, 12, 20, 0.6, 50.0, (3.0, 40.0, 8.0, 1.0)), _moe(24, 1.2, 5, 3, (40, 1.5))),
                      _layer("lightning", _lin(2, 12, 20, [0.7, 0.97]), None),
                      _layer("wkv", _wkv(2, 12), _moe(24, 1.2, 6, 2))]}, 10),
    # one head of 70 and of 130 key dims; a latent row of exactly 64 dims; one expert a token
    "B": ({"architecture": "Samovik", "vocab": 67, "width": 48, "norm": {"eps": 1e-5}, "token_side": {"dim": 3},
           "layers": [_layer("lightning", _lin(1, 130, 9, [0.9]), _moe(16, 0.5, 7, 1)),
                      _layer("latent_attention", _lat(2, 24, 8, 40, 56, 0.4, 300.0), _moe(16, 0.5, 4, 1, (8, 2.0))),
                      _layer("wkv", _wkv(1, 70), None)]}, 3),
    # a latent row of 128 dims and heads of 64; decays of one and of zero; no shared expert; no token input
    "C": ({"architecture": "Samovik", "vocab": 300, "width": 64, "norm": {"eps": 1e-5},
           "layers": [_layer("latent_attention", _lat(4, 32, 32, 64, 96, 0.3, 1000.0, (2.0, 64.0, 16.0, 2.0)), _moe(32, 2.0, 12, 4)),
                      _layer("lightning", _lin(3, 64, 64, [0.0, 1.0, 0.5]), _moe(40, 1.0, 3, 2)),
                      _layer("wkv", _wkv(2, 64), _moe(32, 2.0, 12, 4)),
                      _layer("lightning", _lin(3, 40, 72, [0.99, 0.3, 0.8]), _moe(40, 1.0, 3, 2))]}, 40),
    # a width, heads, latents, experts and a vocabulary that are no multiple of 8; no rotation
    "D": ({"architecture": "Samovik", "vocab": 53, "width": 36, "norm": {"eps": 1e-6}, "token_side": {"dim": 5},
           "layers": [_layer("latent_attention", _lat(2, 6, 0, 5, 7, 0.8), _moe(10, 1.0, 5, 2, (6, 1.0))),
                      _layer("wkv", _wkv(3, 5), _moe(10, 1.0, 5, 2, (6, 1.0))),
                      _layer("lightning", _lin(3, 7, 11, [0.6, 0.9, 0.95]), _moe(10, 1.0, 5, 5)),
                      _layer("latent_attention", _lat(3, 5, 2, 6, 9, 0.8, 20.0), None)]}, 7),
    # twenty heads over a latent of 136 dims (more than a row tile holds of one token), all experts chosen
    "E": ({"architecture": "Samovik", "vocab": 80, "width": 56, "norm": {"eps": 1e-6}, "token_side": {"dim": 16},
           "layers": [_layer("latent_attention", _lat(20, 16, 16, 8, 136, 0.35, 5000.0), _moe(24, 3.0, 4, 4, (64, 1.0))),
                      _layer("wkv", _wkv(2, 32), _moe(24, 3.0, 9, 2, (64, 1.0))),
                      _layer("lightning", _lin(2, 32, 24, [0.85, 0.999]), _moe(24, 3.0, 9, 2, (64, 1.0)))]}, 24),
    # a latent of 264 dims (value sums of sixteen groups a warp) and one of 40
    "F": ({"architecture": "Samovik", "vocab": 61, "width": 72, "norm": {"eps": 1e-5}, "token_side": {"dim": 8},
           "layers": [_layer("latent_attention", _lat(5, 16, 24, 32, 264, 0.3, 800.0), _moe(16, 1.0, 5, 2, (24, 1.0))),
                      _layer("latent_attention", _lat(6, 16, 8, 16, 40, 0.4, 60.0, (4.0, 30.0, 4.0, 1.0)), _moe(16, 1.0, 5, 2))]}, 8),
    # no feed-forward anywhere, no cached rows
    "G": ({"architecture": "Samovik", "vocab": 45, "width": 32, "norm": {"eps": 1e-5}, "token_side": {"dim": 8},
           "layers": [_layer("wkv", _wkv(4, 16), None), _layer("lightning", _lin(2, 24, 16, [0.95, 0.8]), None)]}, 12),
}


def _clear_router(E, top, width, gain, bias, g):
    """A router over the code channels whose choices are clear for every pattern of their signs."""
    signs = torch.tensor([[1.0 if (p >> c) & 1 else -1.0 for c in range(CODE)] for p in range(1 << CODE)])
    best, best_gap = None, -1.0
    for _ in range(2000):
        r, b = torch.zeros(E, width), 0.7 * torch.randn(E, generator=g)
        r[:, :CODE] = torch.randn(E, CODE, generator=g)
        z = (signs * 0.98 * gain[:CODE] + bias[:CODE]) @ r[:, :CODE].T + b
        s = z.sort(dim=-1, descending=True).values
        gap = float((s[:, top - 1] - s[:, top]).min()) if top < E else 1.0
        if gap > best_gap:
            best, best_gap = (r, b), gap
        if best_gap > 0.15:
            break
    return best


def make_weights(cfg: dict, seed: int, rank: int):
    """Random tensors for a configuration, scaled so that every mechanism matters: projections large enough for
    attention to be peaked and for the clamps to bite, decays spread over their range, clear routing."""
    from socrates_b200.config import config_from_dict
    from socrates_b200.engine.model import Model
    from socrates_b200.weights.random_init import random_tensors
    params = Model(config_from_dict(cfg).plan()).parameters()
    w = random_tensors(params, seed)
    g = torch.Generator().manual_seed(seed + 1)
    for name in list(w):
        t = w[name].float()
        if name == "embed":
            t = t * 20.0
            t[:, :CODE] = 6.0 * torch.sign(torch.randn(t.shape[0], CODE, generator=g))
        elif name in ("head", "side.embed"):
            t = t * 20.0
        elif name.endswith(".w1"):
            t = 0.3 * torch.randn(rank, t.shape[1], generator=g)
        elif name.endswith(".w2"):
            t = 0.6 * torch.randn(t.shape[0], rank, generator=g)
        elif name.endswith(".alpha"):
            t = 0.7 + 0.5 * torch.rand((), generator=g)
        elif name.endswith((".mix.q", ".mix.k", ".mix.r", ".mix.v", ".mix.dkv", ".mix.uk")):
            t = t * 10.0
        elif params[name].role == "matrix":
            t = t * 6.0
        if name.endswith((".mix.o", ".down")) or name.endswith(".side.proj"):
            t[:CODE] *= 0.2
        if name.endswith(".side.norm"):
            t = 0.5 * t
            t[:CODE] *= 0.2
        # everything is stored as bfloat16, so both engines and the plain statement read equal values
        w[name] = t.to(torch.bfloat16)
    for i, l in enumerate(cfg["layers"]):
        if l.get("mlp") is None:
            continue
        r = l["mlp"]["router"]
        router, bias = _clear_router(r["experts"], r["top"], cfg["width"], w[f"l{i}.norm2"].float(), w[f"l{i}.norm2.b"].float(), g)
        w[f"l{i}.mlp.router"], w[f"l{i}.mlp.router.b"] = router.to(torch.bfloat16), bias.to(torch.bfloat16)
    return w


# (Model D with seed 5: a head of 5 dims whose first output nearly cancels, so that the norm behind it makes a tenth of
# the row out of a rounding of the input.)
SEEDS = {"D": 14}


def make_folder(tmp_path, name: str, seed: int = None, cfg: dict = None, rank: int = 6):
    """(folder, config dict, weights as float64) of the tiny model `name`."""
    cfg, rank = TINY[name] if cfg is None else (cfg, rank)
    seed = SEEDS.get(name, 5) if seed is None else seed
    w = make_weights(cfg, seed, rank)
    folder = Path(tmp_path) / f"samovik_{name}"
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_weights(folder, w)
    return folder, cfg, {k: v.double() for k, v in w.items()}


def save_weights(folder, w):
    from safetensors.torch import save_file
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, str(Path(folder) / "model.safetensors"))
