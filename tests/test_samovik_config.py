"""The Samovik configuration, its plan, tensor names and cache needs; the plain statement checked on itself.
Nothing here needs a GPU."""

import json
import math

import pytest
import torch

import plain_samovik as plain
from samovik_tiny import CODE, SEEDS, TINY, make_weights
from socrates_b200.config import ConfigError, SamovikConfig, config_from_dict, known_architectures
from socrates_b200.engine.model import Model

F64 = torch.float64


def test_registry_and_round_trip():
    assert "Samovik" in known_architectures()
    for name, (cfg, _) in TINY.items():
        c = config_from_dict(cfg)
        assert isinstance(c, SamovikConfig)
        assert config_from_dict(json.loads(json.dumps(c.to_dict()))) == c, name
    assert config_from_dict(TINY["C"][0]).side_dim == 0 and config_from_dict(TINY["A"][0]).side_dim == 12


def test_plan_parts():
    plan = config_from_dict(TINY["A"][0]).plan()
    assert [e.layer for e in plan.order] == [0, 1, 2, 3]
    assert [l.mixer.kind for l in plan.layers] == ["token_shift_mixing", "latent_attention", "decayed_linear_attention",
                                                   "token_shift_mixing"]
    assert all(l.arrangement == "pre_norm_after" for l in plan.layers)
    assert plan.layers[2].feed_forward is None and len(plan.layers[2].norms) == 1
    assert [l.params["after"].params["index"] for l in plan.layers] == [0, 1, 2, 3]
    assert plan.layers[0].feed_forward.params["shared"]["limit"] == 0.7
    assert plan.layers[3].feed_forward.params["shared"] is None
    pos = plan.layers[1].mixer.params["position"]
    assert pos.params["pairing"] == "halves" and pos.params["scaling"]["factor"] == 3.0
    assert plan.final_norm.kind == "dynamic_tanh"
    assert all(l.params["after"] is None for l in config_from_dict(TINY["C"][0]).plan().layers)
    assert config_from_dict(TINY["D"][0]).plan().layers[0].mixer.params["position"].kind == "none"


def test_tensor_names_and_cache_needs():
    m = Model(config_from_dict(TINY["A"][0]).plan())
    p = m.parameters()
    for n in ("embed", "head", "side.embed", "final.norm", "final.norm.b", "final.norm.alpha", "l0.norm1.alpha", "l0.norm2.b",
              "l0.mix.mu.w", "l0.mix.w0", "l0.mix.w1", "l0.mix.w2", "l0.mix.u", "l0.mix.norm", "l0.mlp.router.b", "l0.mlp.e5.up",
              "l0.mlp.shared.down", "l0.side.gate", "l1.mix.q", "l1.mix.dkv.norm", "l1.mix.g", "l2.mix.norm", "l2.side.norm"):
        assert n in p, n
    for n in ("l2.norm2", "l2.mlp.router", "l3.mlp.shared.up", "l1.mix.uq", "l1.mix.dq", "l0.mlp.e6.up", "l0.mlp.correction"):
        assert n not in p, n
    assert p["l0.norm1.alpha"].shape == () and p["side.embed"].shape == (97, 4 * 12)
    assert p["l0.mix.w1"].matches((17, 40)) and p["l0.mix.w2"].matches((24, 17)) and not p["l0.mix.w1"].matches((17, 41))
    assert p["l1.mix.q"].shape == (3 * 12, 40) and p["l1.mix.dkv"].shape == (24, 40) and p["l1.mix.g"].shape == (3, 40)
    needs = m.cache_needs()
    assert needs[0].paged is None and needs[0].state_specs()["S"].shape == (3, 8, 8)
    assert needs[0].state_specs()["x"].shape == (1, 40)
    assert needs[1].paged.num_kv_heads == 1 and needs[1].paged.head_dim == 24 and needs[1].paged.value_dim == 20
    assert needs[2].state_specs()["S"].shape == (2, 12, 20)
    assert not any(n.startswith("side") or ".side." in n for n in Model(config_from_dict(TINY["C"][0]).plan()).parameters())


def test_refusals():
    def broken(change):
        cfg = json.loads(json.dumps(TINY["A"][0]))
        change(cfg)
        return cfg
    for change in (lambda c: c["layers"][0].update(type="lstm"),
                   lambda c: c["layers"][1]["mixer"].update(rot_dim=3),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=2),
                   lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"),
                   lambda c: c["layers"][2]["mixer"].update(decay=[0.5]),
                   lambda c: c["layers"][0]["mlp"].update(kind="dense"),
                   lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
                   lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"),
                   lambda c: c["token_side"].pop("dim"),
                   lambda c: c["norm"].pop("eps")):
        with pytest.raises(ConfigError):
            config_from_dict(broken(change))


def test_plain_rotation():
    """Rotations depend on the distance only; stretched ones keep fast dims, divide slow ones and carry a factor."""
    g = torch.Generator().manual_seed(3)
    for scaling in (None, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}):
        rot = {"dims": 12, "base": 100.0, "scaling": scaling}
        q, k = torch.randn(1, 1, 12, generator=g, dtype=F64), torch.randn(1, 1, 12, generator=g, dtype=F64)
        a = (plain.rotate_halves(q, torch.tensor([7]), rot) * plain.rotate_halves(k, torch.tensor([3]), rot)).sum()
        b = (plain.rotate_halves(q, torch.tensor([104]), rot) * plain.rotate_halves(k, torch.tensor([100]), rot)).sum()
        assert abs(float(a - b)) < 1e-9
        m = plain.frequencies(rot)[1]
        assert abs(float(plain.rotate_halves(q, torch.tensor([9]), rot).norm() / q.norm()) - m) < 1e-9
    f, m = plain.frequencies({"dims": 64, "base": 10000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}})
    exact = plain.frequencies({"dims": 64, "base": 10000.0})[0]
    assert f[0] == exact[0] and abs(float(f[-1] / exact[-1]) - 0.25) < 1e-12 and abs(m - (0.1 * math.log(4.0) + 1)) < 1e-12
    assert bool(((f <= exact) & (f >= exact / 4)).all())


def test_plain_recurrences_continue_from_a_state():
    cfg, rank = TINY["A"]
    w = {k: v.double() for k, v in make_weights(cfg, 2, rank).items()}
    h = torch.randn(30, cfg["width"], generator=torch.Generator().manual_seed(4), dtype=F64)
    whole = plain.lightning(h, w, "l2.mix.", cfg["layers"][2]["mixer"], 1e-6)[0]
    first, S = plain.lightning(h[:11], w, "l2.mix.", cfg["layers"][2]["mixer"], 1e-6)
    assert torch.allclose(torch.cat([first, plain.lightning(h[11:], w, "l2.mix.", cfg["layers"][2]["mixer"], 1e-6, S)[0]]), whole, atol=1e-12)
    m = cfg["layers"][0]["mixer"]
    whole = plain.wkv(h, w, "l0.mix.", m, 1e-6)[0]
    first, S, last = plain.wkv(h[:11], w, "l0.mix.", m, 1e-6)
    assert torch.allclose(torch.cat([first, plain.wkv(h[11:], w, "l0.mix.", m, 1e-6, S, last)[0]]), whole, atol=1e-12)
    lost = torch.cat([first, plain.wkv(h[11:], w, "l0.mix.", m, 1e-6, S)[0]])      # without the token before
    assert not torch.allclose(lost[11], whole[11], atol=1e-3) and torch.allclose(lost[:11], whole[:11])


def test_plain_latent_form_equals_the_form_with_keys_and_values():
    """q . (W_uk c) = (W_uk^T q) . c and W_uv sum_j p c_j = sum_j p (W_uv c_j); the gate is one factor a head."""
    cfg, rank = TINY["A"]
    w = {k: v.double() for k, v in make_weights(cfg, 2, rank).items()}
    m, p, T = cfg["layers"][1]["mixer"], "l1.mix.", 25
    h = torch.randn(T, cfg["width"], generator=torch.Generator().manual_seed(5), dtype=F64)
    pos = torch.arange(T)
    a = plain.latent_attention(h, w, p, m, 1e-6, pos)
    H, dn, dr, dv, r = 3, 8, 4, 12, 20
    q = (h @ w[p + "q"].T).view(T, H, dn + dr)
    down = h @ w[p + "dkv"].T
    row = torch.cat([plain.rotate_halves(down[:, None, r:], pos, m["rot"])[:, 0], plain.rms(down[:, :r], 1e-6) * w[p + "dkv.norm"]], -1)
    ql = torch.cat([plain.rotate_halves(q[..., dn:], pos, m["rot"]), torch.einsum("ihd,hdr->ihr", q[..., :dn], w[p + "uk"].view(H, dn, r))], -1)
    s = torch.einsum("ihd,jd->hij", ql, row) * m["scale"]
    s = s.masked_fill(~torch.ones(T, T, dtype=torch.bool).tril(), -math.inf)
    o = torch.einsum("hij,jr->ihr", torch.softmax(s, -1), row[:, dr:]) * plain.sigmoid(h @ w[p + "g"].T)[..., None]
    b = torch.einsum("ihr,her->ihe", o, w[p + "uv"].view(H, dv, r)).reshape(T, -1) @ w[p + "o"].T
    assert torch.allclose(a, b, atol=1e-10)


def test_plain_experts_and_clear_routing():
    """Weights of the chosen experts sum to one; every tiny model's choices stay clear of a tie in its own sequences."""
    g = torch.Generator().manual_seed(9)
    for name, (cfg, rank) in TINY.items():
        w = {k: v.double() for k, v in make_weights(cfg, SEEDS.get(name, 5), rank).items()}
        ids = torch.randint(0, cfg["vocab"], (60,), generator=g)
        gaps, seen = [], set()
        original = plain.choose

        def watch(h, ww, p, top):
            z = h @ ww[p + "router"].T + ww[p + "router.b"]
            s = z.sort(-1, descending=True).values
            gaps.append(float((s[:, top - 1] - s[:, top]).min()) if top < z.shape[1] else 1.0)
            chosen, share = original(h, ww, p, top)
            assert torch.allclose(share.sum(-1), torch.ones(h.shape[0], dtype=F64))
            seen.update((p, int(e)) for e in chosen.flatten())
            return chosen, share
        plain.choose = watch
        try:
            plain.forward(cfg, w, ids.tolist())
        finally:
            plain.choose = original
        assert min(gaps, default=1.0) > 0.03, (name, gaps)
        if not gaps:
            continue                                     # no routers in this one
        routed = [l["mlp"]["router"] for l in cfg["layers"] if l["mlp"]]
        assert len(seen) > sum(min(r["experts"], r["top"] + 1) for r in routed) - len(routed), name    # choices vary
    assert CODE == 6
