"""The Kusirax configuration, its plan, tensor names and cache needs; chunked page groups; frequencies scaled by
wavelength; the plain statement checked on itself.  Nothing here needs a GPU."""

import json
import math
import random

import pytest
import torch

import plain_kusirax as plain
from kusirax_tiny import CODE, SEEDS, TINY, make_weights
from socrates_b200.cache import CacheManager, pages_for
from socrates_b200.cache.manager import CacheNeeds, PagedKVSpec
from socrates_b200.config import ConfigError, KusiraxConfig, PartSpec, config_from_dict, known_architectures
from socrates_b200.engine.model import Model
from socrates_b200.parts import build_part

F64 = torch.float64


def test_registry_and_round_trip():
    assert "Kusirax" in known_architectures()
    for name, (cfg, _) in TINY.items():
        c = config_from_dict(cfg)
        assert isinstance(c, KusiraxConfig)
        assert config_from_dict(json.loads(json.dumps(c.to_dict()))) == c, name


def test_plan_parts():
    plan = config_from_dict(TINY["A"][0]).plan()
    assert [e.layer for e in plan.order] == [0, 1, 2, 3, 4]
    assert [l.mixer.kind for l in plan.layers] == ["token_shift_mixing", *["mixed_value_attention"] * 4]
    assert all(l.arrangement == "post_norm" and l.params["residual_scale"] == 1.5 for l in plan.layers)
    assert [l.mixer.params.get("values") for l in plan.layers] == [None, "keep", "blend", "blend", "blend"]
    assert plan.layers[3].feed_forward is None and len(plan.layers[3].norms) == 1
    assert plan.layers[0].feed_forward.params["activation"] == "gelu_tanh"
    moe = plan.layers[1].feed_forward.params
    assert (moe["weighting"], moe["unit"], moe["groups"], moe["keep_groups"], moe["scale"]) == ("sigmoid", "relu_squared", 3, 2, 1.3)
    pos = plan.layers[1].mixer.params["position"].params
    assert pos["rotary_dim"] == 12 and pos["scaling"]["kind"] == "wavelength"
    cut = plan.layers[2].mixer.params
    assert cut["chunk"] == 20 and cut["softcap"] == 6.0 and cut["bias"] and cut["distance_slopes"] and cut["position"].kind == "none"
    att = plan.layers[4].mixer.params
    assert att["chunk"] is None and att["softcap"] is None and not att["bias"] and not att["distance_slopes"]
    assert plan.embedding.kind == "normed_embedding" and plan.head.params["tied_to"] == "embed"
    # the first layer that blends keeps its values, whichever its kind; one that does not blend is passed over
    kinds = lambda name: [l.mixer.params.get("values") for l in config_from_dict(TINY[name][0]).plan().layers]
    assert kinds("B") == ["keep", "blend", None] and kinds("C") == ["keep", None, "blend", None]
    assert kinds("E") == [None, None, "keep"]


def test_tensor_names_and_cache_needs():
    m = Model(config_from_dict(TINY["A"][0]).plan())
    p = m.parameters()
    for n in ("embed", "embed.norm", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.mu.w", "l0.mix.w0", "l0.mix.w1", "l0.mix.w2",
              "l0.mix.u", "l0.mix.norm", "l0.mlp.gate", "l0.mlp.up", "l0.mlp.down", "l1.mix.vmix", "l1.mlp.router", "l1.mlp.e5.up",
              "l1.mlp.e0.down", "l2.mix.q.b", "l2.mix.k.b", "l2.mix.v.b", "l2.mix.vmix", "l3.norm1"):
        assert n in p, n
    for n in ("head", "l3.norm2", "l1.mix.q.b", "l1.mlp.e0.gate", "l1.mlp.e6.up", "l1.mlp.router.b", "l0.mix.q", "l3.mlp.up"):
        assert n not in p, n
    assert p["l1.mix.vmix"].shape == () and p["l2.mix.o"].shape == (40, 6 * 16)
    assert p["l0.mix.w1"].matches((17, 40)) and p["l0.mix.w2"].matches((24, 17))
    needs = m.cache_needs()
    assert needs[0].paged is None and needs[0].state_specs()["S"].shape == (3, 8, 8)
    assert needs[1].paged == PagedKVSpec(2, 24, None, 16) and needs[2].paged == PagedKVSpec(2, 40, None, 16, chunk=20)
    assert "l0.mix.vmix" not in Model(config_from_dict(TINY["E"][0]).plan()).parameters()


def test_refusals():
    def broken(change):
        cfg = json.loads(json.dumps(TINY["A"][0]))
        change(cfg)
        return cfg
    for change in (lambda c: c["layers"][0].update(type="lstm"),
                   lambda c: c.pop("postln_alpha"),
                   lambda c: c["layers"][1]["mixer"].update(kv_heads=3),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26),
                   lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("low"),
                   lambda c: c["layers"][2]["mixer"].update(vdim=24),               # blends with values of another width
                   lambda c: c["layers"][2]["mixer"]["mask"].update(size=0),
                   lambda c: c["layers"][2]["mixer"].update(softcap=-1.0),
                   lambda c: c["layers"][1]["mlp"].update(kind="table"),
                   lambda c: c["layers"][0]["mlp"].pop("ff"),
                   lambda c: c["layers"][1]["mlp"]["router"].update(top=5),
                   lambda c: c["layers"][1]["mlp"]["router"].update(groups={"count": 4, "keep": 1}),
                   lambda c: c["norm"].pop("eps")):
        with pytest.raises(ConfigError):
            config_from_dict(broken(change))


def test_frequencies_by_wavelength():
    """The part's table against the plain one, pair by pair; every branch is taken; one ulp of float32 at most."""
    for dims, base, sc in ((64, 1e4, (8.0, 1.0, 4.0, 512.0)), (48, 5e5, (4.0, 0.5, 3.0, 4096.0)), (6, 30.0, (2.0, 1.0, 2.0, 20.0))):
        scaling = dict(zip(("factor", "low", "high", "original"), sc))
        rot = build_part("position", PartSpec("rotary", {
            "head_dim": dims, "rotary_dim": dims, "theta": base, "pairing": "halves", "table_precision": "float64",
            "scaling": {"kind": "wavelength", **scaling}}), "")
        got, want = rot.inv_freq().double(), plain.frequencies({"dims": dims, "base": base, "scaling": scaling})
        exact = plain.frequencies({"dims": dims, "base": base})
        assert bool(((got - want).abs() <= 1.2e-7 * want).all()) and rot.magnitude == 1.0
        share = want / exact
        if dims > 8:
            assert bool((share == 1.0).any()) and bool(((share - 1.0 / sc[0]).abs() < 1e-12).any())
            assert bool(((share < 0.999) & (share > 1.001 / sc[0])).any())
    with pytest.raises(ValueError):
        build_part("position", PartSpec("rotary", {"head_dim": 8, "theta": 10.0, "scaling": {
            "kind": "wavelength", "factor": 2.0, "low": 2.0, "high": 2.0, "original": 8}}), "")


# ------------------------------------------------------------------------------------------ chunked page groups
def chunked(chunk, pages, rows=3, max_len=320):
    needs = [CacheNeeds(PagedKVSpec(1, 4)), CacheNeeds(PagedKVSpec(1, 4, chunk=chunk)), None, CacheNeeds(PagedKVSpec(1, 4, chunk=chunk))]
    return CacheManager(needs, max_rows=rows, max_len=max_len, page_size=16, num_pages=pages, dtype=torch.float32, device="cpu")


def test_a_finished_chunk_gives_its_pages_back():
    m = chunked(40, 20)
    assert len(m.groups) == 2                                   # both chunked layers share one group
    full, cut = m.groups
    m.assign(0)
    assert m.reserve(0, 79)
    m.commit(0, 79)                                             # the next query (79) sees keys 40..79: blocks 2, 3, 4
    assert cut.row_pages[0][:2] == [0, 0] and len(cut.owned(0)) == 3 and len(full.owned(0)) == 5
    m.reserve(0, 80)
    m.commit(0, 80)                                             # the next query (80) begins a chunk: nothing is in sight
    assert cut.owned(0) == [] and cut.first_needed_block(80) == 5
    m.check()
    assert m.pages_needed(0, 97) == [2, 2]
    assert m.reserve(0, 97)
    m.commit(0, 97)
    assert len(cut.owned(0)) == 2 and cut.row_pages[0][5] != 0 and int(cut.host_table[0, 4]) == 0
    m.check()
    m.release(0)
    assert m.free_pages() == [20, 20]


def test_a_chunk_edge_inside_a_page_keeps_the_page():
    m = chunked(40, 20)
    m.assign(1)
    m.reserve(1, 41)
    m.commit(1, 41)                                             # chunk 1 starts at 40, in the middle of block 2 (32..47)
    assert m.groups[1].row_pages[1][:2] == [0, 0] and m.groups[1].row_pages[1][2] != 0
    m.check()


def test_chunks_beside_a_window_are_refused():
    with pytest.raises(ValueError):
        PagedKVSpec(1, 4, window=8, chunk=8)
    with pytest.raises(ValueError):
        PagedKVSpec(1, 4, chunk=0)


@pytest.mark.parametrize("seed", range(4))
def test_random_orders_lose_no_page_of_a_chunked_group(seed):
    rng = random.Random(seed)
    chunk = rng.choice([7, 16, 40, 100])
    m = chunked(chunk, rng.choice([8, 14, 30]), rows=4, max_len=160)
    live = {}
    for _ in range(300):
        op = rng.random()
        free_rows = [r for r in range(4) if not m.active[r]]
        if op < 0.25 and free_rows:
            r = rng.choice(free_rows)
            m.assign(r)
            live[r] = 0
        elif op < 0.8 and live:
            r = rng.choice(list(live))
            new_len = min(160, live[r] + rng.choice([1, 1, 2, 7, 16, 33]))
            if m.reserve(r, new_len):
                for p in range(live[r], new_len):               # every key a query of the portion sees has a page
                    for b in range((p - p % chunk) // 16, p // 16 + 1):
                        assert m.groups[1].row_pages[r][b] != 0
                m.commit(r, new_len)
                live[r] = new_len
        elif live:
            r = rng.choice(list(live))
            m.release(r)
            del live[r]
        m.check()
        for r, n in live.items():
            assert len(m.groups[1].owned(r)) <= pages_for(chunk, 16) + 1
    for r in list(live):
        m.release(r)
    assert all(f == g.allocator.num_pages for f, g in zip(m.free_pages(), m.groups))


def test_the_scheduler_asks_for_a_chunk_not_for_the_whole_row():
    from socrates_b200.engine.scheduler import Request, Scheduler, TooLong
    needs = [CacheNeeds(PagedKVSpec(1, 4, chunk=32))]
    m = CacheManager(needs, max_rows=2, max_len=640, page_size=16, num_pages=5, dtype=torch.float32, device="cpu")
    Scheduler(m, max_batch=2, max_len=640, token_budget=64, max_queue=8).submit(Request(list(range(300)), 20))
    m = CacheManager(needs, max_rows=2, max_len=640, page_size=16, num_pages=3, dtype=torch.float32, device="cpu")
    with pytest.raises(TooLong):
        Scheduler(m, max_batch=2, max_len=640, token_budget=64, max_queue=8).submit(Request(list(range(300)), 20))


# ------------------------------------------------------------------------------------------ the plain statement
def test_plain_chunks_and_slopes():
    seen = plain.visible(10, 4)
    assert seen[3].tolist() == [True] * 4 + [False] * 6 and seen[4].tolist() == [False] * 4 + [True] + [False] * 5
    assert seen[9, 8] and not seen[9, 7] and plain.visible(5, None).sum() == 15
    assert torch.allclose(plain.slopes(8), torch.tensor([2.0 ** -(h + 1) for h in range(8)], dtype=F64))
    assert abs(float(plain.slopes(3)[0]) - 2.0 ** (-8.0 / 3.0)) < 1e-15


def test_plain_rotation_depends_on_the_distance_only():
    g = torch.Generator().manual_seed(3)
    for rot in ({"dims": 8, "base": 100.0}, {"dims": 6, "base": 50.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 40}}):
        q, k = torch.randn(1, 1, 8, generator=g, dtype=F64), torch.randn(1, 1, 8, generator=g, dtype=F64)
        at = lambda t, p: plain.rotate_halves(t, torch.tensor([p]), rot)
        assert abs(float((at(q, 7) * at(k, 3)).sum() - (at(q, 104) * at(k, 100)).sum())) < 1e-9
        assert abs(float(at(q, 9).norm() - q.norm())) < 1e-12           # why the norm may come before the rotation


def test_plain_values_are_blended_from_the_first_layer():
    """A layer with lambda one passes the first layer's values on; with lambda zero it keeps its own."""
    cfg, rank = TINY["B"]
    w = {k: v.double() for k, v in make_weights(cfg, 2, rank).items()}
    h = torch.randn(20, cfg["width"], generator=torch.Generator().manual_seed(5), dtype=F64)
    m, eps, pos = cfg["layers"][1]["mixer"], 1e-5, torch.arange(20)
    _, first = plain.attention(h, w, "l0.mix.", cfg["layers"][0]["mixer"], eps, pos, None, distance=True)
    run = lambda lam, vf: plain.attention(h, {**w, "l1.mix.vmix": torch.tensor(lam, dtype=F64)}, "l1.mix.", m, eps, pos, vf)[0]
    own = plain.attention(h, w, "l1.mix.", {**m, "v_mix": False}, eps, pos)[0]
    assert torch.allclose(run(0.0, first), own) and torch.allclose(run(0.4, None), own)
    other = {**w, "l1.mix.v": w["l1.mix.v"] * 0}
    swapped = plain.attention(h, {**other, "l1.mix.vmix": torch.tensor(1.0, dtype=F64)}, "l1.mix.", m, eps, pos, first)[0]
    assert torch.allclose(run(1.0, first), swapped) and not torch.allclose(run(1.0, first), own)


def test_plain_recurrence_continues_from_a_state():
    cfg, rank = TINY["A"]
    w = {k: v.double() for k, v in make_weights(cfg, 2, rank).items()}
    h = torch.randn(30, cfg["width"], generator=torch.Generator().manual_seed(4), dtype=F64)
    m = cfg["layers"][0]["mixer"]
    whole = plain.wkv(h, w, "l0.mix.", m, 1e-6)[0]
    first, S, last = plain.wkv(h[:11], w, "l0.mix.", m, 1e-6)
    assert torch.allclose(torch.cat([first, plain.wkv(h[11:], w, "l0.mix.", m, 1e-6, S, last)[0]]), whole, atol=1e-12)


def test_plain_choice_and_clear_routing():
    z = torch.tensor([3.0, -4.0, -4.0, 1.0, 1.5, -4.0], dtype=F64)
    ids, share = plain.choose(z, {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 2, "keep": 1}})
    assert ids == [4, 3] and abs(float(share.sum()) - 2.0) < 1e-12        # two good ones beat one far ahead
    for name, (cfg, rank) in TINY.items():
        w = {k: v.double() for k, v in make_weights(cfg, SEEDS.get(name, 5), rank).items()}
        ids = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(9)).tolist()
        gaps, seen = [], set()
        original = plain.choose

        def watch(z, router):
            chosen, share = original(z, router)
            for d in (0.02, -0.02):                       # a little larger or smaller: the same choice
                assert set(original(z * (1 + d), router)[0]) == set(chosen), name
            noise = 0.01 * torch.randn(z.shape, generator=torch.Generator().manual_seed(len(gaps))).to(F64)
            assert set(original(z + noise, router)[0]) == set(chosen), name
            gaps.append(1)
            seen.add((router["experts"], router["top"], tuple(sorted(chosen))))
            return chosen, share
        plain.choose = watch
        try:
            plain.forward(cfg, w, ids)
        finally:
            plain.choose = original
        if gaps:
            assert len(seen) > 3, name                    # choices vary
    assert CODE == 3 and math.isclose(float(plain.gelu_tanh(torch.tensor(1.0, dtype=F64))), 0.8411919906082768)
