"""The Kusirax decoder in the engine against the plain statement of its equations.

Parts alone; the stream after every layer; whole prompts; token-by-token decoding; portions down to two tokens;
unequal requests in one batch against each alone; rows, pages and state slots that are used again; a planted key that
decides an attention output: far back, at page borders and on either side of a tile of keys, and the first key of a
chunk against the last one of the chunk before, in prompts and decoded; a planted write that the state must carry over
hundreds of tokens; values of the first layer; long decoding; greedy generation through the engine's entry point and
scheduler; the command line; a replay through bin/trace_run.
"""

import json

import pytest
import torch

import plain_kusirax as plain
from bofusun_tiny import Harness, rel_err
from kusirax_tiny import TINY, make_folder, save_weights
from traces import Trace, compare, last_decoded, mixed, portions, run_trace, whole

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {torch.float32: 2e-4, torch.bfloat16: 6e-2}
PART_TOL = {torch.float32: 1e-4, torch.bfloat16: 4e-2}
DTYPES = [torch.float32, torch.bfloat16]
NAMES = list(TINY)
F64 = torch.float64


def tokens(vocab, n, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def part_err(got, want):
    return float((got - want).abs().max() / want.abs().max())


def run_part(h, part, x, dtype, sizes, entry=None, v_first=None):
    """Feed x [n, width] through a mixer (entry: its place in the run order) or a feed-forward in portions; `v_first`
    [n, values]: what the layer that keeps its values left for a mixer that blends."""
    from socrates_b200.engine.context import CacheView
    from socrates_b200.engine.runner import StepEntry
    n, got, start, k = x.shape[0], [], 0, 0
    h.cache.assign(1)
    while start < n:
        c = min(sizes[min(k, len(sizes) - 1)], n - start)
        assert h.cache.reserve(1, start + c)
        ctx = h.runner.prepare([StepEntry(1, [0] * c, start, [c - 1])])
        xin = x[start:start + c].to(dtype).to(DEV).contiguous()
        if v_first is not None:
            ctx.buffers.take("mv_first_values", c, (v_first.shape[1],), torch.float32).copy_(v_first[start:start + c].float())
        b = part.forward(ctx, xin) if entry is None else part.forward(ctx, xin, CacheView(h.cache, entry, True))
        assert b.plain
        got.append(b.partial.double().sum(0).cpu())
        h.cache.commit(1, start + c)
        start, k = start + c, k + 1
    h.cache.release(1)
    assert int(h.runner.status.item()) == 0
    return torch.cat(got)


def plain_mixer(kind, x, w, pre, m, eps, v_first=None):
    if kind == "wkv":
        return plain.wkv(x, w, pre, m, eps)[0]
    return plain.attention(x, w, pre, m, eps, torch.arange(x.shape[0]), v_first, distance=kind == "attention_2")[0]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_mixers_alone(tmp_path, dtype, name):
    g = torch.Generator().manual_seed(4)
    folder, cfg, w = make_folder(tmp_path, name)
    h = Harness(folder, dtype, max_len=320)
    for i, l in enumerate(cfg["layers"]):
        n, m = (170 if name in ("B", "C") else 70), l["mixer"]
        part, v_first = h.model.layers[i].mixer, None
        x = torch.randn(n, cfg["width"], generator=g).bfloat16().double()
        if getattr(part, "values", None) == "blend":
            v_first = torch.randn(n, m["kv_heads"] * m["vdim"], generator=g).double()
        want = plain_mixer(l["type"], x, w, f"l{i}.mix.", m, cfg["norm"]["eps"], v_first)
        for sizes in ((n,), (1,), (33, 2, 1, 30, 1)):
            got = run_part(h, part, x, dtype, sizes, entry=i, v_first=v_first)
            assert part_err(got, want) < PART_TOL[dtype], (i, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_feed_forwards_alone(tmp_path, dtype, name):
    """Inputs whose code channels are plus or minus one common size, as in the stream (clear routing)."""
    g = torch.Generator().manual_seed(6)
    folder, cfg, w = make_folder(tmp_path, name)
    h = Harness(folder, dtype, max_len=96)
    for i, l in enumerate(cfg["layers"]):
        if l["mlp"] is None:
            continue
        x = torch.randn(50, cfg["width"], generator=g)
        x[:, :3] = torch.sign(x[:, :3]) * (0.6 + 2.0 * torch.rand(50, 1, generator=g))
        x = x.bfloat16().double()
        x[:, 1:3] = torch.sign(x[:, 1:3]) * x[:, :1].abs()
        want = (plain.dense if l["mlp"]["kind"] == "dense" else lambda *a: plain.experts(*a, l["mlp"]))(x, w, f"l{i}.mlp.")
        for sizes in ((50,), (1,), (7, 2, 16)):
            got = run_part(h, h.model.layers[i].feed_forward, x, dtype, sizes)
            assert part_err(got, want) < PART_TOL[dtype], (i, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_stream_after_every_layer(tmp_path, dtype, name):
    import socrates_b200.engine.context as C
    folder, cfg, w = make_folder(tmp_path, name)
    ids = tokens(cfg["vocab"], 45, 11)
    want, got = [], []
    plain.forward(cfg, w, ids, want)
    h = Harness(folder, dtype)
    original = C.StepContext.__init__

    def patched(self, *a, **k):
        original(self, *a, **k)

        def look(i, stream):
            assert stream.pending is None and torch.equal(stream.rows, stream.residual.to(dtype))
            got.append(stream.residual.double().cpu())
        self.after_run = look
    C.StepContext.__init__ = patched
    try:
        h.step([("a", ids)])
    finally:
        C.StepContext.__init__ = original
    assert len(got) == len(want) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(got, want)):
        assert part_err(a, b) < (1e-4 if dtype == torch.float32 else 6e-2), i


# ------------------------------------------------------------------------------------------
# whole models

@pytest.fixture(scope="module")
def models(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("kusirax")
    out = {}
    for name in TINY:
        folder, cfg, w = make_folder(tmp, name)
        seqs = [tokens(cfg["vocab"], n, 50 + i) for i, n in enumerate((150, 23, 77, 4))]
        out[name] = (folder, cfg, w, seqs, [plain.forward(cfg, w, s) for s in seqs])
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_decoding_and_portions(models, dtype, name):
    folder, cfg, w, seqs, want = models[name]
    h = Harness(folder, dtype)
    ids, ref = seqs[0], want[0]
    ways = {"whole": h.run("w", ids, (len(ids),)), "token by token": h.run("d", ids, (1,)), "pairs": h.run("p", ids, (2,)),
            "ragged": h.run("r", ids, (7, 2, 16, 3, 2, 33, 5, 17, 2, 1, 1, 1, 40)),
            "prompt then decoded": h.run("t", ids, (len(ids) - 100, 1))}
    for way, got in ways.items():
        assert rel_err(got, ref) < TOL[dtype], way
    if dtype == torch.float32:          # how the tokens were cut changes rounding only
        for way, got in ways.items():
            assert rel_err(got, ways["whole"]) < 5e-5, way
    # the first tokens of a sequence, alone
    assert rel_err(h.run("f", seqs[3], (1,)), want[3]) < TOL[dtype]
    assert rel_err(h.run("g", seqs[3], (4,)), want[3]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_requests_in_one_batch(models, dtype, name):
    """Four requests of 150, 23, 77 and 4 tokens: portions of some beside single tokens of others, a request that
    joins late and one that sits steps out; each must come out as it does alone."""
    folder, cfg, w, seqs, want = models[name]
    h = Harness(folder, dtype)
    alone = [Harness(folder, dtype).run("x", s, (len(s),)) for s in seqs] if dtype == torch.float32 else None
    fed, got = [0] * 4, [[] for _ in seqs]
    plan = [[(0, 60), (1, 1)], [(0, 1), (1, 1), (2, 30)], [(0, 2), (2, 1), (3, 4)], [(1, 20), (2, 1)],
            [(0, 30), (1, 1), (2, 44)], [(0, 1), (2, 1)], [(0, 56)]]
    for step in plan:
        entries = [(f"r{i}", seqs[i][fed[i]:fed[i] + c]) for i, c in step if fed[i] < len(seqs[i])]
        ended = [f"r{i}" for i, c in step if fed[i] < len(seqs[i]) and fed[i] + c >= len(seqs[i])]
        out = h.step(entries, end=ended)
        for i, c in step:
            if f"r{i}" in out:
                got[i].append(out[f"r{i}"])
                fed[i] += out[f"r{i}"].shape[0]
    for i, s in enumerate(seqs):
        mine = torch.cat(got[i])
        assert mine.shape[0] == len(s)
        assert rel_err(mine, want[i]) < TOL[dtype], i
        if alone is not None:
            assert rel_err(mine, alone[i]) < 5e-5, i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_rows_pages_and_state_slots_are_used_again(models, dtype, name):
    """Two rows and a pool of 12 pages of 16 slots serve eight requests one after another, in portions and token by
    token: every page is handed out several times, dirty from its previous owner, chunked layers give pages back on the
    way, and every state slot starts from zero again although its last owner left something behind."""
    folder, cfg, w, seqs, want = models[name]
    h = Harness(folder, dtype, max_rows=2, max_len=160, pages=12)
    order = [0, 1, 2, 3, 2, 0, 3, 1]
    for k in range(0, len(order), 2):
        a, b = order[k], order[k + 1]
        ga = h.run(f"a{k}", seqs[a], (31, 1, 2, 64))
        fed, gb = 0, []
        while fed < len(seqs[b]):                       # the second of the pair decodes token by token
            gb.append(h.step([(f"b{k}", seqs[b][fed:fed + 1])], end=[f"b{k}"] if fed + 1 == len(seqs[b]) else [])[f"b{k}"])
            fed += 1
        assert rel_err(ga, want[a]) < TOL[dtype] and rel_err(torch.cat(gb), want[b]) < TOL[dtype], k
    assert h.cache.free_pages() == [12] * len(h.cache.groups)


def test_a_chunked_layer_holds_no_more_than_its_chunk(models):
    """Decoding 150 tokens of model D (chunks of 7) and C (33 and 100): pages of chunks that are over are free again."""
    for name in ("C", "D"):
        folder, cfg, w, seqs, want = models[name]
        h = Harness(folder, torch.float32, max_rows=1, max_len=160)
        for i, t in enumerate(seqs[0]):
            h.step([("a", [t])])
            for g in h.cache.groups:
                if g.spec.chunk is not None:
                    n = i + 1
                    assert len(g.owned(0)) == (-(-n // 16) - (n - n % g.spec.chunk) // 16 if n % g.spec.chunk or n % 16 else 0), (name, n)


# ------------------------------------------------------------------------------------------
# planted keys and writes

def _plant(kind, dim, vdim, chunk=None):
    m = {"heads": 2, "kv_heads": 1, "dim": dim, "vdim": vdim, "scale": 14.0 / dim, "v_mix": False}
    if kind == "attention_2":
        m.update(heads=1, softcap=40.0, mask={"size": chunk})
    return {"architecture": "Kusirax", "vocab": 50, "width": 48, "norm": {"eps": 1e-6}, "postln_alpha": 2.0,
            "layers": [{"type": kind, "mixer": m, "mlp": None}]}


def _planted(cfg, w, n, at, seed):
    """(inputs, weights): the key at `at` and the queries at the last, the 12th and the 28th before it point the same
    way, and no other key does."""
    m, width, last = cfg["layers"][0]["mixer"], cfg["width"], n - 1
    g = torch.Generator().manual_seed(seed)
    x = torch.randn(n, width, generator=g)
    u = x[at] / x[at].norm()
    planted = x[at].clone()
    x = x - (x @ u)[:, None] * u[None, :]
    x[at] = planted
    x = x.bfloat16().double()
    for p in (last - 28, last - 12):
        x[p] = x[last]
    e = torch.ones(m["dim"], dtype=F64) / m["dim"] ** 0.5
    w2 = dict(w)
    boost = 14.0 * m["dim"] ** 0.5 * 0.2
    for name, H, row in (("k", m["kv_heads"], x[at]), ("q", m["heads"], x[last])):
        t = w["l0.mix." + name].view(H, m["dim"], width) + boost * e[None, :, None] * (row / row.norm())[None, None, :]
        w2["l0.mix." + name] = t.reshape(H * m["dim"], width).bfloat16().double()
    return x, w2


def _check_planted(folder, cfg, w2, x, want, dtype, at, watched, where):
    n, last = x.shape[0], x.shape[0] - 1
    save_weights(folder, w2)
    h = Harness(folder, dtype, max_len=320)
    for sizes in ((n,), (last - 20, 1), (max(1, at + 1), 2, max(1, last - 20 - at - 3), 1)):
        got = run_part(h, h.model.layers[0].mixer, x, dtype, sizes, entry=0)
        if dtype == torch.float32:
            assert part_err(got, want) < PART_TOL[dtype], (where, at, sizes)
            continue
        err = (got - want).abs().max(-1).values / want.abs().max()
        assert float(err[watched].max()) < 0.08, (where, at, sizes)
        assert float(err.median()) < 0.02 and float(err.max()) < 0.15, (where, at, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(64, 64), (24, 40), (128, 128)])
def test_one_planted_key_decides_attention(tmp_path, dtype, dims):
    """Without rotation a planted pair scores high at every distance.  The key is far back among hundreds, on the last
    and first slot of a page, on either side of a tile of 64 keys, right behind a query; read in a prompt, decoded,
    and from an earlier portion; with heads that run on the tensor cores in the bfloat16 engine and heads that do not."""
    folder, cfg, w = make_folder(tmp_path, "plant", cfg=_plant("attention", *dims))
    m, n = cfg["layers"][0]["mixer"], 300
    last = n - 1
    for where, at in {"far": 2, "first": 0, "end of a page": 15, "start of a page": 16, "end of a tile": 63,
                      "start of a tile": 64, "later": 192, "near": last - 3}.items():
        x, w2 = _planted(cfg, w, n, at, 8)
        want = plain_mixer("attention", x, w2, "l0.mix.", m, 1e-6)
        lost = x.clone()
        lost[at] = x[at + 1]
        assert part_err(plain_mixer("attention", lost, w2, "l0.mix.", m, 1e-6)[last:], want[last:]) > 0.2, where
        _check_planted(folder, cfg, w2, x, want, dtype, at, [p for p in (last - 28, last - 12, last) if p > at], where)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(64, 64), (24, 40)])
@pytest.mark.parametrize("chunk", [45, 64, 100])
def test_a_planted_key_inside_and_outside_a_chunk(tmp_path, dtype, dims, chunk):
    """The first key of the last query's chunk decides its output; the last key of the chunk before must not be seen,
    although a query that saw it would look at nothing else.  Chunks that end on pages and tiles, and that do not."""
    folder, cfg, w = make_folder(tmp_path, "plant", cfg=_plant("attention_2", *dims, chunk))
    m, n = cfg["layers"][0]["mixer"], 294
    last = n - 1
    start = last - last % chunk
    assert last - 12 > start + 2
    for where, at in {"inside": start, "outside": start - 1, "one in": start + 1, "a page before": start - 17}.items():
        x, w2 = _planted(cfg, w, n, at, 9)
        want = plain_mixer("attention_2", x, w2, "l0.mix.", m, 1e-6)
        original = plain.visible

        def wrong(T, c):
            seen = original(T, c).clone()
            for p in (last - 12, last):
                seen[p, at] = at < start            # a query that sees one key too many, or one too few
            return seen
        plain.visible = wrong
        try:
            other = plain_mixer("attention_2", x, w2, "l0.mix.", m, 1e-6)
        finally:
            plain.visible = original
        assert part_err(other[last:], want[last:]) > 0.2 and part_err(other[last - 12:last - 11], want[last - 12:last - 11]) > 0.2, where
        _check_planted(folder, cfg, w2, x, want, dtype, at, [last - 12, last], where)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_state_carries_one_write_over_hundreds_of_tokens(tmp_path, dtype):
    """Decays of one, and keys that only token 3's input excites: what it writes is ALL that token 299 reads, in a
    prompt, decoded, and across portions (a lost or re-zeroed state reads nothing)."""
    cfg = {"architecture": "Kusirax", "vocab": 50, "width": 48, "norm": {"eps": 1e-6}, "postln_alpha": 2.0,
           "layers": [{"type": "wkv", "mlp": None, "mixer": {"heads": 3, "dim": 8}}]}
    folder, cfg, w = make_folder(tmp_path, "carry", cfg=cfg)
    n, width = 300, cfg["width"]
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(12))
    u = x[3] / x[3].norm()
    planted = x[3].clone()
    x = x - (x @ u)[:, None] * u[None, :]
    x[3] = planted
    x = x.bfloat16().double()
    u, w2, k = x[3] / x[3].norm(), dict(w), w["l0.mix.k"]
    w2["l0.mix.k"] = (torch.linspace(0.5, 1.5, k.shape[0], dtype=F64)[:, None] * u[None, :]).bfloat16().double()
    w2["l0.mix.mu.k"] = torch.zeros(width, dtype=F64)
    w2["l0.mix.w0"] = torch.full_like(w["l0.mix.w0"], -30.0)
    save_weights(folder, w2)
    m = cfg["layers"][0]["mixer"]
    want = plain_mixer("wkv", x, w2, "l0.mix.", m, 1e-6)
    lost = x.clone()
    lost[3] = x[4]
    assert part_err(plain_mixer("wkv", lost, w2, "l0.mix.", m, 1e-6)[-5:], want[-5:]) > 0.3
    h = Harness(folder, dtype, max_len=320)
    for sizes in ((n,), (280, 1), (4, 2, 150, 1)):
        err = (run_part(h, h.model.layers[0].mixer, x, dtype, sizes, entry=0) - want).abs().max(-1).values / want.abs().max()
        if dtype == torch.float32:
            assert float(err[3:].quantile(0.95)) < 1e-3, sizes
        else:       # a head's row is ONE write as its query sees it, normed: where that nears zero rounding decides
            assert float(err[3:].quantile(0.8)) < 0.05 and float(err[3:].median()) < 0.02, sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_values_of_the_first_layer_reach_the_others(models, dtype):
    """With lambda one every later layer's values are the first one's: what its own projection gives no longer counts,
    also for keys of earlier portions (the blended values are what the cache holds)."""
    folder, cfg, w, seqs, _ = models["A"]
    w2 = {**w, **{f"l{i}.mix.vmix": torch.ones((), dtype=F64) for i in (2, 3, 4)}}
    plain_logits = plain.forward(cfg, w2, seqs[2])
    assert rel_err(plain.forward(cfg, w, seqs[2]), plain_logits) > 0.1
    import tempfile
    from pathlib import Path
    with tempfile.TemporaryDirectory() as tmp:
        (Path(tmp) / "config.json").write_text(json.dumps(cfg))
        for own in (1.0, 0.0):
            save_weights(tmp, {**w2, **{f"l{i}.mix.v": w[f"l{i}.mix.v"] * own for i in (2, 3, 4)}})
            h = Harness(tmp, dtype)
            assert rel_err(h.run("w", seqs[2], (77,)), plain_logits) < TOL[dtype]
            assert rel_err(h.run("c", seqs[2], (20, 1, 30, 1)), plain_logits) < TOL[dtype]


def test_long_decoding(models):
    """400 tokens decoded one by one after a short prompt, two requests side by side, in float32."""
    for name in ("A", "D"):
        folder, cfg, w, _, _ = models[name]
        a, b = tokens(cfg["vocab"], 410, 77), tokens(cfg["vocab"], 300, 78)
        ra, rb = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
        h = Harness(folder, torch.float32, max_len=448)
        ga, gb = [h.step([("a", a[:10])])["a"]], []
        for t in range(10, 410):
            entries = [("a", a[t:t + 1])]
            if t - 10 < 300:
                entries.append(("b", b[t - 10:t - 9]))
            out = h.step(entries)
            ga.append(out["a"])
            if "b" in out:
                gb.append(out["b"])
        assert rel_err(torch.cat(ga), ra) < TOL[torch.float32] and rel_err(torch.cat(gb), rb) < TOL[torch.float32]


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_prompt_of_many_segments(models, dtype):
    """1,100 tokens in one step: the recurrence runs as segments side by side, attention over many tiles and chunks."""
    folder, cfg, w, _, _ = models["C"]
    ids = tokens(cfg["vocab"], 1100, 31)
    want = plain.forward(cfg, w, ids)
    h = Harness(folder, dtype, max_rows=1, max_len=1120)
    assert rel_err(h.run("w", ids, (1100,)), want) < TOL[dtype]
    assert rel_err(h.run("c", ids, (513, 2, 500, 80, 1)), want) < TOL[dtype]


# ------------------------------------------------------------------------------------------
# the entry point, the scheduler, the command line, the replay

@pytest.mark.parametrize("dtype,graphs", [("float32", False), ("bfloat16", True)])
@pytest.mark.parametrize("name", ["A", "B", "C", "E", "F", "G"])
def test_greedy_generation_through_the_entry_point(models, name, dtype, graphs):
    """Five requests through Engine: queued, admitted as rows come free, prompts cut by the token budget, decoded side
    by side (bfloat16: through recorded graphs), 60 new tokens each.  Every produced token is the plain statement's
    choice, or within its margin."""
    from socrates_b200 import Engine
    folder, cfg, w, seqs, _ = models[name]
    prompts = [seqs[0][:70], seqs[1], seqs[2][:40], seqs[3], seqs[0][70:101]]
    eng = Engine(str(folder), device="cuda:0", dtype=dtype, compile=graphs, max_batch=3, max_len=160,
                 max_new_tokens=60, token_budget=48)
    reqs = [eng.submit(p) for p in prompts]
    while eng.scheduler.has_work():
        assert eng.step()
        eng.scheduler.check()
    margin = 1e-3 if dtype == "float32" else 8e-2
    for p, r in zip(prompts, reqs):
        assert r.done and len(r.output) == 60
        logits = plain.forward(cfg, w, list(p) + r.output[:-1])
        scale = float(logits.abs().max())
        for i, tok in enumerate(r.output):
            row = logits[len(p) - 1 + i]
            best = int(torch.argmax(row))
            assert tok == best or float(row[best] - row[tok]) <= margin * scale, (i, tok, best)
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program(models, tmp_path, dtype):
    """bin/trace_run on model A: whole, tail decoded, portions, and a mix of up to four live requests
    in a pool that only holds the busiest step."""
    folder, cfg, w, seqs, want = models["A"]
    named = {f"s{i}": s for i, s in enumerate(seqs[:3])}
    reference = {k: want[i].numpy() for i, k in enumerate(named)}
    trace = Trace()
    for k, ids in named.items():
        whole(trace, "w:" + k, ids)
        last_decoded(trace, "d:" + k, ids, tail=20)
        portions(trace, "p:" + k, ids)
    mixed(trace, {f"m{j}:{k}": ids for j in range(2) for k, ids in named.items()}, seed=5, tail=20)
    result = run_trace(folder, dtype, trace, trace.most_held, tmp_path / "out")
    worst, where = compare(trace, result, reference, key=lambda rid: rid.split(":")[1])
    assert worst < TOL[torch.float32 if dtype == "float32" else torch.bfloat16], where


def test_command_line(models, tmp_path):
    """The generation command line on a Kusirax folder, and on a bare config.json with random weights."""
    import subprocess
    import sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    folder, cfg, _, _, _ = models["C"]
    common = ["--max-new-tokens", "7", "--max-len", "96", "--max-batch", "2"]
    proc = subprocess.run([sys.executable, "-m", "socrates_b200.inference_paged", "--model", str(folder),
                           "--num-prompts", "3", "--prompt-len", "21", "--prompt", "hello", *common],
                          cwd=str(root), capture_output=True, text=True, timeout=300)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert "4 requests, 2 rows" in proc.stdout and "> hello" in proc.stdout
    path = tmp_path / "config.json"
    path.write_text(json.dumps(TINY["B"][0]))
    proc = subprocess.run([sys.executable, "-m", "socrates_b200.inference_paged", "--random-config", str(path),
                           "--num-prompts", "2", "--prompt-len", "30", "--dtype", "float32", *common],
                          cwd=str(root), capture_output=True, text=True, timeout=300)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert "2 requests, 2 rows" in proc.stdout and "tok/s" in proc.stdout.splitlines()[-1]
