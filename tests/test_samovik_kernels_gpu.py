"""The kernels of the Samovik decoder alone, against plain float64 statements of what they compute."""

import math

import pytest
import torch

import plain_samovik as plain

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def err(got, want):
    return float((got - want).abs().max() / want.abs().max())


@pytest.mark.parametrize("d", [37, 40, 1024])
@pytest.mark.parametrize("dtype", DTYPES)
def test_dynamic_tanh_fold(d, dtype):
    """tanh(alpha x) * w + b of a stream to which a normed branch of several parts is added first; some rows only."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(d)
    N, eps = 9, 1e-5
    x, parts = torch.randn(N, d, generator=g) * 2, torch.randn(3, N, d, generator=g)
    gain, bias, post = (torch.randn(d, generator=g) for _ in range(3))
    alpha = torch.tensor([0.7])
    b = plain.rms(parts.double().sum(0), eps) * post.double()
    want_x = x.double() + b
    w = {"n": gain.double(), "n.b": bias.double(), "n.alpha": alpha.double()[0]}
    want = plain.dyn_tanh(want_x, w, "n")
    tol = 1e-5 if dtype == torch.float32 else 8e-3
    idx = i32([4, 0, 8])
    res, out, few = x.to(DEV), torch.empty(N, d, device=DEV, dtype=dtype), torch.empty(3, d, device=DEV, dtype=dtype)
    kw = dict(branch_gain=post.to(DEV), branch_eps=eps, tanh_alpha=alpha.to(DEV), tanh_bias=bias.to(DEV))
    ops.fold_rmsnorm(res, parts.to(DEV), gain.to(DEV), few, 0.0, idx, **kw)
    assert torch.equal(res.cpu(), x) and err(few.double().cpu(), want[[4, 0, 8]]) < tol
    ops.fold_rmsnorm(res, parts.to(DEV), gain.to(DEV), out, 0.0, **kw)
    assert err(out.double().cpu(), want) < tol and err(res.double().cpu(), want_x) < 1e-5


def walk(q, k, v, w, u, S):
    """The recurrence token by token: q, k, w [T, H, D], v [T, H, Dv], u [H, D] or None, S [H, D, Dv]."""
    rows = []
    for t in range(q.shape[0]):
        kv = k[t][:, :, None] * v[t][:, None, :]
        after = w[t][:, :, None] * S + kv
        rows.append(torch.einsum("hde,hd->he", after if u is None else S + u[:, :, None] * kv, q[t]).reshape(-1))
        S = after
    return torch.stack(rows), S


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(2, 12, 20), (1, 70, 9), (3, 130, 8), (2, 5, 7), (3, 64, 64), (2, 128, 40), (1, 256, 72), (2, 32, 136)])
@pytest.mark.parametrize("kind", ["fixed", "channel", "fixed bonus", "channel after"])
def test_linear_recurrence(dtype, shape, kind):
    """Three requests in one launch, continued from states; decays fixed and per channel, read after the write and
    before it with a bonus; SiLU on the way in; portions cut into segments of 16, 33 and 64 tokens and not cut."""
    from socrates_b200.kernels import ops
    H, D, Dv = shape
    g = torch.Generator().manual_seed(sum(shape) + len(kind))
    lens, slots = [150, 1, 40], [3, 0, 2]
    N, C = sum(lens), H * D
    cols = 2 * C + H * Dv
    proj = torch.randn(N, cols + 3 if D % 2 else cols, generator=g).to(dtype)      # ragged rows and whole 16-byte pieces
    p = proj.double()
    fixed, silu = "fixed" in kind, "bonus" not in kind
    decay = torch.rand(H, generator=g) * 0.5 + 0.5
    raw, base = torch.randn(N, C, generator=g) - 2, torch.randn(C, generator=g) * 0.5
    u = torch.rand(H, D, generator=g) if kind in ("channel", "fixed bonus") else None
    act = plain.silu if silu else (lambda z: z)
    q, k, v = (act(t).view(N, H, -1) for t in (p[:, :C], p[:, C:2 * C], p[:, 2 * C:cols]))
    w = decay.double()[None, :, None].expand(N, H, D) if fixed else torch.exp(-torch.exp(raw.double() + base.double())).view(N, H, D)
    state = torch.randn(5, H, D, Dv, generator=g)
    want, after, at = [], {}, 0
    for n, s in zip(lens, slots):
        sl = slice(at, at + n)
        o, after[s] = walk(q[sl], k[sl], v[sl], w[sl], u.double() if u is not None else None, state[s].double())
        want.append(o)
        at += n
    want = torch.cat(want)
    starts = i32([0, 150, 151, N])
    kw = dict(silu_qk=silu, silu_v=silu, bonus=u.to(DEV) if u is not None else None)
    kw.update(dict(decay=decay.to(DEV)) if fixed else dict(raw_decay=(raw.to(DEV), 0), decay_base=base.to(DEV)))
    pd = proj.to(DEV)
    for seg in (16, 33, 64, 1000):
        st, out = state.to(DEV), torch.empty(N, H * Dv, device=DEV)
        n = 2 * (N // seg)
        ops.linear_recurrence(out, (pd, 0), (pd, C), (pd, 2 * C), st, starts, i32(slots), dtype, seg_len=seg,
                              seg_state=torch.empty(max(1, n * C * Dv), device=DEV), seg_prod=torch.empty(max(1, n * C), device=DEV), **kw)
        assert err(out.double().cpu(), want) < 2e-5, seg
        for s in slots:
            assert err(st[s].double().cpu(), after[s]) < 2e-5, (seg, s)
        assert torch.equal(st[[1, 4]].cpu(), state[[1, 4]])
    # the inputs as partial sums of a product cut along K
    parts = torch.randn(3, N, proj.shape[1], generator=g)
    parts[2] = proj.float() - parts[0] - parts[1]
    st, out = state.to(DEV), torch.empty(N, H * Dv, device=DEV)
    ps = parts.to(DEV)
    ops.linear_recurrence(out, (ps, 0), (ps, C), (ps, 2 * C), st, starts, i32(slots), dtype, seg_len=1000, **kw)
    assert err(out.double().cpu(), want) < 2e-5


def test_linear_recurrence_segments_follow_the_shape():
    from socrates_b200.kernels import ops
    assert ops.linear_recurrence_scratch(40, 1, 2, 8, 8) == (0, 0)
    seg = ops.linear_recurrence_segment(2048, 1)
    assert ops.linear_recurrence_scratch(2048, 1, 2, 8, 16) == (2 * (2048 // seg) * 2 * 8 * 16, 2 * (2048 // seg) * 2 * 8)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,groups", [(24, 3), (256, 1), (256, 8), (35, 5), (2048, 32), (4096, 1), (640, 5), (1056, 1)])
def test_norm_gate(dtype, C, groups):
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(C)
    N, eps = 11, 1e-5
    x, gain = torch.randn(N, C, generator=g), torch.randn(C, generator=g)
    gate = torch.randn(N, C + 8, generator=g).to(dtype)
    y = plain.rms(x.double().view(N, groups, -1), eps).view(N, C) * gain.double()
    parts = torch.randn(2, N, C + 8, generator=g)
    parts[1] = gate.float() - parts[0]
    for act, f in (("sigmoid", plain.sigmoid), ("silu", plain.silu)):
        want = y * f(gate.double()[:, 8:])
        for src in (gate, parts):
            out = torch.empty(N, C, device=DEV, dtype=dtype)
            ops.norm_gate(out, x.to(DEV), gain.to(DEV), (src.to(DEV), 8), groups, eps, act)
            assert err(out.double().cpu(), want) < (1e-5 if dtype == torch.float32 else 1e-2), act


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [40, 37, 2056])
def test_token_shift_mix_and_its_tail(dtype, d):
    """Blends with the token before: inside a portion, from the slot at its start, from zero in a fresh slot; the
    portion's last token is kept for the next."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(d)
    lens, slots = [5, 1, 3], [2, 3, 0]
    x, mu, last = torch.randn(9, d, generator=g).to(dtype), torch.rand(3, d, generator=g), torch.randn(4, 1, d, generator=g)
    last[3] = 0
    prev = torch.cat([last[2].double(), x[:4].double(), last[3].double(), last[0].double(), x[6:8].double()])
    want = x.double()[None] + (prev - x.double())[None] * mu.double()[:, None]
    out, ld = torch.empty(3, 9, d, device=DEV, dtype=dtype), last.to(DEV)
    ops.token_shift_mix(out, x.to(DEV), mu.to(DEV), ld, i32([2] * 5 + [3] + [0] * 3))
    assert err(out.double().cpu(), want) < (1e-6 if dtype == torch.float32 else 8e-3)
    assert torch.equal(ld.cpu(), last)
    ops.short_conv_tail(ld, x.to(DEV), None, 2, i32([0, 5, 6, 9]), i32(slots))
    assert torch.equal(ld[[2, 3, 0], 0].cpu(), x[[4, 5, 8]].float()) and torch.equal(ld[1].cpu(), last[1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,top,K", [(3, 1, 40), (16, 4, 192), (33, 5, 37), (70, 70, 256), (12, 12, 1030)])
def test_router(dtype, E, top, K):
    """Choices and weights against the plain statement, ties aside; the same bits alone and among 600 tokens."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(E)
    N = 600
    x, router, bias = torch.randn(N, K, generator=g).to(dtype), torch.randn(E, K, generator=g) * 0.3, torch.randn(E, generator=g)
    w = {"router": router.double(), "router.b": bias.double()}
    ids, share = plain.choose(x.double(), w, "", top)
    dense = torch.zeros(N, E, dtype=torch.float64).scatter_(1, ids, share)
    z = (x.double() @ router.double().T + bias.double()).sort(-1, descending=True).values
    gap = (z[:, :-1] - z[:, 1:])[:, :top].min(-1).values > 1e-4
    xd, rd, bd = x.to(DEV), router.to(DEV), bias.to(DEV)

    def run(rows):
        n = rows.shape[0]
        o = (torch.empty(n, E, device=DEV), torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV))
        ops.moe_router(rows, rd, bd, *o, top)
        return o
    weights, got, picked = run(xd)
    assert float(gap.double().mean()) > 0.5
    assert torch.equal(got.cpu().long()[gap], ids[gap])
    assert err(weights.double().cpu()[gap], dense[gap]) < 1e-4 and err(picked.double().cpu()[gap], share[gap]) < 1e-4
    for n in (0, 417):
        one = run(xd[n:n + 1].contiguous())
        assert all(torch.equal(a[0], b[n]) for a, b in zip(one, (weights, got, picked)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,F,Fs", [(4, 16, 24), (5, 10, 0), (3, 8, 6)])
def test_clamped_experts_units(dtype, experts, F, Fs):
    """All experts' units and the shared one's with clamps of their own; what an unchosen expert would read is not read."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(F)
    N, W = 13, experts * F + Fs
    x = (torch.randn(N, 2 * W, generator=g) * 2).to(dtype)
    weights = torch.rand(N, experts, generator=g) * (torch.rand(N, experts, generator=g) > 0.4)
    e = torch.arange(W) // F
    limit = torch.where(torch.arange(W) < experts * F, 1.3, 0.6).double()
    gt, up = torch.minimum(x.double()[:, :W], limit), torch.maximum(torch.minimum(x.double()[:, W:], limit), -limit)
    scale = torch.cat([weights.double(), torch.ones(N, 1, dtype=torch.float64)], -1)[:, e.clamp(max=experts)]
    want = gt * plain.sigmoid(1.702 * gt) * (up + 1) * scale
    dead = torch.cat([scale == 0] * 2, -1)
    parts = torch.randn(3, N, 2 * W, generator=g)
    parts[2] = x.float() - parts[0] - parts[1]
    for src in (x, parts):
        src = src.clone()
        src[..., dead] = float("nan")
        out = torch.empty(N, W, device=DEV, dtype=dtype)
        ops.moe_glu_clamp(out, src.to(DEV), weights.to(DEV), experts, F, 1.3, 0.6, 1.702, 1.0)
        assert err(out.double().cpu(), want) < (1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_gelu_lookup(dtype):
    """gelu times a slice of the token's row; an id below zero stands for a token that was sampled on the device."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(1)
    N, F, V = 7, 12, 20
    x, table = (torch.randn(N, F, generator=g) * 2).to(dtype), torch.randn(V, 3 * F, generator=g).to(dtype)
    ids, feedback = [3, 0, 19, -1, 5, -3, 3], [7, 8, 11]
    real = [3, 0, 19, 7, 5, 11, 3]
    want = plain.gelu_tanh(x.double()) * table.double()[real][:, F:2 * F]
    parts = torch.stack([x.float() * 0.25, x.float() * 0.75])
    for src in (x, parts):
        out = torch.empty(N, F, device=DEV, dtype=dtype)
        ops.gelu_lookup(out, src.to(DEV), table.to(DEV), F, i32(ids), i32(feedback))
        assert err(out.double().cpu(), want) < (1e-5 if dtype == torch.float32 else 1e-2)


def test_tanh_activation():
    from socrates_b200.kernels import ops
    x = torch.linspace(-8, 8, 60, device=DEV).view(3, 20)
    out = torch.empty_like(x)
    ops.bias_act(out, x, None, "tanh")
    assert torch.allclose(out.double(), torch.tanh(x.double()), atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,A,B", [(3, 8, 20), (2, 128, 96), (4, 48, 64), (1, 5, 7), (2, 200, 264)])
@pytest.mark.parametrize("transposed", [False, True])
def test_matrix_per_head(dtype, H, A, B, transposed):
    """Few tokens, a prompt portion, and ragged heads, with values carried in front of every head."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(A)
    w = torch.randn(H * A, B, generator=g).to(dtype)
    nin, nout = (A, B) if transposed else (B, A)
    for N, carry in ((1, 0), (8, 8), (16, 2), (33, 8), (150, 4), (70, 0)):
        x = torch.randn(N, H * (carry + nin) + (-H * (carry + nin)) % 8, generator=g).to(dtype)
        xh = x[:, :H * (carry + nin)].double().view(N, H, carry + nin)
        wh = w.double().view(H, A, B)
        y = torch.einsum("nhi,hio->nho" if transposed else "nhi,hoi->nho", xh[..., carry:], wh)
        want = torch.cat([xh[..., :carry], y], -1).reshape(N, -1)
        out = torch.empty(N, H * (carry + nout), device=DEV, dtype=dtype)
        ops.head_matmul(out, carry, carry + nout, x.to(DEV), carry, carry + nin, w.to(DEV), H, transposed, carry)
        assert err(out.double().cpu(), want) < (1e-5 if dtype == torch.float32 else 1e-2), N


def paged_rows(lens, D, page, g, dtype):
    """Cached rows of two requests scattered over pages that hold garbage elsewhere."""
    width = max(-(-n // page) for n in lens)
    total = sum(-(-n // page) for n in lens)
    perm = (torch.randperm(total, generator=g) + 1).tolist()
    pool = torch.full((total + 1, 1, page, D), 50.0, dtype=dtype)
    table, rows = torch.zeros(len(lens), width, dtype=torch.int32), []
    for r, n in enumerate(lens):
        x = torch.randn(n, D, generator=g).to(dtype)
        rows.append(x.double())
        for b in range(-(-n // page)):
            table[r, b] = perm.pop()
            part = x[b * page:(b + 1) * page]
            pool[int(table[r, b]), 0, :part.shape[0]] = part
    return pool, table, rows


def one_head_attention(q, rows, first, rank, scale, window):
    """q [n, H, D] of the tokens at first, first + 1, ... over cached rows [T, D]; values are the last `rank` dims."""
    n, T = q.shape[0], rows.shape[0]
    s = torch.einsum("ihd,jd->hij", q, rows) * scale
    i, j = torch.arange(first, first + n)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & ((i - j < window) if window else torch.ones(1, 1, dtype=torch.bool))
    return torch.einsum("hij,jr->ihr", torch.softmax(s.masked_fill(~seen, -math.inf), -1), rows[:, rows.shape[1] - rank:])


@pytest.mark.parametrize("H,dr,rank", [(3, 8, 40), (16, 32, 96), (20, 16, 136), (5, 24, 264), (70, 0, 64), (1, 8, 8), (33, 64, 512)])
@pytest.mark.parametrize("window", [0, 9, 100])
def test_attention_over_one_cached_head(H, dr, rank, window):
    """Prompt tiles behind earlier tokens, and single tokens in 1, 3 and 16 key shares, of two requests; with windows
    shorter than a page and longer than a tile; one query's score stands out so that a wrong key shows."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(H + rank)
    D, page, lens, new = dr + rank, 16, [203, 61], [90, 33]
    pool, table, rows = paged_rows(lens, D, page, g, torch.bfloat16)
    scale = 1.5 / D ** 0.5
    N = sum(new)
    q = torch.randn(N, H, D, generator=g).to(torch.bfloat16)
    q[89] = rows[0][202 - (7 if window else 180)].to(torch.bfloat16) * 2       # the last query of request 0 picks one key
    gate = torch.randn(N, H + 3, generator=g).to(torch.bfloat16)
    f = plain.sigmoid(gate.double()[:, :H])[..., None]
    want = torch.cat([one_head_attention(q[:90].double(), rows[0], 113, rank, scale, window),
                      one_head_attention(q[90:].double(), rows[1], 28, rank, scale, window)])
    first = [113, 28]
    positions = i32([113 + i for i in range(90)] + [28 + i for i in range(33)])
    args = (q.view(N, H * D).to(DEV), pool.to(DEV), rank, table.to(DEV), i32([0] * 90 + [1] * 33), positions,
            i32([0, 90, N]), i32([0, 1]), i32(first), H, scale, window)
    assert ops.attention_latent_supports(H, D, rank)
    for gt, ref in ((None, want), (gate.to(DEV), want * f)):
        out = torch.empty(N, H * rank, device=DEV, dtype=torch.bfloat16)
        ops.attention_latent(out, *args, gate=gt, prompt=True)
        assert err(out.double().cpu(), ref.reshape(N, -1)) < 1e-2
        for NP in (1, 3, 16):
            out = torch.empty(N, H * rank, device=DEV, dtype=torch.bfloat16)
            ops.attention_latent(out, *args, gate=gt, num_partitions=NP,
                                 part_o=torch.empty(N * H * NP * rank, device=DEV), part_ml=torch.empty(N * H * NP * 2, device=DEV))
            assert err(out.double().cpu(), ref.reshape(N, -1)) < 1e-2, NP


@pytest.mark.parametrize("window", [5, 64, 65])
def test_latent_attention_at_a_windows_edge(window):
    """The key just inside the window decides the output, the same key just outside it must not be seen."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(window)
    D, rank, H, T = 24, 16, 2, 150
    pool, table, rows = paged_rows([T], D, 16, g, torch.bfloat16)
    q = torch.zeros(T, H, D)
    for i in range(T):                                       # query i wants key i - window + 1 (even i) or i - window (odd i)
        j = max(0, i - window + (1 if i % 2 == 0 else 0))
        q[i] = 4.0 * rows[0][j].float()
    q = q.to(torch.bfloat16)
    want = one_head_attention(q.double(), rows[0], 0, rank, 0.5, window)
    args = (q.view(T, -1).to(DEV), pool.to(DEV), rank, table.to(DEV), i32([0] * T), i32(list(range(T))), i32([0, T]), i32([0]),
            i32([0]), H, 0.5, window)
    for prompt in (True, False):
        out = torch.empty(T, H * rank, device=DEV, dtype=torch.bfloat16)
        ops.attention_latent(out, *args, prompt=prompt)
        assert err(out.double().cpu(), want.reshape(T, -1)) < 1e-2


@pytest.mark.parametrize("dtype", DTYPES)
def test_value_heads_beyond_256_dims_on_the_cuda_cores(dtype):
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    rank, dr, H, T = 300, 6, 3, 40
    pool, table, rows = paged_rows([T], rank + dr, 16, g, dtype)
    q = torch.randn(T, H, rank + dr, generator=g).to(dtype)
    want = one_head_attention(q.double(), rows[0], 0, rank, 0.1, 0)
    v_pool = pool[..., dr:].contiguous()
    for NP in (1, 3):
        out = torch.empty(T, H * rank, device=DEV, dtype=dtype)
        ops.attention_bias(out, q.view(T, -1).to(DEV), pool.to(DEV), v_pool.to(DEV), table.to(DEV), i32([0] * T), i32(list(range(T))),
                           H, 0.1, num_partitions=NP, part_o=torch.empty(T * H * NP * rank, device=DEV), part_ml=torch.empty(T * H * NP * 2, device=DEV))
        assert err(out.double().cpu(), want.reshape(T, -1)) < (1e-5 if dtype == torch.float32 else 1e-2)
