"""The kernels of the Kusirax decoder alone, against plain float64 statements of what they compute."""

import pytest
import torch

import plain_kusirax as plain

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def err(got, want):
    return float((got - want).abs().max() / want.abs().max())


# ------------------------------------------------------------------------------------------ scores
def attend(q, k, v, positions, scale, cap, slopes, chunk):
    """q [n, H, D] at `positions`, k, v [T, G, *]: dense softmax attention with mapped scores, one query at a time."""
    H, G = q.shape[1], k.shape[1]
    rows = []
    for i, p in enumerate(positions):
        lo = p - p % chunk if chunk else 0
        s = torch.einsum("hd,jhd->hj", q[i], k[lo:p + 1].repeat_interleave(H // G, dim=1)) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        if slopes is not None:
            s = s - slopes[:, None] * (p - torch.arange(lo, p + 1, dtype=F64))[None]
        rows.append(torch.einsum("hj,jhe->he", torch.softmax(s, -1), v[lo:p + 1].repeat_interleave(H // G, dim=1)).reshape(-1))
    return torch.stack(rows)


class Paged:
    """Keys and values of several rows in shuffled pages; slots no query may see hold NaN."""

    def __init__(self, lens, G, dk, dv, dtype, g, BS=16):
        total = sum(-(-n // BS) for n in lens)
        order = (torch.randperm(total, generator=g) + 1).tolist()
        self.k, self.v = [torch.randn(n, G, dk, generator=g).to(dtype) for n in lens], [torch.randn(n, G, dv, generator=g).to(dtype) for n in lens]
        kp, vp = torch.full((total + 1, G, BS, dk), float("nan")), torch.full((total + 1, G, BS, dv), float("nan"))
        table = torch.zeros(len(lens), max(-(-n // BS) for n in lens) + 1, dtype=torch.int32)
        for r, n in enumerate(lens):
            for b in range(-(-n // BS)):
                page = order.pop()
                table[r, b] = page
                part = slice(b * BS, min(n, (b + 1) * BS))
                kp[page, :, :part.stop - part.start] = self.k[r][part].transpose(0, 1).float()
                vp[page, :, :part.stop - part.start] = self.v[r][part].transpose(0, 1).float()
        self.k_pool, self.v_pool, self.table = kp.to(dtype).to(DEV), vp.to(dtype).to(DEV), table.to(DEV)


MAPS = [dict(cap=0.0, slopes=False, chunk=0), dict(cap=2.5, slopes=False, chunk=0), dict(cap=0.0, slopes=True, chunk=0),
        dict(cap=0.0, slopes=False, chunk=20), dict(cap=4.0, slopes=True, chunk=48), dict(cap=1.5, slopes=True, chunk=7),
        dict(cap=30.0, slopes=True, chunk=100), dict(cap=60.0, slopes=True, chunk=48)]


def case(H, G, dk, dv, dtype, m, seed):
    """Three rows of 150, 64 and 37 keys; a scale that makes peaked weights; sharp scores on both sides of every edge."""
    g = torch.Generator().manual_seed(seed)
    lens = [150, 64, 37]
    pages = Paged(lens, G, dk, dv, dtype, g)
    slopes = plain.slopes(H) if m["slopes"] else None
    kw = dict(softcap=m["cap"], slopes=slopes.float().to(DEV) if slopes is not None else None, chunk=m["chunk"])
    return g, lens, pages, slopes, kw, 3.0 / dk ** 0.5


@pytest.mark.parametrize("m", MAPS, ids=str)
@pytest.mark.parametrize("shape", [(8, 2, 64, 64), (6, 1, 128, 128), (3, 3, 64, 64), (12, 1, 64, 64)])
def test_tcgen05_tiles_with_mapped_scores(shape, m):
    """Portions that start anywhere: at a chunk's edge, one before and one after it, in the middle of a page."""
    from socrates_b200.kernels import ops
    H, G, dk, dv = shape
    g, lens, pages, slopes, kw, scale = case(H, G, dk, dv, torch.bfloat16, m, 3)
    firsts = [0, 63, 20]
    q = [torch.randn(n - f, H, dk, generator=g).bfloat16() for n, f in zip(lens, firsts)]
    want = torch.cat([attend(q[r].double(), pages.k[r].double(), pages.v[r].double(), range(firsts[r], lens[r]), scale,
                             m["cap"], slopes, m["chunk"]) for r in range(3)])
    counts = [n - f for n, f in zip(lens, firsts)]
    starts = [0, counts[0], counts[0] + counts[1], sum(counts)]
    out = torch.empty(sum(counts), H * dv, dtype=torch.bfloat16, device=DEV)
    status = i32([0])
    ops.attention_prefill_tcgen05(out, torch.cat(q).reshape(-1, H * dk).to(DEV), pages.k_pool, pages.v_pool, pages.table,
                                  i32(starts), i32([0, 1, 2]), i32(firsts), H, scale, status, **kw)
    assert int(status.item()) == 0 and err(out.double().cpu(), want) < 8e-3


@pytest.mark.parametrize("m", MAPS, ids=str)
@pytest.mark.parametrize("shape", [(8, 2, 64, 64), (4, 4, 128, 128), (12, 1, 32, 32), (16, 1, 128, 128), (5, 5, 16, 16)])
@pytest.mark.parametrize("parts", [1, 3, 6])
def test_decode_on_tensor_cores_with_mapped_scores(shape, m, parts):
    from socrates_b200.kernels import ops
    H, G, dk, dv = shape
    g, lens, pages, slopes, kw, scale = case(H, G, dk, dv, torch.bfloat16, m, 4)
    where = [(0, p) for p in (0, 6, 7, 19, 20, 47, 48, 99, 100, 149)] + [(1, 63), (2, 36), (2, 15), (2, 16)]
    q = torch.randn(len(where), H, dk, generator=g).bfloat16()
    want = torch.cat([attend(q[i:i + 1].double(), pages.k[r].double(), pages.v[r].double(), [p], scale, m["cap"], slopes, m["chunk"])
                      for i, (r, p) in enumerate(where)])
    N = len(where)
    out = torch.empty(N, H * dv, dtype=torch.bfloat16, device=DEV)
    po, pm = torch.empty(N * H * parts * dv, device=DEV), torch.empty(N * H * parts * 2, device=DEV)
    ops.attention_decode_mma(out, q.reshape(N, -1).to(DEV), pages.k_pool, pages.v_pool, pages.table, i32([r for r, _ in where]),
                             i32([p for _, p in where]), H, scale, 0, parts, po, pm, **kw)
    assert err(out.double().cpu(), want) < 8e-3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", MAPS, ids=str)
@pytest.mark.parametrize("shape", [(8, 2, 24, 40), (3, 3, 6, 5), (10, 1, 128, 64)])
def test_cuda_core_attention_with_mapped_scores(shape, m, dtype):
    from socrates_b200.kernels import ops
    H, G, dk, dv = shape
    g, lens, pages, slopes, kw, scale = case(H, G, dk, dv, dtype, m, 5)
    tol = 2e-5 if dtype == torch.float32 else 6e-3
    firsts = [0, 50, 19]
    counts = [n - f for n, f in zip(lens, firsts)]
    q = [torch.randn(c, H, dk, generator=g).to(dtype) for c in counts]
    want = torch.cat([attend(q[r].double(), pages.k[r].double(), pages.v[r].double(), range(firsts[r], lens[r]), scale,
                             m["cap"], slopes, m["chunk"]) for r in range(3)])
    N = sum(counts)
    starts = [0, counts[0], counts[0] + counts[1], N]
    qd, out = torch.cat(q).reshape(N, -1).to(DEV), torch.empty(N, H * dv, dtype=dtype, device=DEV)
    rows = i32([r for r in range(3) for _ in range(counts[r])])
    pos = i32([p for r in range(3) for p in range(firsts[r], lens[r])])
    for parts in (1, 4):
        po, pm = torch.empty(N * H * parts * dv, device=DEV), torch.empty(N * H * parts * 2, device=DEV)
        out.zero_()
        ops.attention_bias(out, qd, pages.k_pool, pages.v_pool, pages.table, rows, pos, H, scale, num_partitions=parts,
                           part_o=po, part_ml=pm, **kw)
        assert err(out.double().cpu(), want) < tol, parts
    if ops.attention_bias_tile_supports(H, G, dk, dv, dtype):
        out.zero_()
        ops.attention_bias_tile(out, qd, pages.k_pool, pages.v_pool, pages.table, i32(starts), i32([0, 1, 2]), i32(firsts), H,
                                scale, **kw)
        assert err(out.double().cpu(), want) < tol


@pytest.mark.parametrize("cap", [50.0, 55.0, 70.0])
@pytest.mark.parametrize("sign", [-1.0, 1.0])
def test_scores_at_the_cap(cap, sign):
    """Every key of a row at minus the cap, or at plus the cap, but for one key a little off it: weights that take the
    running maximum's place must neither vanish nor overflow."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(1)
    n, H, D = 150, 2, 64
    pages = Paged([n], 1, D, D, torch.bfloat16, g)
    u = torch.ones(D)
    k = (u[None] * 4.0 * (1 + 0.2 * torch.rand(n, 1, generator=g))).bfloat16()
    k[20] = (u * sign * -1.0).bfloat16()                # this one alone is far from the rest for its queries
    pages.k[0] = k[:, None]
    for p in range(n):
        pages.k_pool[int(pages.table[0, p // 16]), 0, p % 16] = k[p].to(DEV)
    q = (sign * u[None, None] * torch.linspace(2.0, 4.0, n)[:, None, None]).repeat(1, H, 1).bfloat16()
    slopes = torch.tensor([0.0, 0.3], dtype=F64)
    want = attend(q.double(), pages.k[0].double(), pages.v[0].double(), range(n), 0.4, cap, slopes, 0)
    out, status = torch.empty(n, H * D, dtype=torch.bfloat16, device=DEV), i32([0])
    ops.attention_prefill_tcgen05(out, q.reshape(n, -1).to(DEV), pages.k_pool, pages.v_pool, pages.table, i32([0, n]), i32([0]),
                                  i32([0]), H, 0.4, status, softcap=cap, slopes=slopes.float().to(DEV))
    assert int(status.item()) == 0 and err(out.double().cpu(), want) < 8e-3


def test_far_keys_keep_an_exact_slope():
    """At position 20,000 the slope times the distance is still exact for near keys: equal scores but for the slope."""
    from socrates_b200.kernels import ops
    H, D, BS, n = 2, 64, 64, 20000
    k = torch.zeros(n // BS + 2, 1, BS, D, dtype=torch.bfloat16, device=DEV)
    v = torch.randn(k.shape, generator=torch.Generator().manual_seed(1)).bfloat16().to(DEV)
    table = torch.arange(1, n // BS + 2, dtype=torch.int32, device=DEV)[None].contiguous()
    q = torch.ones(3, H * D, dtype=torch.bfloat16, device=DEV)
    slopes = torch.tensor([0.5, 0.04], device=DEV)
    pos = [n - 1, n - 2, n - 3]
    vals = v[1:].reshape(-1, D)[:n].double().cpu()
    want = []
    for p in pos:
        for s in (0.5, 0.04):
            a = torch.softmax(-s * (p - torch.arange(p + 1, dtype=F64)), 0)
            want.append(a @ vals[:p + 1])
    want = torch.stack(want).view(3, -1)
    out = torch.empty(3, H * D, dtype=torch.bfloat16, device=DEV)
    po, pm = torch.empty(3 * H * 4 * D, device=DEV), torch.empty(3 * H * 8, device=DEV)
    ops.attention_decode_mma(out, q, k, v, table, i32([0, 0, 0]), i32(pos), H, 0.1, 0, 4, po, pm, slopes=slopes)
    assert err(out.double().cpu(), want) < 6e-3
    status = i32([0])
    ops.attention_prefill_tcgen05(out, q, k, v, table, i32([0, 3]), i32([0]), i32([n - 3]), H, 0.1, status, slopes=slopes)
    assert int(status.item()) == 0 and err(out.double().cpu(), want[[2, 1, 0]]) < 6e-3


# ------------------------------------------------------------------------------------------ q, k, v on their way in
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(4, 2, 24, 16, 12), (3, 3, 6, 5, 6), (8, 2, 128, 128, 64), (4, 1, 64, 64, 64), (2, 2, 64, 64, 0),
                                   (6, 2, 128, 128, 48), (2, 1, 256, 256, 96), (4, 4, 128, 64, 128)])
@pytest.mark.parametrize("n", [5, 700])
def test_unit_norm_rotation_bias_and_shared_values(dtype, shape, n):
    """Five tokens take the kernels of a decode step, 700 those of a prompt.  Whole rows and partial sums; with and
    without a bias; the layer that keeps its values and one that blends them."""
    from socrates_b200.kernels import ops
    H, G, D, E, R = shape
    g = torch.Generator().manual_seed(D + n)
    width, BS, eps = H * D + G * (D + E), 16, 1e-5
    x, bias = torch.randn(n, width, generator=g).to(dtype), torch.randn(width, generator=g)
    first = torch.randn(n, G * E, generator=g)
    pages = -(-n // BS)
    table = (torch.randperm(pages, generator=g) + 1).to(torch.int32)[None].to(DEV)
    positions = torch.arange(n)
    rot = {"dims": R, "base": 100.0} if R else None
    inv_freq = (plain.frequencies(rot) if R else torch.zeros(1)).float().to(DEV)
    parts = torch.randn(3, n, width, generator=g)
    parts[2] = x.float() - parts[0] - parts[1]
    tol = (3e-5 if n < 100 else 1e-4) if dtype == torch.float32 else 8e-3       # float32 angles: position * 2^-24
    for source in (x.to(DEV), parts.to(DEV)):
        for b in (None, bias):
            y = x.double() + (b.double() if b is not None else 0.0)
            q, k, v = y[:, :H * D].view(n, H, D), y[:, H * D:(H + G) * D].view(n, G, D), y[:, (H + G) * D:].view(n, G, E)
            want_q, want_k = (plain.unit(plain.rotate_halves(t, positions, rot), eps) for t in (q, k))
            for mode in (None, "keep", "blend"):
                qo = torch.empty(n, H * D, dtype=dtype, device=DEV)
                kp = torch.zeros(pages + 1, G, BS, D, dtype=dtype, device=DEV)
                vp = torch.zeros(pages + 1, G, BS, E, dtype=dtype, device=DEV)
                vf = first.to(DEV)
                ops.qk_norm_rope_kvwrite(source, qo, kp, vp, None, None, inv_freq, R, positions.to(torch.int32).to(DEV),
                                         torch.zeros(n, dtype=torch.int32, device=DEV), table, eps, H, G, D, value_dim=E,
                                         bias=b.to(DEV) if b is not None else None, unit_norm=True, values=mode, blend=0.3,
                                         v_first=vf)
                assert err(qo.double().cpu().view(n, H, D), want_q) < tol, mode
                got_k = kp[table[0].long()].transpose(1, 2).reshape(-1, G, D)[:n].double().cpu()
                got_v = vp[table[0].long()].transpose(1, 2).reshape(-1, G, E)[:n].double().cpu()
                assert err(got_k, want_k) < tol, mode
                want_v = 0.7 * v + 0.3 * first.double().view(n, G, E) if mode == "blend" else v
                assert err(got_v, want_v) < tol, mode
                assert err(vf.double().cpu().view(n, G, E), v if mode == "keep" else first.double().view(n, G, E)) < (1e-5 if mode != "keep" else tol)


# ------------------------------------------------------------------------------------------ the norm after the sum
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,parts", [(37, 1), (40, 3), (1024, 14), (2048, 2)])
def test_norm_after_the_scaled_sum(dtype, d, parts):
    """The normed row becomes the float32 residual and, where asked, its rounding; a bias on the branch; no branch."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(d)
    N, eps, alpha = 9, 1e-5, 1.7
    x, delta = torch.randn(N, d, generator=g) * 2, torch.randn(parts, N, d, generator=g)
    gain, bias = torch.randn(d, generator=g), torch.randn(d, generator=g)
    for b in (None, bias):
        total = alpha * x.double() + delta.double().sum(0) + (b.double() if b is not None else 0.0)
        want = plain.unit(total, eps) * gain.double()
        for out in (None, torch.empty(N, d, dtype=dtype, device=DEV)):
            res = x.to(DEV)
            ops.fold_rmsnorm(res, delta.to(DEV), gain.to(DEV), out, eps, branch_bias=b.to(DEV) if b is not None else None,
                             res_scale=alpha, norm_residual=True)
            assert err(res.double().cpu(), want) < 1e-5
            if out is not None:
                assert torch.equal(out, res.to(dtype))
    res = x.to(DEV)
    ops.fold_rmsnorm(res, None, gain.to(DEV), None, eps, res_scale=alpha, norm_residual=True)
    assert err(res.double().cpu(), plain.unit(alpha * x.double(), eps) * gain.double()) < 1e-5


# ------------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("K,E,top,count,keep", [(40, 6, 2, 3, 2), (37, 5, 2, 1, 1), (1024, 64, 6, 8, 3), (64, 12, 4, 6, 2), (33, 4, 3, 4, 3),
                                                (128, 160, 8, 4, 1), (64, 9, 9, 3, 3)])
@pytest.mark.parametrize("n", [3, 600])
def test_sigmoid_routing_in_groups(dtype, K, E, top, count, keep, n):
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(K + E)
    x, router = torch.randn(n, K, generator=g).to(dtype), torch.randn(E, K, generator=g) / K ** 0.5
    w = torch.full((n, E), float("nan"), device=DEV)
    ids, picked = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
    ops.moe_router(x.to(DEV), router.to(DEV), None, w, ids, picked, top, sigmoid=True, groups=count, keep=keep, scale=1.6)
    z = x.double() @ router.double().T
    cfg = {"experts": E, "top": top, "scale": 1.6, "groups": {"count": count, "keep": keep}}
    close = 0
    for t in range(n):
        want_ids, share = plain.choose(z[t], cfg)
        if ids[t].tolist() != want_ids:
            close += 1                                      # a tie that float32 turns; never more than a few
            continue
        want = torch.zeros(E, dtype=F64)
        want[want_ids] = share
        assert err(w[t].double().cpu(), want) < 1e-5 and err(picked[t].double().cpu(), share) < 1e-5
    assert close <= n // 100
    assert torch.allclose(w.sum(-1).cpu(), torch.full((n,), 1.6), atol=1e-4)


def test_a_group_counts_with_its_two_largest():
    """One expert far ahead in a group of weak ones loses to a group of two good ones; groups of one expert count alone."""
    from socrates_b200.kernels import ops
    def run(z, top, count, keep):
        E = len(z)
        w, ids, picked = torch.empty(1, E, device=DEV), torch.empty(1, top, dtype=torch.int32, device=DEV), torch.empty(1, top, device=DEV)
        ops.moe_router(torch.ones(1, 4, device=DEV), (torch.tensor(z)[:, None] / 4).repeat(1, 4).to(DEV), None, w, ids, picked,
                       top, sigmoid=True, groups=count, keep=keep)
        return ids[0].tolist()
    assert run([3.0, -4.0, -4.0, 1.0, 1.5, -4.0], 2, 2, 1) == [4, 3]
    assert run([3.0, -4.0, -4.0, 1.0, 1.5, -4.0], 3, 2, 2) == [0, 4, 3]
    assert run([0.5, -1.0, 2.0, 1.0], 2, 4, 2) == [2, 3]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,F,n", [(5, 10, 7), (6, 24, 40), (16, 128, 300)])
def test_units_without_a_gate(dtype, E, F, n):
    """relu squared times the weight; what an unchosen expert would read is NaN."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(F)
    x = torch.randn(n, E * F, generator=g).to(dtype)
    w = torch.rand(n, E, generator=g) * (torch.rand(n, E, generator=g) < 0.4)
    want = (torch.clamp(x.double(), min=0.0) ** 2).view(n, E, F) * w.double()[:, :, None]
    dirty = x.clone().view(n, E, F)
    dirty[w == 0] = float("nan")
    parts = torch.randn(3, n, E * F, generator=g)
    parts[2] = x.float() - parts[0] - parts[1]
    for source in (dirty.view(n, -1).to(DEV), parts.to(DEV)):
        out = torch.empty(n, E * F, dtype=dtype, device=DEV)
        ops.moe_act(out, source, w.to(DEV), E, F)
        assert err(out.double().cpu().view(n, E, F), want) < (2e-5 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("interleaved", [False, True])
def test_gelu_gate_kernel(dtype, interleaved):
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(2)
    for n, F in ((3, 10), (40, 64)):
        gate, up = (torch.randn(n, F, generator=g).to(dtype) * 3 for _ in range(2))
        want = plain.gelu_tanh(gate.double()) * up.double()
        x = (torch.stack([gate, up], -1).reshape(n, -1) if interleaved else torch.cat([gate, up], -1)).to(DEV)
        out = torch.empty(n, F, dtype=dtype, device=DEV)
        ops.silu_mul(out, x, interleaved=interleaved, act="gelu_tanh")
        assert err(out.double().cpu(), want) < (1e-5 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("M,variant", [(1, 0), (20, 0), (64, 0), (65, 0), (300, 128), (300, 160), (300, 256), (600, 1256), (2100, 0)])
def test_gelu_in_the_products_epilogue(M, variant):
    """Every kernel that carries a gated epilogue: weight streaming with 16, 32 and 64 columns, the persistent kernel
    in its widths, the pair kernel."""
    from socrates_b200.kernels import ops
    g = torch.Generator().manual_seed(M)
    K, F = 136, 168
    x = torch.randn(M, K, generator=g).bfloat16()
    gate, up = ((torch.randn(F, K, generator=g) / K ** 0.5 * 2).bfloat16() for _ in range(2))
    w = torch.stack([gate, up], 1).reshape(2 * F, K).contiguous().to(DEV)
    want = plain.gelu_tanh(x.double() @ gate.double().T) * (x.double() @ up.double().T)
    status = i32([0])
    for dtype in (torch.bfloat16, torch.float32):
        out = torch.empty(M, F, dtype=dtype, device=DEV)
        ops.gemm_tcgen05(out, x.to(DEV), w, status, 1, variant=variant, epilogue=2)
        assert int(status.item()) == 0 and err(out.double().cpu(), want) < (5e-3 if dtype == torch.bfloat16 else 1e-5)
        ops.gemm_tcgen05(out, x.to(DEV), w, status, 1, variant=variant, epilogue=1)          # silu is still silu
        assert err(out.double().cpu(), plain.silu(x.double() @ gate.double().T) * (x.double() @ up.double().T)) < (5e-3 if dtype == torch.bfloat16 else 1e-5)
