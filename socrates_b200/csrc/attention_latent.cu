// Paged causal attention of many query heads over ONE cached head whose rows are keys and values at once
// (bfloat16): the row of a token is [turning part (dr) | latent (rank)], the whole row is its key and the latent its
// value.  Both products run on mma.sync (m16n8k16, float32 accumulation):
//
//   s = (q . row) * scale ,  softmax over the visible rows (float32) ,  o = sum_j p_j latent_j
//   every softmax weight enters the value product as two bfloat16 terms (high and low): 2^-17 of it is lost
//   o may be multiplied by sigmoid(gate), one gate per head
//
// A block of four warps serves up to 16 * MT rows = (token, head) pairs: the heads of one decoded token, or of a few
// consecutive tokens of a prompt portion.  A tile of 64 cached rows is brought into shared memory once (cp.async, the
// next tile on its way meanwhile) and used by both products: warp w makes the scores of keys 16 w .. 16 w + 15 for all
// rows, the block agrees on the rows' maxima, and warp w then adds the weighted latents of every fourth group of eight
// value dims.  For decoding the visible keys of a token are cut into shares (grid.z), merged by the kernel the other
// attention kernels use.
#include <math.h>

#include "attention_mma.cuh"
#include "attention_reduce.cuh"

using namespace sb;

namespace {

struct LatentAttnArgs {
    bf16* out;                 // [N, H*rank]
    const bf16* q;             // [N, H*D]
    const bf16* pool;          // [pages, 1, BS, D]
    const int* table;
    int table_width;
    const int* token_rows;     // QT == 1: a tile is one token of the step
    const int* positions;
    const int* seq_starts;     // QT > 1: a tile is QT consecutive tokens of a request
    const int* seq_rows;
    const int* seq_first_pos;
    const bf16* gate;          // [N, gate_stride], head h at column h; or null
    long long gate_stride;
    float* part_o;             // [N, H, NP, rank]
    float* part_ml;            // [N, H, NP, 2]
    int R, N, H, D, dr, rank, BS, window, QT, HG, NP;
    float scale_log2;          // scale * log2(e)
};

constexpr int PLD = KT + 8;    // row stride of the weight tiles

__device__ __forceinline__ float head_gate(const LatentAttnArgs& a, int n, int h) {
    if (a.gate == nullptr) return 1.f;
    return 1.0f / (1.0f + expf(-__bfloat162float(a.gate[(size_t)n * a.gate_stride + h])));
}

template <int MT, int NT>
__global__ void __launch_bounds__(THREADS) latent_attention_kernel(LatentAttnArgs a) {
    sb::pdl_launch_dependents();
    constexpr int ROWS = 16 * MT;
    extern __shared__ __align__(16) unsigned char lsm[];
    const int D = a.D, Dp = (D + 15) & ~15, LD = Dp + 8, rank = a.rank, BS = a.BS;
    bf16* Qs = reinterpret_cast<bf16*>(lsm);             // [ROWS][LD]
    bf16* Ks = Qs + ROWS * LD;                           // [2][KT][LD]
    bf16* Ph = Ks + 2 * KT * LD;                         // [ROWS][PLD] high terms of the weights
    bf16* Pl = Ph + ROWS * PLD;                          // low terms
    float* red = reinterpret_cast<float*>(Pl + ROWS * PLD);     // [4][ROWS]
    int* pages = reinterpret_cast<int*>(red + 4 * ROWS);        // the pages of this block's keys
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    sb::pdl_wait();
    // ---- which rows: tokens n0 .. n0 + nq - 1 of cache row `row`, heads h0 .. h0 + hn - 1
    int n0, nq, row, pos0;
    if (a.QT == 1) {
        n0 = blockIdx.y;
        nq = 1;
        row = a.token_rows[n0];
        pos0 = a.positions[n0];
    } else {
        int r = 0, ti = gridDim.y - 1 - blockIdx.y;      // late tiles see more keys: they start first
        for (; r < a.R; ++r) {
            const int nt = (a.seq_starts[r + 1] - a.seq_starts[r] + a.QT - 1) / a.QT;
            if (ti < nt) break;
            ti -= nt;
        }
        if (r == a.R) return;
        n0 = a.seq_starts[r] + ti * a.QT;
        nq = min(a.QT, a.seq_starts[r + 1] - n0);
        row = a.seq_rows[r];
        pos0 = a.seq_first_pos[r] + ti * a.QT;
    }
    const int h0 = blockIdx.x * a.HG, hn = min(a.HG, a.H - h0), live = nq * a.HG;
    const int pos_last = pos0 + nq - 1;
    const int lo_all = (a.window > 0 && pos0 + 1 > a.window) ? pos0 + 1 - a.window : 0;
    const int per = (pos_last + 1 - lo_all + a.NP - 1) / a.NP;
    const int lo = lo_all + (int)blockIdx.z * per, hi = min(pos_last + 1, lo + per);     // this share: lo .. hi - 1
    const int* table = a.table + (size_t)row * a.table_width;
    const int first_page = lo / BS;
    if (lo < hi)
        for (int i = tid; i <= (hi - 1) / BS - first_page; i += THREADS) pages[i] = table[first_page + i];
    // ---- the queries; rows past the tile's and columns past D are zero
    for (int i = tid; i < ROWS * (LD / 8); i += THREADS) {
        const int rr = i / (LD / 8), c = (i - rr * (LD / 8)) * 8, qi = rr / a.HG, g = rr - qi * a.HG;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (rr < live && g < hn && c < D) v = *reinterpret_cast<const uint4*>(a.q + ((size_t)(n0 + qi) * a.H + h0 + g) * D + c);
        *reinterpret_cast<uint4*>(Qs + rr * LD + c) = v;
    }
    __syncthreads();
    // lanes that share a cached row while it is copied: the power of two that covers its 16-byte pieces
    const int CH = Dp / 8, cw = CH <= 4 ? 4 : CH <= 8 ? 8 : CH <= 16 ? 16 : 32;
    const int krow = warp * (32 / cw) + lane / cw, kstep = 4 * (32 / cw), kc = lane % cw;
    auto load_tile = [&](int stage, int k0) {
        bf16* dst = Ks + stage * KT * LD;
        for (int key = krow; key < KT; key += kstep) {
            const int pos = k0 + key;
            const bool have = pos < hi;
            const bf16* src = a.pool;
            if (have) src = a.pool + ((size_t)pages[pos / BS - first_page] * BS + pos % BS) * D;
            for (int c = kc; c < CH; c += cw) {
                const bool in = have && c * 8 < D;
                cp_async16(smem_u32(dst + key * LD + c * 8), in ? src + c * 8 : a.pool, in ? 16 : 0);
            }
        }
        cp_async_commit();
    };
    float m[MT][2], l[MT][2], o[MT][NT][4];
#pragma unroll
    for (int t = 0; t < MT; ++t) {
        m[t][0] = m[t][1] = -INFINITY;
        l[t][0] = l[t][1] = 0.f;
#pragma unroll
        for (int j = 0; j < NT; ++j) o[t][j][0] = o[t][j][1] = o[t][j][2] = o[t][j][3] = 0.f;
    }
    const int tiles = lo < hi ? (hi - lo + KT - 1) / KT : 0;
    if (tiles > 0) load_tile(0, lo);
    for (int it = 0; it < tiles; ++it) {
        const int k0 = lo + it * KT;
        const bf16* K = Ks + (it & 1) * KT * LD;
        cp_async_wait<0>();
        __syncthreads();                                 // the tile is here; nobody reads the other stage any more
        if (it + 1 < tiles) load_tile((it + 1) & 1, k0 + KT);
        // ---- scores of this warp's 16 keys
        float s[MT][2][4];
#pragma unroll
        for (int t = 0; t < MT; ++t)
#pragma unroll
            for (int j = 0; j < 2; ++j) s[t][j][0] = s[t][j][1] = s[t][j][2] = s[t][j][3] = 0.f;
        const uint32_t kaddr = smem_u32(K + (warp * 16 + (lane & 7) + ((lane >> 4) << 3)) * LD + ((lane >> 3) & 1) * 8);
        const uint32_t qaddr = smem_u32(Qs + (lane & 15) * LD + (lane >> 4) * 8);
#pragma unroll 2
        for (int d = 0; d < Dp; d += 16) {
            uint32_t b[4];
            ldmatrix_x4(b, kaddr + d * 2);
#pragma unroll
            for (int t = 0; t < MT; ++t) {
                uint32_t q[4];
                ldmatrix_x4(q, qaddr + (t * 16 * LD + d) * 2);
                mma_bf16(s[t][0], q, b[0], b[1]);
                mma_bf16(s[t][1], q, b[2], b[3]);
            }
        }
        // ---- scale, mask, the rows' maxima over this warp's keys
#pragma unroll
        for (int t = 0; t < MT; ++t)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int rr = t * 16 + (lane >> 2) + 8 * e, qi = rr / a.HG, pos = pos0 + qi;
                const int low = (a.window > 0 && pos + 1 > a.window) ? pos + 1 - a.window : 0;
                const int high = min(hi, rr < live ? pos + 1 : 0);
                float mx = -INFINITY;
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        const int key = k0 + warp * 16 + j * 8 + (lane & 3) * 2 + c;
                        float& x = s[t][j][2 * e + c];
                        x = (key >= low && key < high) ? x * a.scale_log2 : -INFINITY;
                        mx = fmaxf(mx, x);
                    }
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                if ((lane & 3) == 0) red[warp * ROWS + rr] = mx;
            }
        __syncthreads();
        // ---- weights in two terms, and the factors of what was summed before
#pragma unroll
        for (int t = 0; t < MT; ++t)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int rr = t * 16 + (lane >> 2) + 8 * e;
                const float mx = fmaxf(fmaxf(red[rr], red[ROWS + rr]), fmaxf(red[2 * ROWS + rr], red[3 * ROWS + rr]));
                const float m_new = fmaxf(m[t][e], mx), base = m_new == -INFINITY ? 0.f : m_new;
                const float f = ex2_approx(m[t][e] - base);
                m[t][e] = m_new;
                float sum = 0.f;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const float p0 = ex2_approx(s[t][j][2 * e] - base), p1 = ex2_approx(s[t][j][2 * e + 1] - base);
                    sum += p0 + p1;
                    const float g0 = __bfloat162float(__float2bfloat16_rn(p0)), g1 = __bfloat162float(__float2bfloat16_rn(p1));
                    const int at = rr * PLD + warp * 16 + j * 8 + (lane & 3) * 2;
                    *reinterpret_cast<uint32_t*>(Ph + at) = pack_bf16(g0, g1);
                    *reinterpret_cast<uint32_t*>(Pl + at) = pack_bf16(p0 - g0, p1 - g1);
                }
                l[t][e] = l[t][e] * f + sum;
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    o[t][j][2 * e] *= f;
                    o[t][j][2 * e + 1] *= f;
                }
            }
        __syncthreads();
        // ---- the weighted latents: this warp's value dims, all 64 keys
        const uint32_t paddr = ((lane & 15) * PLD + (lane >> 4) * 8) * 2;
        const uint32_t ph = smem_u32(Ph) + paddr, pl = smem_u32(Pl) + paddr;
        const uint32_t vaddr = smem_u32(K + lane * LD + a.dr);
#pragma unroll
        for (int kk = 0; kk < KT; kk += 32) {
            uint32_t b[NT][4];
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const int dim = (warp + 4 * j) * 8;
                if (dim < rank) ldmatrix_x4_trans(b[j], vaddr + (kk * LD + dim) * 2);
            }
#pragma unroll
            for (int t = 0; t < MT; ++t)
#pragma unroll
                for (int k2 = 0; k2 < 2; ++k2) {
                    uint32_t w[4], w2[4];
                    ldmatrix_x4(w, ph + (t * 16 * PLD + kk + k2 * 16) * 2);
                    ldmatrix_x4(w2, pl + (t * 16 * PLD + kk + k2 * 16) * 2);
#pragma unroll
                    for (int j = 0; j < NT; ++j)
                        if ((warp + 4 * j) * 8 < rank) {
                            mma_bf16(o[t][j], w, b[j][2 * k2], b[j][2 * k2 + 1]);
                            mma_bf16(o[t][j], w2, b[j][2 * k2], b[j][2 * k2 + 1]);
                        }
                }
        }
    }
    // ---- the rows' sums over all warps' keys
    __syncthreads();
#pragma unroll
    for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float x = l[t][e];
            x += __shfl_xor_sync(0xffffffffu, x, 1);
            x += __shfl_xor_sync(0xffffffffu, x, 2);
            if ((lane & 3) == 0) red[warp * ROWS + t * 16 + (lane >> 2) + 8 * e] = x;
        }
    __syncthreads();
#pragma unroll
    for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int rr = t * 16 + (lane >> 2) + 8 * e, qi = rr / a.HG, g = rr - qi * a.HG;
            if (rr >= live || g >= hn) continue;
            const int n = n0 + qi, h = h0 + g;
            const float sum = (red[rr] + red[ROWS + rr]) + (red[2 * ROWS + rr] + red[3 * ROWS + rr]);
            const float gate = head_gate(a, n, h);
            if (a.NP == 1) {
                const float f = gate / sum;
                bf16* y = a.out + ((size_t)n * a.H + h) * rank;
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    const int dim = (warp + 4 * j) * 8 + (lane & 3) * 2;
                    if (dim < rank) *reinterpret_cast<uint32_t*>(y + dim) = pack_bf16(o[t][j][2 * e] * f, o[t][j][2 * e + 1] * f);
                }
            } else {                                     // the gate scales the output, so it may scale every share
                const size_t slot = ((size_t)n * a.H + h) * a.NP + blockIdx.z;
                float* y = a.part_o + slot * rank;
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    const int dim = (warp + 4 * j) * 8 + (lane & 3) * 2;
                    if (dim < rank) *reinterpret_cast<float2*>(y + dim) = make_float2(o[t][j][2 * e] * gate, o[t][j][2 * e + 1] * gate);
                }
                if (warp == 0 && (lane & 3) == 0) {      // an empty share has sum 0 and is skipped by the merge
                    a.part_ml[slot * 2] = m[t][e] * 0.6931471805599453f;
                    a.part_ml[slot * 2 + 1] = sum;
                }
            }
        }
}

size_t smem_bytes(int MT, int D, int pages) {
    const size_t LD = ((D + 15) & ~15) + 8;
    return (16 * MT * LD + 2 * KT * LD + 2 * 16 * MT * PLD) * sizeof(bf16) + 4 * 16 * MT * sizeof(float) + (size_t)pages * sizeof(int);
}

constexpr size_t SMEM_MAX = 220 * 1024;

template <int MT, int NT>
void launch_latent(const LatentAttnArgs& a, dim3 grid, size_t smem, cudaStream_t stream) {
    static sb::OncePerDevice once;
    if (!once.flag()) {
        cudaFuncSetAttribute(latent_attention_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_MAX);
        once.flag() = true;
    }
    sb::launch(latent_attention_kernel<MT, NT>, grid, dim3(THREADS), smem, stream, a);
}

}  // namespace

// Row tiles (of 16 rows) a block may hold for a latent of `rank` dims: what the accumulators leave room for.
static int most_row_tiles(int rank) { return rank <= 128 ? 4 : rank <= 256 ? 2 : 1; }

extern "C" int sb_attention_latent_supports(int H, int D, int rank) {
    return H >= 1 && D % 8 == 0 && rank % 8 == 0 && (D - rank) % 8 == 0 && rank >= 8 && rank <= 512 && D >= rank && D <= 640;
}

// prompt = 0: every token a tile of its own, its keys in NP shares.  prompt = 1: tiles of consecutive tokens, NP = 1.
extern "C" int sb_attention_latent(void* out, const void* q, const void* pool, const int* table, int table_width,
                                   const int* token_rows, const int* positions, const int* seq_starts, const int* seq_rows,
                                   const int* seq_first_pos, int R, const void* gate, long long gate_stride, int N, int H,
                                   int D, int rank, int BS, int window, float scale, int prompt, int NP, float* part_o,
                                   float* part_ml, cudaStream_t stream) {
    SB_REQUIRE(sb_attention_latent_supports(H, D, rank), "attention_latent: rows of %d dims with a latent of %d (multiples of 8, up to 640 and 512)", D, rank);
    SB_REQUIRE(N >= 0 && N <= 65535 && R >= 0 && BS > 0 && table_width > 0 && window >= 0, "attention_latent: bad sizes N=%d BS=%d", N, BS);
    SB_REQUIRE(NP >= 1 && NP <= 65535 && (NP == 1 || (part_o != nullptr && part_ml != nullptr && !prompt)),
               "attention_latent: %d shares need scratch and single tokens", NP);
    SB_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(pool)) & 15) == 0 &&
                   ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(part_o)) & 7) == 0,
               "attention_latent: q and the pool must start on 16-byte boundaries");
    if (N == 0 || R == 0) return 0;
    LatentAttnArgs a;
    a.out = (bf16*)out; a.q = (const bf16*)q; a.pool = (const bf16*)pool; a.table = table; a.table_width = table_width;
    a.token_rows = token_rows; a.positions = positions; a.seq_starts = seq_starts; a.seq_rows = seq_rows;
    a.seq_first_pos = seq_first_pos; a.gate = (const bf16*)gate; a.gate_stride = gate_stride; a.part_o = part_o;
    a.part_ml = part_ml; a.R = R; a.N = N; a.H = H; a.D = D; a.dr = D - rank; a.rank = rank; a.BS = BS; a.window = window;
    a.NP = NP; a.scale_log2 = scale * LOG2E;
    int MT = most_row_tiles(rank);
    if (!prompt) while (MT > 1 && 16 * (MT / 2) >= H) MT /= 2;
    while (MT > 1 && smem_bytes(MT, D, table_width) > SMEM_MAX) MT /= 2;
    const size_t smem = smem_bytes(MT, D, table_width);
    SB_REQUIRE(smem <= SMEM_MAX, "attention_latent: rows of %d dims and a table of %d pages do not fit shared memory", D, table_width);
    a.HG = H < 16 * MT ? H : 16 * MT;
    a.QT = prompt ? (16 * MT) / a.HG : 1;
    const dim3 grid((H + a.HG - 1) / a.HG, a.QT == 1 ? N : N / a.QT + R, NP);
    SB_REQUIRE(grid.y <= 65535, "attention_latent: %d tokens exceed one launch", N);
    const int NT = rank <= 64 ? 2 : rank <= 128 ? 4 : rank <= 256 ? 8 : 16;
#define SB_LATENT(M_, N_) if (MT == M_ && NT == N_) launch_latent<M_, N_>(a, grid, smem, stream)
    SB_LATENT(1, 2); SB_LATENT(2, 2); SB_LATENT(4, 2); SB_LATENT(1, 4); SB_LATENT(2, 4); SB_LATENT(4, 4);
    SB_LATENT(1, 8); SB_LATENT(2, 8); SB_LATENT(1, 16);
#undef SB_LATENT
    if (NP > 1) {
        const int threads = rank >= 128 ? 128 : ((rank + 31) / 32) * 32;
        sb::launch(sb::attn_reduce_kernel<bf16>, dim3(H, N), dim3(threads), 0, stream, (bf16*)out, (const float*)part_o,
                   (const float*)part_ml, H, rank, NP);
    }
    SB_LAUNCH_CHECK();
}
