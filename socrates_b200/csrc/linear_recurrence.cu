// Recurrences with a matrix state per head, and the small steps around them.
//
//   linear_recurrence:  per head, S a [D, Dv] float32 state carried from token to token in the request's slot:
//        w_t = decay_h  (one constant per head)   or   exp(-exp(raw_t + base))  (per head and key channel)
//        S_t = diag(w_t) S_(t-1) + k_t v_t^T
//        o_t = S_t^T q_t                                        (read after the write)
//        o_t = (S_(t-1) + diag(u) k_t v_t^T)^T q_t              (with a bonus u: read before it)
//      q, k and v may pass SiLU first.  o is written as float32 rows [N, H*Dv].
//   norm_gate:          y = o / sqrt(mean(o^2) + eps) * gain * act(gate), the mean over each of `groups` equal
//      groups of columns (heads, or all heads together)
//   token_shift_mix:    m_s = x + (x' - x) mu_s with x' the request's token before (its slot's row for the first
//      token of a portion), for several mu at once
//
// All arithmetic is float32.  A matrix input is [N, stride] in T or float32 partial sums of a product cut along K.
#include <math.h>

#include "common.cuh"

using namespace sb;

namespace {

// A matrix in T, or partial sums that are added on the way in.
struct Rows {
    const void* x;
    const float* parts;
    int S;
    long long part_stride;
    long long stride;          // elements between rows
    int off;                   // first column
};

template <typename T>
__device__ __forceinline__ float read_rows(const Rows& a, int n, int c) {
    const size_t at = (size_t)n * a.stride + a.off + c;
    if (a.parts == nullptr) return to_float(((const T*)a.x)[at]);
    float v = 0.f;
    for (int s0 = 0; s0 < a.S; s0 += 8) {              // eight loads in flight, added in order
        float p[8];
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (s0 + j < a.S) p[j] = __ldg(a.parts + (size_t)(s0 + j) * a.part_stride + at);
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (s0 + j < a.S) v += p[j];
    }
    return v;
}

// Two float32 values in one register pair: the multiply-adds of two neighbouring state rows in one instruction.
using pair2 = unsigned long long;
__device__ __forceinline__ pair2 fma2(pair2 a, pair2 b, pair2 c) {
    pair2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ pair2 mul2(pair2 a, pair2 b) {
    pair2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ pair2 pack2(float x, float y) {
    pair2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
    return d;
}
__device__ __forceinline__ void unpack2(pair2 a, float& x, float& y) { asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a)); }

// A thread's RR rows of a row vector in shared memory as pairs: runs of up to four neighbouring rows (row_of), so that
// the lanes of a row group read neighbouring 16-byte pieces.
template <int RG, int RR>
__device__ __forceinline__ int row_of(int rg, int i) {
    constexpr int W = RR < 4 ? RR : 4;
    return (i / W) * (RG * W) + rg * W + i % W;
}
template <int RG, int RR>
__device__ __forceinline__ void load_pairs(pair2 (&d)[RR / 2], const float* row, int rg) {
    if constexpr (RR == 2) {
        d[0] = *reinterpret_cast<const pair2*>(row + row_of<RG, RR>(rg, 0));
    } else {
#pragma unroll
        for (int i = 0; i < RR / 2; i += 2) {
            const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(row + row_of<RG, RR>(rg, 2 * i));
            d[i] = x.x;
            d[i + 1] = x.y;
        }
    }
}

// 16 bytes of T as floats.
template <typename T>
__device__ __forceinline__ void widen(const uint4& raw, float (&f)[Vec16<T>::N]) {
#pragma unroll
    for (int e = 0; e < Vec16<T>::N; ++e) f[e] = to_float(reinterpret_cast<const T*>(&raw)[e]);
}

__device__ __forceinline__ float silu_f(float z) { return __fdividef(z, 1.0f + expf(-z)); }

struct RecArgs {
    Rows q, k, v, w;           // w: raw decays; w.x and w.parts null: the constant
    const float* decay;        // [H] constants, or null
    const float* base;         // [H*D] added to the raw decays, or null
    const float* bonus;        // [H*D] or null: read after the write
    int silu_qk, silu_v;
    int pieces;                // every input row is whole 16-byte pieces (matrices, no partial sums)
    float* state;              // [rows, H, D, Dv]
    float* out;                // [N, H*Dv]
    const int* seq_starts;
    const int* seq_rows;
    int R, H, D, Dv;
    // Long portions are cut into segments of `seg_len` tokens that run side by side (the recurrence is linear in
    // S with a diagonal decay).  Step 1 walks the segments of requests that have several from a zero state and
    // leaves their end states and the products of their decays; a scan turns those into the states BEFORE each
    // segment and leaves the request's state; step 2 walks every segment again from its true start and writes the
    // outputs.  A request with one segment is walked once, in step 2, from and to its slot.
    int seg_len;
    float* seg_state;          // [segments, H, D, Dv]
    float* seg_prod;           // [segments, H, D]
};

constexpr int THREADS = 256;

// Block g of the step's segments (request 0's, then request 1's, ...): its request, its number within the request,
// how many that request has, and where its scratch begins (segments of requests with several only).
__device__ __forceinline__ bool find_segment(int g, const int* seq_starts, int R, int seg_len, int& r, int& ci, int& nc,
                                             int& slot) {
    int multi = 0;
    for (r = 0; r < R; ++r) {
        nc = (seq_starts[r + 1] - seq_starts[r] + seg_len - 1) / seg_len;
        if (g < nc) { ci = g; slot = multi + g; return true; }
        g -= nc;
        if (nc > 1) multi += nc;
    }
    return false;
}

// Thread (row group, column group) holds RR neighbouring key rows x 4 neighbouring value columns of the state in
// registers, two rows a register pair; the RG lanes of a column group are neighbours in a warp and join their shares
// of o by shuffles.  TB tokens are staged in shared memory at a time (activations, decays and the bonus' dot product
// made there) while the raw values of the next TB are on their way into registers.
template <typename T, int RG, int RR, int STEP>
__global__ void __launch_bounds__(THREADS, 2) linear_recurrence_kernel(RecArgs a) {
    sb::pdl_launch_dependents();
    constexpr int DP = RG * RR, CG = THREADS / RG, COLS = CG * 4, TB = DP > 128 ? 8 : 16, P = RR / 2;
    constexpr int VT = Vec16<T>::N;
    constexpr int PQ = (TB * DP / VT + THREADS - 1) / THREADS, PV = (TB * COLS / VT + THREADS - 1) / THREADS;      // 16-byte
    constexpr int PW = (TB * DP / 4 + THREADS - 1) / THREADS;                                   // pieces a thread stages
    constexpr bool outputs = STEP == 2;
    __shared__ __align__(16) float qs[outputs ? TB : 1][DP], ks[TB][DP], ws[TB][DP], vs[TB][COLS], os[outputs ? TB : 1][COLS];
    __shared__ float bt[TB], us[DP], bs[DP];
    const int tid = threadIdx.x, rg = tid & (RG - 1), cg = tid / RG, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.x, c0 = blockIdx.z * COLS, D = a.D, Dv = a.Dv, H = a.H;
    const bool channel = a.w.x != nullptr || a.w.parts != nullptr, before = a.bonus != nullptr;
    for (int d = tid; d < DP; d += THREADS) {          // constants of the model: before the wait
        us[d] = (d < D && before) ? a.bonus[h * D + d] : 0.f;
        bs[d] = (d < D && a.base != nullptr) ? a.base[h * D + d] : 0.f;
    }
    const float fixed = channel ? 1.f : a.decay[h];
    sb::pdl_wait();
    int r, ci, nc, slot;
    if (!find_segment(blockIdx.y, a.seq_starts, a.R, a.seg_len, r, ci, nc, slot)) return;
    if (!outputs && nc == 1) return;
    const int t0 = a.seq_starts[r] + ci * a.seg_len, t1 = min(a.seq_starts[r + 1], t0 + a.seg_len);
    const int j0 = c0 + cg * 4;
    // where the state comes from (null: zero) and goes to (null: nowhere)
    float* slot_state = a.state + ((size_t)a.seq_rows[r] * H + h) * D * Dv;
    float* seg_state = nc > 1 ? a.seg_state + ((size_t)slot * H + h) * D * Dv : nullptr;
    const float* from = outputs ? (nc > 1 ? seg_state : slot_state) : nullptr;
    float* to = outputs ? (nc > 1 ? nullptr : slot_state) : seg_state;
    const bool vec = Dv % 4 == 0;
    pair2 S[P][4], A[P];
    {
        float x[RR][4];
#pragma unroll
        for (int i = 0; i < RR; ++i) {
#pragma unroll
            for (int c = 0; c < 4; ++c) x[i][c] = 0.f;
            const int row = row_of<RG, RR>(rg, i);
            if (from != nullptr && row < D) {
                const float* p = from + (size_t)row * Dv + j0;
                if (vec) {
                    if (j0 < Dv) {
                        const float4 y = *reinterpret_cast<const float4*>(p);
                        x[i][0] = y.x; x[i][1] = y.y; x[i][2] = y.z; x[i][3] = y.w;
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < 4; ++c)
                        if (j0 + c < Dv) x[i][c] = p[c];
                }
            }
        }
#pragma unroll
        for (int i = 0; i < P; ++i) {
            A[i] = pack2(1.f, 1.f);
#pragma unroll
            for (int c = 0; c < 4; ++c) S[i][c] = pack2(x[2 * i][c], x[2 * i + 1][c]);
        }
    }
    // Staging.  `pieces`: raw 16-byte pieces of the next TB tokens travel in registers while these are walked, and are
    // widened, activated and put into shared memory when their turn comes.  Otherwise (partial sums, ragged rows) the
    // values are read when they are staged.
    const bool pieces = a.pieces;
    uint4 rq[outputs ? PQ : 1], rk[PQ], rv[PV];
    float4 rw[PW];
    auto fetch = [&](int tc) {
#pragma unroll
        for (int e = 0; e < PQ; ++e) {
            const int i = (tid + e * THREADS) * VT, tt = i / DP, d = i - tt * DP;
            const bool have = tt < TB && d < D && tc + tt < t1;
            rk[e] = have ? __ldg(reinterpret_cast<const uint4*>((const T*)a.k.x + (size_t)(tc + tt) * a.k.stride + a.k.off + h * D + d))
                         : make_uint4(0u, 0u, 0u, 0u);
            if constexpr (outputs)
                rq[e] = have ? __ldg(reinterpret_cast<const uint4*>((const T*)a.q.x + (size_t)(tc + tt) * a.q.stride + a.q.off + h * D + d))
                             : make_uint4(0u, 0u, 0u, 0u);
        }
        if (channel) {
#pragma unroll
            for (int e = 0; e < PW; ++e) {
                const int i = (tid + e * THREADS) * 4, tt = i / DP, d = i - tt * DP;
                rw[e] = tt < TB && d < D && tc + tt < t1
                            ? __ldg(reinterpret_cast<const float4*>((const float*)a.w.x + (size_t)(tc + tt) * a.w.stride + a.w.off + h * D + d))
                            : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
#pragma unroll
        for (int e = 0; e < PV; ++e) {
            const int i = (tid + e * THREADS) * VT, tt = i / COLS, c = i - tt * COLS;
            rv[e] = tt < TB && c0 + c < Dv && tc + tt < t1
                        ? __ldg(reinterpret_cast<const uint4*>((const T*)a.v.x + (size_t)(tc + tt) * a.v.stride + a.v.off + h * Dv + c0 + c))
                        : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    auto put = [&](float* dst, const uint4& raw, bool silu) {
        float f[VT];
        widen<T>(raw, f);
#pragma unroll
        for (int e = 0; e < VT; e += 4) {
            float4 x = make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]);
            if (silu) { x.x = silu_f(x.x); x.y = silu_f(x.y); x.z = silu_f(x.z); x.w = silu_f(x.w); }
            *reinterpret_cast<float4*>(dst + e) = x;
        }
    };
    pair2 w[P];
#pragma unroll
    for (int i = 0; i < P; ++i) w[i] = pack2(fixed, fixed);
    if (pieces) fetch(t0);
    for (int tc = t0; tc < t1; tc += TB) {
        const int nt = min(TB, t1 - tc);
        __syncthreads();                               // the walk over the tokens before is over
        if (pieces) {
#pragma unroll
            for (int e = 0; e < PQ; ++e) {
                const int i = (tid + e * THREADS) * VT;
                if (i >= TB * DP) continue;
                put(&ks[0][0] + i, rk[e], a.silu_qk);
                if constexpr (outputs) put(&qs[0][0] + i, rq[e], a.silu_qk);
            }
            if (channel) {
#pragma unroll
                for (int e = 0; e < PW; ++e) {
                    const int i = (tid + e * THREADS) * 4, d = i % DP;
                    if (i >= TB * DP) continue;
                    float4 x = rw[e];
                    x.x = expf(-expf(x.x + bs[d]));
                    x.y = expf(-expf(x.y + bs[d + 1]));
                    x.z = expf(-expf(x.z + bs[d + 2]));
                    x.w = expf(-expf(x.w + bs[d + 3]));
                    *reinterpret_cast<float4*>(&ws[0][0] + i) = x;
                }
            }
#pragma unroll
            for (int e = 0; e < PV; ++e) {
                const int i = (tid + e * THREADS) * VT;
                if (i < TB * COLS) put(&vs[0][0] + i, rv[e], a.silu_v);
            }
        } else {
            for (int i = tid; i < nt * DP; i += THREADS) {
                const int tt = i / DP, d = i - tt * DP;
                float q = 0.f, k = 0.f, x = 1.f;
                if (d < D) {
                    if (outputs) q = read_rows<T>(a.q, tc + tt, h * D + d);
                    k = read_rows<T>(a.k, tc + tt, h * D + d);
                    if (channel) x = expf(-expf(read_rows<float>(a.w, tc + tt, h * D + d) + bs[d]));
                }
                if (outputs) qs[outputs ? tt : 0][d] = a.silu_qk ? silu_f(q) : q;
                ks[tt][d] = a.silu_qk ? silu_f(k) : k;
                ws[tt][d] = x;
            }
            for (int i = tid; i < nt * COLS; i += THREADS) {
                const int tt = i / COLS, c = i - tt * COLS;
                const float v = c0 + c < Dv ? read_rows<T>(a.v, tc + tt, h * Dv + c0 + c) : 0.f;
                vs[tt][c] = a.silu_v ? silu_f(v) : v;
            }
        }
        __syncthreads();
        if (pieces && tc + TB < t1) fetch(tc + TB);    // in flight while these tokens are walked
        if (outputs && before) {                       // sum_i q_i u_i k_i of every token: what the bonus gives per value
            for (int tt = warp; tt < nt; tt += THREADS / 32) {
                float b = 0.f;
                for (int d = lane; d < DP; d += 32) b = fmaf(qs[outputs ? tt : 0][d] * us[d], ks[tt][d], b);
                b = warp_sum(b);
                if (lane == 0) bt[tt] = b;
            }
            __syncthreads();
        }
#pragma unroll 2
        for (int tt = 0; tt < nt; ++tt) {
            const float4 v = *reinterpret_cast<const float4*>(&vs[tt][cg * 4]);
            const pair2 vv[4] = {pack2(v.x, v.x), pack2(v.y, v.y), pack2(v.z, v.z), pack2(v.w, v.w)};
            pair2 k[P];
            load_pairs<RG, RR>(k, ks[tt], rg);
            if (channel) load_pairs<RG, RR>(w, ws[tt], rg);
            if constexpr (!outputs) {
#pragma unroll
                for (int i = 0; i < P; ++i) {
                    A[i] = mul2(A[i], w[i]);
#pragma unroll
                    for (int c = 0; c < 4; ++c) S[i][c] = fma2(w[i], S[i][c], mul2(k[i], vv[c]));
                }
            } else {
                pair2 q[P], oo[4] = {0ull, 0ull, 0ull, 0ull};
                load_pairs<RG, RR>(q, qs[tt], rg);
                if (before) {
#pragma unroll
                    for (int i = 0; i < P; ++i)
#pragma unroll
                        for (int c = 0; c < 4; ++c) {
                            oo[c] = fma2(q[i], S[i][c], oo[c]);
                            S[i][c] = fma2(w[i], S[i][c], mul2(k[i], vv[c]));
                        }
                } else {
#pragma unroll
                    for (int i = 0; i < P; ++i)
#pragma unroll
                        for (int c = 0; c < 4; ++c) {
                            S[i][c] = fma2(w[i], S[i][c], mul2(k[i], vv[c]));
                            oo[c] = fma2(q[i], S[i][c], oo[c]);
                        }
                }
                float o[4];
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    float x, y;
                    unpack2(oo[c], x, y);
                    o[c] = x + y;
                }
                // the RG lanes' shares: lanes split the four columns among themselves, then add what is left
                const bool b0 = rg & 1, b1 = rg & 2;
                const float p0 = __shfl_xor_sync(0xffffffffu, b0 ? o[0] : o[2], 1);
                const float p1 = __shfl_xor_sync(0xffffffffu, b0 ? o[1] : o[3], 1);
                const float e0 = (b0 ? o[2] : o[0]) + p0, e1 = (b0 ? o[3] : o[1]) + p1;
                float t = (b1 ? e1 : e0) + __shfl_xor_sync(0xffffffffu, b1 ? e0 : e1, 2);
#pragma unroll
                for (int sh = 4; sh < RG; sh <<= 1) t += __shfl_xor_sync(0xffffffffu, t, sh);
                if (rg < 4) {
                    const int c = cg * 4 + 2 * (rg & 1) + (rg >> 1);
                    os[tt][c] = before ? fmaf(bt[tt], vs[tt][c], t) : t;
                }
            }
        }
        if constexpr (outputs) {
            __syncthreads();
            for (int i = tid; i < nt * COLS; i += THREADS) {
                const int tt = i / COLS, c = i - tt * COLS;
                if (c0 + c < Dv) a.out[(size_t)(tc + tt) * H * Dv + h * Dv + c0 + c] = os[tt][c];
            }
        }
    }
    if (to != nullptr) {
#pragma unroll
        for (int i = 0; i < P; ++i) {
            float x[2][4], w[2];
#pragma unroll
            for (int c = 0; c < 4; ++c) unpack2(S[i][c], x[0][c], x[1][c]);
            unpack2(A[i], w[0], w[1]);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int row = row_of<RG, RR>(rg, 2 * i + e);
                if (row >= D) continue;
                float* p = to + (size_t)row * Dv + j0;
                if (vec) {
                    if (j0 < Dv) *reinterpret_cast<float4*>(p) = make_float4(x[e][0], x[e][1], x[e][2], x[e][3]);
                } else {
#pragma unroll
                    for (int c = 0; c < 4; ++c)
                        if (j0 + c < Dv) p[c] = x[e][c];
                }
                if (!outputs && blockIdx.z == 0 && cg == 0) a.seg_prod[((size_t)slot * H + h) * D + row] = w[e];
            }
        }
    }
}

// Between the two steps, for requests with several segments: each segment's end state (from zero) is replaced by
// the state before that segment, and the slot gets the state after the last.
__global__ void __launch_bounds__(256) recurrence_scan_kernel(RecArgs a) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    const int h = blockIdx.x, r = blockIdx.y;
    int slot = 0;
    for (int p = 0; p < r; ++p) {
        const int c = (a.seq_starts[p + 1] - a.seq_starts[p] + a.seg_len - 1) / a.seg_len;
        if (c > 1) slot += c;
    }
    const int nc = (a.seq_starts[r + 1] - a.seq_starts[r] + a.seg_len - 1) / a.seg_len;
    if (nc <= 1) return;
    const int size = a.D * a.Dv;
    float* S = a.state + ((size_t)a.seq_rows[r] * a.H + h) * size;
    for (int i = blockIdx.z * 256 + threadIdx.x; i < size; i += 256 * gridDim.z) {
        const int row = i / a.Dv;
        float s = S[i];
        for (int k0 = 0; k0 < nc; k0 += 8) {           // eight segments' loads in flight
            float e[8], p[8];
#pragma unroll
            for (int k = 0; k < 8; ++k)
                if (k0 + k < nc) {
                    const size_t at = (size_t)(slot + k0 + k) * a.H + h;
                    e[k] = a.seg_state[at * size + i];
                    p[k] = a.seg_prod[at * a.D + row];
                }
#pragma unroll
            for (int k = 0; k < 8; ++k)
                if (k0 + k < nc) {
                    a.seg_state[((size_t)(slot + k0 + k) * a.H + h) * size + i] = s;
                    s = fmaf(p[k], s, e[k]);
                }
        }
        S[i] = s;
    }
}

template <typename T, int RG, int RR>
void launch_sized(RecArgs a, int blocks, int seg_blocks, cudaStream_t stream) {
    constexpr int COLS = THREADS / RG * 4;
    const int zs = (a.Dv + COLS - 1) / COLS;
    if (seg_blocks > 0) {
        sb::launch(linear_recurrence_kernel<T, RG, RR, 1>, dim3(a.H, blocks, zs), dim3(THREADS), 0, stream, a);
        int slices = (a.D * a.Dv + 255) / 256;
        if (slices > 16) slices = 16;
        sb::launch(recurrence_scan_kernel, dim3(a.H, a.R, slices), dim3(256), 0, stream, a);
    }
    sb::launch(linear_recurrence_kernel<T, RG, RR, 2>, dim3(a.H, blocks, zs), dim3(THREADS), 0, stream, a);
}

template <typename T>
void launch_recurrence(const RecArgs& a, int blocks, int seg_blocks, cudaStream_t stream) {
    if (a.D <= 32) launch_sized<T, 16, 2>(a, blocks, seg_blocks, stream);
    else if (a.D <= 64) launch_sized<T, 16, 4>(a, blocks, seg_blocks, stream);
    else if (a.D <= 128) launch_sized<T, 16, 8>(a, blocks, seg_blocks, stream);
    else launch_sized<T, 32, 8>(a, blocks, seg_blocks, stream);
}

struct NormGateArgs {
    const float* x;            // [N, C]
    Rows gate;
    const float* gain;         // [C]
    void* out;                 // [N, C] in T
    int C, groups;
    float eps;
    int act;                   // 0: sigmoid; 1: SiLU
};

// Rows whose groups are whole 16-byte pieces: a thread takes four neighbouring columns and keeps them.  The lanes of a
// group (len / 4, a power of two up to 32) add up by shuffles, or, with one group, the whole block does.
template <typename T>
__global__ void __launch_bounds__(512) norm_gate_vec_kernel(NormGateArgs a) {
    sb::pdl_launch_dependents();
    __shared__ float scratch[33];
    const int n = blockIdx.x, len = a.C / a.groups, lanes = len / 4;
    sb::pdl_wait();
    const float4* x = reinterpret_cast<const float4*>(a.x + (size_t)n * a.C);
    T* y = (T*)a.out + (size_t)n * a.C;
    constexpr int MOST = 4;                            // pieces a thread keeps (columns up to 4 * MOST * threads)
    float4 v[MOST];
    float ss[MOST];
#pragma unroll
    for (int e = 0; e < MOST; ++e) {
        const int i = threadIdx.x + e * blockDim.x;
        v[e] = i < a.C / 4 ? x[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        ss[e] = v[e].x * v[e].x + v[e].y * v[e].y + v[e].z * v[e].z + v[e].w * v[e].w;
    }
    if (a.groups == 1) {
        const float total = block_sum((ss[0] + ss[1]) + (ss[2] + ss[3]), scratch);
        ss[0] = ss[1] = ss[2] = ss[3] = total;
    } else {
#pragma unroll
        for (int e = 0; e < MOST; ++e)
            for (int o = 1; o < lanes; o <<= 1) ss[e] += __shfl_xor_sync(0xffffffffu, ss[e], o);
    }
#pragma unroll
    for (int e = 0; e < MOST; ++e) {
        const int i = threadIdx.x + e * blockDim.x, c = 4 * i;
        if (i >= a.C / 4) continue;
        const float rinv = 1.0f / sqrtf(ss[e] / (float)len + a.eps);
        float z[4];
        const size_t at = (size_t)n * a.gate.stride + a.gate.off + c;
        if (a.gate.parts != nullptr) {
            z[0] = z[1] = z[2] = z[3] = 0.f;
            for (int s0 = 0; s0 < a.gate.S; s0 += 8) {
                float4 p[8];
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (s0 + j < a.gate.S) p[j] = __ldg(reinterpret_cast<const float4*>(a.gate.parts + (size_t)(s0 + j) * a.gate.part_stride + at));
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (s0 + j < a.gate.S) { z[0] += p[j].x; z[1] += p[j].y; z[2] += p[j].z; z[3] += p[j].w; }
            }
        } else if constexpr (sizeof(T) == 2) {
            const uint2 raw = *reinterpret_cast<const uint2*>((const T*)a.gate.x + at);
#pragma unroll
            for (int j = 0; j < 4; ++j) z[j] = to_float(reinterpret_cast<const T*>(&raw)[j]);
        } else {
            const float4 raw = *reinterpret_cast<const float4*>((const T*)a.gate.x + at);
            z[0] = raw.x; z[1] = raw.y; z[2] = raw.z; z[3] = raw.w;
        }
        const float4 g = __ldg(reinterpret_cast<const float4*>(a.gain + c));
        const float o[4] = {v[e].x * rinv * g.x, v[e].y * rinv * g.y, v[e].z * rinv * g.z, v[e].w * rinv * g.w};
        alignas(16) T r[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) r[j] = from_float<T>(o[j] * (a.act ? silu_f(z[j]) : __fdividef(1.0f, 1.0f + expf(-z[j]))));
        if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(y + c) = *reinterpret_cast<const uint2*>(r);
        else *reinterpret_cast<float4*>(y + c) = *reinterpret_cast<const float4*>(r);
    }
}

// A block per token.  Many groups: a warp per group; few: the block goes through them one by one.
template <typename T>
__global__ void __launch_bounds__(512) norm_gate_kernel(NormGateArgs a) {
    sb::pdl_launch_dependents();
    extern __shared__ float row[];
    __shared__ float scratch[33];
    const int n = blockIdx.x, len = a.C / a.groups;
    const bool by_warp = a.groups >= 4;
    const int start = by_warp ? (int)(threadIdx.x & 31) : (int)threadIdx.x, hop = by_warp ? 32 : (int)blockDim.x;
    const int warps = blockDim.x >> 5;
    sb::pdl_wait();
    const float* x = a.x + (size_t)n * a.C;
    T* y = (T*)a.out + (size_t)n * a.C;
    for (int g = by_warp ? (int)(threadIdx.x >> 5) : 0; g < a.groups; g += by_warp ? warps : 1) {
        float ss = 0.f;
#pragma unroll 4
        for (int i = start; i < len; i += hop) {
            const float v = x[g * len + i];
            row[g * len + i] = v;                      // read again by the same thread only
            ss += v * v;
        }
        const float total = by_warp ? warp_sum(ss) : block_sum(ss, scratch);
        const float rinv = 1.0f / sqrtf(total / (float)len + a.eps);
#pragma unroll 4
        for (int i = start; i < len; i += hop) {
            const int c = g * len + i;
            const float z = read_rows<T>(a.gate, n, c);
            const float s = 1.0f / (1.0f + expf(-z));
            y[c] = from_float<T>(row[c] * rinv * a.gain[c] * (a.act ? z * s : s));
        }
    }
}

constexpr int MAX_MIXES = 8;

template <typename T>
__global__ void __launch_bounds__(256) token_shift_mix_kernel(T* __restrict__ out, const T* __restrict__ x,
                                                              const float* __restrict__ mu, const float* __restrict__ last,
                                                              const int* __restrict__ token_rows, int mixes, int N, int d) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    const int n = blockIdx.x, row = token_rows[n];
    const bool first = n == 0 || token_rows[n - 1] != row;         // of its request's portion
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < d; i += gridDim.y * blockDim.x) {
        const float h = to_float(x[(size_t)n * d + i]);
        const float diff = (first ? last[(size_t)row * d + i] : to_float(x[(size_t)(n - 1) * d + i])) - h;
        for (int s = 0; s < mixes; ++s) out[((size_t)s * N + n) * d + i] = from_float<T>(fmaf(diff, mu[s * d + i], h));
    }
}

// d a multiple of the 16-byte vector: a thread mixes one vector.
template <typename T>
__global__ void __launch_bounds__(256) token_shift_mix_vec_kernel(T* __restrict__ out, const T* __restrict__ x,
                                                                  const float* __restrict__ mu, const float* __restrict__ last,
                                                                  const int* __restrict__ token_rows, int mixes, int N, int d) {
    sb::pdl_launch_dependents();
    constexpr int VEC = Vec16<T>::N;
    sb::pdl_wait();
    const int n = blockIdx.x, row = token_rows[n];
    const bool first = n == 0 || token_rows[n - 1] != row;
    for (int i = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; i < d; i += gridDim.y * blockDim.x * VEC) {
        Vec16<T> hv, pv;
        hv.load(x + (size_t)n * d + i);
        float h[VEC], diff[VEC];
        if (first) {
#pragma unroll
            for (int e = 0; e < VEC; e += 4) {
                const float4 p = *reinterpret_cast<const float4*>(last + (size_t)row * d + i + e);
                diff[e] = p.x; diff[e + 1] = p.y; diff[e + 2] = p.z; diff[e + 3] = p.w;
            }
        } else {
            pv.load(x + (size_t)(n - 1) * d + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) diff[e] = pv.get(e);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            h[e] = hv.get(e);
            diff[e] -= h[e];
        }
        for (int s = 0; s < mixes; ++s) {
            alignas(16) T y[VEC];
#pragma unroll
            for (int e = 0; e < VEC; e += 4) {
                const float4 m = __ldg(reinterpret_cast<const float4*>(mu + s * d + i + e));
                y[e] = from_float<T>(fmaf(diff[e], m.x, h[e]));
                y[e + 1] = from_float<T>(fmaf(diff[e + 1], m.y, h[e + 1]));
                y[e + 2] = from_float<T>(fmaf(diff[e + 2], m.z, h[e + 2]));
                y[e + 3] = from_float<T>(fmaf(diff[e + 3], m.w, h[e + 3]));
            }
            *reinterpret_cast<uint4*>(out + ((size_t)s * N + n) * d + i) = *reinterpret_cast<const uint4*>(y);
        }
    }
}

Rows rows_of(const void* x, int S, long long part_stride, long long stride, int off) {
    Rows r;
    r.x = S > 0 ? nullptr : x;
    r.parts = S > 0 ? (const float*)x : nullptr;
    r.S = S; r.part_stride = part_stride; r.stride = stride; r.off = off;
    return r;
}

}  // namespace

extern "C" int sb_linear_recurrence_supports(int D, int Dv) { return D >= 1 && D <= 256 && Dv >= 1; }

// Each of q, k, v, w: pointer, S (0: a matrix in the model dtype, w float32; else S float32 partial sums), the
// stride between partial sums, the stride between rows, the first column.  seg_len >= every portion: one launch.
extern "C" int sb_linear_recurrence(float* out, const void* q, int qS, long long qp, long long qs, int qo, const void* k,
                                    int kS, long long kp, long long ks, int ko, const void* v, int vS, long long vp,
                                    long long vs, int vo, const void* w, int wS, long long wp, long long ws, int wo,
                                    const float* decay, const float* base, const float* bonus, int silu_qk, int silu_v,
                                    float* state, const int* seq_starts, const int* seq_rows, int R, int H, int D, int Dv,
                                    int N, int seg_len, int longest, float* seg_state, float* seg_prod, int dtype,
                                    cudaStream_t stream) {
    SB_REQUIRE(R >= 0 && H > 0 && N >= 0 && sb_linear_recurrence_supports(D, Dv),
               "linear_recurrence: %d heads of %d (keys, at most 256) and %d (values) dims", H, D, Dv);
    SB_REQUIRE((w != nullptr) != (decay != nullptr), "linear_recurrence: decays are constants or come per token, not both");
    SB_REQUIRE(seg_len >= 1 && longest >= 0, "linear_recurrence: segments of %d tokens", seg_len);
    if (R == 0 || N == 0) return 0;
    const bool several = longest > seg_len;
    SB_REQUIRE(!several || (seg_state != nullptr && seg_prod != nullptr), "linear_recurrence: several segments need scratch");
    const int blocks = several ? N / seg_len + R : R;
    SB_REQUIRE(blocks <= 65535 && (Dv + 31) / 32 <= 65535, "linear_recurrence: %d segments exceed one launch", blocks);
    RecArgs a;
    a.q = rows_of(q, qS, qp, qs, qo); a.k = rows_of(k, kS, kp, ks, ko); a.v = rows_of(v, vS, vp, vs, vo);
    a.w = rows_of(w, wS, wp, ws, wo);
    const int vec = dtype == SB_BF16 ? 8 : 4;
    auto whole = [](const Rows& r, int n) {
        return r.parts == nullptr && r.stride % n == 0 && r.off % n == 0 && (reinterpret_cast<uintptr_t>(r.x) & 15) == 0;
    };
    a.pieces = N > R && D % vec == 0 && Dv % vec == 0 && whole(a.q, vec) && whole(a.k, vec) && whole(a.v, vec) &&
               (w == nullptr || whole(a.w, 4));
    a.decay = decay; a.base = base; a.bonus = bonus; a.silu_qk = silu_qk; a.silu_v = silu_v; a.state = state; a.out = out;
    a.seq_starts = seq_starts; a.seq_rows = seq_rows; a.R = R; a.H = H; a.D = D; a.Dv = Dv;
    a.seg_len = several ? seg_len : N; a.seg_state = seg_state; a.seg_prod = seg_prod;
    if (dtype == SB_F32) launch_recurrence<float>(a, blocks, several, stream);
    else if (dtype == SB_BF16) launch_recurrence<__nv_bfloat16>(a, blocks, several, stream);
    else SB_REQUIRE(false, "linear_recurrence: unknown dtype %d", dtype);
    SB_LAUNCH_CHECK();
}

extern "C" int sb_norm_gate(void* out, const float* x, const void* gate, int gS, long long gp, long long gs, int go,
                            const float* gain, int N, int C, int groups, float eps, int act, int dtype,
                            cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && C > 0 && groups >= 1 && C % groups == 0, "norm_gate: %d columns in %d groups", C, groups);
    SB_REQUIRE(act == 0 || act == 1, "norm_gate: unknown gate %d", act);
    const size_t smem = (size_t)C * sizeof(float);
    SB_REQUIRE(smem <= 160 * 1024, "norm_gate: rows of %d values do not fit a block's shared memory", C);
    if (N == 0) return 0;
    NormGateArgs a;
    a.x = x; a.gate = rows_of(gate, gS, gp, gs, go); a.gain = gain; a.out = out; a.C = C; a.groups = groups; a.eps = eps;
    a.act = act;
    const int threads = N <= 256 ? 512 : 256;         // few rows: more of a row in flight
    const int len = C / groups, lanes = len / 4;
    const bool grouped = groups == 1 || (lanes <= 32 && (lanes & (lanes - 1)) == 0);
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (C % 4 == 0 && len % 4 == 0 && grouped && C <= 4 * 4 * 512 && gs % 4 == 0 && gp % 4 == 0 && go % 4 == 0 && aligned(x) &&
        aligned(gate) && aligned(gain) && aligned(out)) {
        const int wide = C <= 4 * 256 || (C <= 4 * 4 * 256 && N > 256) ? 256 : 512;
        if (dtype == SB_F32) sb::launch(norm_gate_vec_kernel<float>, dim3(N), dim3(wide), 0, stream, a);
        else if (dtype == SB_BF16) sb::launch(norm_gate_vec_kernel<__nv_bfloat16>, dim3(N), dim3(wide), 0, stream, a);
        else SB_REQUIRE(false, "norm_gate: unknown dtype %d", dtype);
        SB_LAUNCH_CHECK();
    }
    if (dtype == SB_F32) {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(norm_gate_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        sb::launch(norm_gate_kernel<float>, dim3(N), dim3(threads), smem, stream, a);
    } else if (dtype == SB_BF16) {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(norm_gate_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        sb::launch(norm_gate_kernel<__nv_bfloat16>, dim3(N), dim3(threads), smem, stream, a);
    } else {
        SB_REQUIRE(false, "norm_gate: unknown dtype %d", dtype);
    }
    SB_LAUNCH_CHECK();
}

// out [mixes, N, d] in the model dtype; mu float32 [mixes, d]; last float32 [rows, d].
extern "C" int sb_token_shift_mix(void* out, const void* x, const float* mu, const float* last, const int* token_rows,
                                  int mixes, int N, int d, int dtype, cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && d > 0 && mixes >= 1 && mixes <= MAX_MIXES, "token_shift_mix: bad sizes N=%d d=%d mixes=%d", N, d, mixes);
    if (N == 0) return 0;
    const int vec = dtype == SB_BF16 ? 8 : 4;
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool wide = d % vec == 0 && aligned(out) && aligned(x) && aligned(mu) && aligned(last);
    const int items = wide ? d / vec : d, threads = items >= 256 ? 256 : ((items + 31) / 32) * 32;
    const dim3 grid(N, (items + threads - 1) / threads);
    SB_REQUIRE(grid.y <= 65535, "token_shift_mix: rows of %d values exceed one launch", d);
    if (dtype == SB_F32) {
        if (wide) sb::launch(token_shift_mix_vec_kernel<float>, grid, dim3(threads), 0, stream, (float*)out, (const float*)x, mu, last, token_rows, mixes, N, d);
        else sb::launch(token_shift_mix_kernel<float>, grid, dim3(threads), 0, stream, (float*)out, (const float*)x, mu, last, token_rows, mixes, N, d);
    } else if (dtype == SB_BF16) {
        if (wide) sb::launch(token_shift_mix_vec_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, (__nv_bfloat16*)out, (const __nv_bfloat16*)x, mu, last, token_rows, mixes, N, d);
        else sb::launch(token_shift_mix_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, (__nv_bfloat16*)out, (const __nv_bfloat16*)x, mu, last, token_rows, mixes, N, d);
    } else {
        SB_REQUIRE(false, "token_shift_mix: unknown dtype %d", dtype);
    }
    SB_LAUNCH_CHECK();
}
