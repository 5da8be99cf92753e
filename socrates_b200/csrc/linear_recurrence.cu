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
    for (int s = 0; s < a.S; ++s) v += a.parts[(size_t)s * a.part_stride + at];
    return v;
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

struct RecArgs {
    Rows q, k, v, w;           // w: raw decays; w.x and w.parts null: the constant
    const float* decay;        // [H] constants, or null
    const float* base;         // [H*D] added to the raw decays, or null
    const float* bonus;        // [H*D] or null: read after the write
    int silu_qk, silu_v;
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
    int step, seg_len;
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
// registers; the RG lanes of a column group are neighbours in a warp and join their shares of o by shuffles.
// TB tokens are staged in shared memory at a time (activations, decays and the bonus' dot product made there)
// while the raw values of the next TB are on their way into registers.
template <typename T, int RG, int RR>
__global__ void __launch_bounds__(THREADS) linear_recurrence_kernel(RecArgs a) {
    sb::pdl_launch_dependents();
    constexpr int DP = RG * RR, CG = THREADS / RG, COLS = CG * 4, TB = DP > 128 ? 8 : 16;
    constexpr int NE = TB * DP / THREADS, NV = TB * COLS / THREADS;
    __shared__ __align__(16) float qs[TB][DP], ks[TB][DP], ws[TB][DP], vs[TB][COLS], os[TB][COLS];
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
    const bool outputs = a.step == 2;
    if (!outputs && nc == 1) return;
    const int t0 = a.seq_starts[r] + ci * a.seg_len, t1 = min(a.seq_starts[r + 1], t0 + a.seg_len);
    const int j0 = c0 + cg * 4, i0 = rg * RR;
    // where the state comes from (null: zero) and goes to (null: nowhere)
    float* slot_state = a.state + ((size_t)a.seq_rows[r] * H + h) * D * Dv;
    float* seg_state = nc > 1 ? a.seg_state + ((size_t)slot * H + h) * D * Dv : nullptr;
    const float* from = outputs ? (nc > 1 ? seg_state : slot_state) : nullptr;
    float* to = outputs ? (nc > 1 ? nullptr : slot_state) : seg_state;
    const bool vec = Dv % 4 == 0;
    float S[RR][4], A[RR];
#pragma unroll
    for (int i = 0; i < RR; ++i) {
        A[i] = 1.f;
#pragma unroll
        for (int c = 0; c < 4; ++c) S[i][c] = 0.f;
        if (from != nullptr && i0 + i < D) {
            const float* p = from + (size_t)(i0 + i) * Dv + j0;
            if (vec) {
                if (j0 < Dv) {
                    const float4 x = *reinterpret_cast<const float4*>(p);
                    S[i][0] = x.x; S[i][1] = x.y; S[i][2] = x.z; S[i][3] = x.w;
                }
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (j0 + c < Dv) S[i][c] = p[c];
            }
        }
    }
    float rq[NE], rk[NE], rw[NE], rv[NV];
    auto fetch = [&](int tc) {
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            const int i = tid + e * THREADS, tt = i / DP, d = i - tt * DP;
            rq[e] = rk[e] = rw[e] = 0.f;
            if (d < D && tc + tt < t1) {
                if (outputs) rq[e] = read_rows<T>(a.q, tc + tt, h * D + d);
                rk[e] = read_rows<T>(a.k, tc + tt, h * D + d);
                if (channel) rw[e] = read_rows<float>(a.w, tc + tt, h * D + d);
            }
        }
#pragma unroll
        for (int e = 0; e < NV; ++e) {
            const int i = tid + e * THREADS, tt = i / COLS, c = i - tt * COLS;
            rv[e] = (c0 + c < Dv && tc + tt < t1) ? read_rows<T>(a.v, tc + tt, h * Dv + c0 + c) : 0.f;
        }
    };
    fetch(t0);
    for (int tc = t0; tc < t1; tc += TB) {
        const int nt = min(TB, t1 - tc);
        __syncthreads();                               // the walk over the tokens before is over
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            const int i = tid + e * THREADS, tt = i / DP, d = i - tt * DP;
            qs[tt][d] = a.silu_qk ? silu_f(rq[e]) : rq[e];
            ks[tt][d] = a.silu_qk ? silu_f(rk[e]) : rk[e];
            ws[tt][d] = channel ? (d < D ? expf(-expf(rw[e] + bs[d])) : 1.f) : fixed;
        }
#pragma unroll
        for (int e = 0; e < NV; ++e) {
            const int i = tid + e * THREADS, tt = i / COLS, c = i - tt * COLS;
            vs[tt][c] = a.silu_v ? silu_f(rv[e]) : rv[e];
        }
        __syncthreads();
        if (tc + TB < t1) fetch(tc + TB);              // in flight while these tokens are walked
        if (!outputs) {
#pragma unroll 2
            for (int tt = 0; tt < nt; ++tt) {
                const float4 v = *reinterpret_cast<const float4*>(&vs[tt][cg * 4]);
#pragma unroll
                for (int i = 0; i < RR; ++i) {
                    const float k = ks[tt][i0 + i], w = ws[tt][i0 + i];
                    A[i] *= w;
                    S[i][0] = fmaf(w, S[i][0], k * v.x);
                    S[i][1] = fmaf(w, S[i][1], k * v.y);
                    S[i][2] = fmaf(w, S[i][2], k * v.z);
                    S[i][3] = fmaf(w, S[i][3], k * v.w);
                }
            }
            continue;
        }
        if (before) {                                  // sum_i q_i u_i k_i of every token: what the bonus gives per value
            for (int tt = warp; tt < nt; tt += THREADS / 32) {
                float b = 0.f;
                for (int d = lane; d < DP; d += 32) b = fmaf(qs[tt][d] * us[d], ks[tt][d], b);
                b = warp_sum(b);
                if (lane == 0) bt[tt] = b;
            }
            __syncthreads();
        }
#pragma unroll 2
        for (int tt = 0; tt < nt; ++tt) {
            const float4 v = *reinterpret_cast<const float4*>(&vs[tt][cg * 4]);
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
            for (int i = 0; i < RR; ++i) {
                const float q = qs[tt][i0 + i], k = ks[tt][i0 + i], w = ws[tt][i0 + i];
                if (before) {
                    o0 = fmaf(q, S[i][0], o0); o1 = fmaf(q, S[i][1], o1); o2 = fmaf(q, S[i][2], o2); o3 = fmaf(q, S[i][3], o3);
                }
                S[i][0] = fmaf(w, S[i][0], k * v.x);
                S[i][1] = fmaf(w, S[i][1], k * v.y);
                S[i][2] = fmaf(w, S[i][2], k * v.z);
                S[i][3] = fmaf(w, S[i][3], k * v.w);
                if (!before) {
                    o0 = fmaf(q, S[i][0], o0); o1 = fmaf(q, S[i][1], o1); o2 = fmaf(q, S[i][2], o2); o3 = fmaf(q, S[i][3], o3);
                }
            }
            // the RG lanes' shares: lanes split the four columns among themselves, then add what is left
            const bool b0 = rg & 1, b1 = rg & 2;
            const float p0 = __shfl_xor_sync(0xffffffffu, b0 ? o0 : o2, 1), p1 = __shfl_xor_sync(0xffffffffu, b0 ? o1 : o3, 1);
            const float e0 = (b0 ? o2 : o0) + p0, e1 = (b0 ? o3 : o1) + p1;
            float o = (b1 ? e1 : e0) + __shfl_xor_sync(0xffffffffu, b1 ? e0 : e1, 2);
#pragma unroll
            for (int sh = 4; sh < RG; sh <<= 1) o += __shfl_xor_sync(0xffffffffu, o, sh);
            if (rg < 4) {
                const int c = cg * 4 + 2 * (rg & 1) + (rg >> 1);
                os[tt][c] = before ? fmaf(bt[tt], vs[tt][c], o) : o;
            }
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < NV; ++e) {
            const int i = tid + e * THREADS, tt = i / COLS, c = i - tt * COLS;
            if (tt < nt && c0 + c < Dv) a.out[(size_t)(tc + tt) * H * Dv + h * Dv + c0 + c] = os[tt][c];
        }
    }
    if (to != nullptr) {
#pragma unroll
        for (int i = 0; i < RR; ++i) {
            if (i0 + i >= D) continue;
            float* p = to + (size_t)(i0 + i) * Dv + j0;
            if (vec) {
                if (j0 < Dv) *reinterpret_cast<float4*>(p) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (j0 + c < Dv) p[c] = S[i][c];
            }
            if (!outputs && blockIdx.z == 0 && cg == 0) a.seg_prod[((size_t)slot * H + h) * D + i0 + i] = A[i];
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
        a.step = 1;
        sb::launch(linear_recurrence_kernel<T, RG, RR>, dim3(a.H, blocks, zs), dim3(THREADS), 0, stream, a);
        int slices = (a.D * a.Dv + 255) / 256;
        if (slices > 16) slices = 16;
        sb::launch(recurrence_scan_kernel, dim3(a.H, a.R, slices), dim3(256), 0, stream, a);
    }
    a.step = 2;
    sb::launch(linear_recurrence_kernel<T, RG, RR>, dim3(a.H, blocks, zs), dim3(THREADS), 0, stream, a);
}

template <typename T>
void launch_recurrence(const RecArgs& a, int blocks, int seg_blocks, cudaStream_t stream) {
    if (a.D <= 32) launch_sized<T, 16, 2>(a, blocks, seg_blocks, stream);
    else if (a.D <= 64) launch_sized<T, 16, 4>(a, blocks, seg_blocks, stream);
    else if (a.D <= 128) launch_sized<T, 32, 4>(a, blocks, seg_blocks, stream);
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

// A block per token.  Many groups: a warp per group; few: the block goes through them one by one.
template <typename T>
__global__ void __launch_bounds__(256) norm_gate_kernel(NormGateArgs a) {
    sb::pdl_launch_dependents();
    extern __shared__ float row[];
    __shared__ float scratch[33];
    const int n = blockIdx.x, len = a.C / a.groups;
    const bool by_warp = a.groups >= 4;
    const int start = by_warp ? (int)(threadIdx.x & 31) : (int)threadIdx.x, hop = by_warp ? 32 : 256;
    sb::pdl_wait();
    const float* x = a.x + (size_t)n * a.C;
    T* y = (T*)a.out + (size_t)n * a.C;
    for (int g = by_warp ? (int)(threadIdx.x >> 5) : 0; g < a.groups; g += by_warp ? 8 : 1) {
        float ss = 0.f;
        for (int i = start; i < len; i += hop) {
            const float v = x[g * len + i];
            row[g * len + i] = v;                      // read again by the same thread only
            ss += v * v;
        }
        const float total = by_warp ? warp_sum(ss) : block_sum(ss, scratch);
        const float rinv = 1.0f / sqrtf(total / (float)len + a.eps);
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
    a.decay = decay; a.base = base; a.bonus = bonus; a.silu_qk = silu_qk; a.silu_v = silu_v; a.state = state; a.out = out;
    a.seq_starts = seq_starts; a.seq_rows = seq_rows; a.R = R; a.H = H; a.D = D; a.Dv = Dv; a.step = 2;
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
    if (dtype == SB_F32) {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(norm_gate_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        sb::launch(norm_gate_kernel<float>, dim3(N), dim3(256), smem, stream, a);
    } else if (dtype == SB_BF16) {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(norm_gate_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        sb::launch(norm_gate_kernel<__nv_bfloat16>, dim3(N), dim3(256), smem, stream, a);
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
