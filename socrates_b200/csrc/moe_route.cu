// Routing of a mixture-of-experts feed-forward, and the small steps around the experts' products.
//
//   logits:      z[n][e] = sum_k x[n][k] * router[e][k]        (float32 weights and sums, a block per token)
//   route:       s = softmax(z) over all E router outputs (float32)
//                c = s + correction                              (the scores experts are CHOSEN by)
//                the E outputs form `groups` equal groups of neighbours; a group's score is its
//                largest c; only the `keep` best groups stay (the others' c count as -inf)
//                the `top` largest c are chosen; their weights are s (no correction, not renormalized)
//                weights[n][e] = s_e for chosen e, else 0 ;  ids[n][k], picked[n][k] = the choices, best first
//   router:      logits and choice in one kernel: the `top` largest of z + bias are chosen; their weights are the
//                softmax over these only
//                or, by scores s = sigmoid(z): the E outputs form groups of neighbours, a group counts with the sum of its
//                two largest s, only the `keep` best groups stay, the `top` largest s there are chosen and weigh
//                s / (their sum + 1e-20) * scale
//   act:         all experts' units without a gate:  act[n][e*F + f] = relu(sum_s in[s][n][e*F + f])^2 * weights[n][e]
//   glu_clamp:   all experts' gated units and the shared one's in one pass, scaled on the way out:
//                g = min(pg, limit) ,  u = clamp(pu, -limit, limit) ,  act = g * sigmoid(alpha g) * (u + offset) * weight
//   scale:       act[n][e*F + f] *= weights[n][e]                (all experts' activations side by side)
//   passthrough: slab[n][:] = x[n][:] * sum of weights[n][e] over e >= first_identity
//                (router outputs past the real experts stand for "the input itself")
//
// Ties go to the lower index.  One warp routes one token.
#include <math.h>

#include "common.cuh"

using namespace sb;

namespace {

// (value, index) of the largest value over a warp; ties go to the lower index.
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oi = __shfl_xor_sync(0xffffffffu, i, o);
        if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
    }
}

constexpr int ROUTE_WARPS = 4;

__global__ void __launch_bounds__(ROUTE_WARPS * 32) moe_route_kernel(
    const float* __restrict__ logits, const float* __restrict__ correction, float* __restrict__ weights,
    int* __restrict__ ids, float* __restrict__ picked, int N, int E, int groups, int keep, int top) {
    sb::pdl_launch_dependents();
    extern __shared__ float rsm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* s = rsm + (size_t)warp * (2 * E + groups);      // scores
    float* c = s + E;                                       // choice scores
    float* gs = c + E;                                      // group scores
    const int n = blockIdx.x * ROUTE_WARPS + warp;
    sb::pdl_wait();
    if (n >= N) return;
    const float* z = logits + (size_t)n * E;
    float mx = -INFINITY;
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, z[e]);
    mx = warp_max(mx);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) {
        const float p = expf(z[e] - mx);
        s[e] = p;
        sum += p;
    }
    sum = warp_sum(sum);
    const float inv = 1.0f / sum;
    for (int e = lane; e < E; e += 32) {
        const float p = s[e] * inv;
        s[e] = p;
        c[e] = p + (correction ? correction[e] : 0.f);
        weights[(size_t)n * E + e] = 0.f;
    }
    __syncwarp();
    if (keep < groups) {
        const int per = E / groups;
        for (int g = lane; g < groups; g += 32) {
            float best = -INFINITY;
            for (int e = g * per; e < (g + 1) * per; ++e) best = fmaxf(best, c[e]);
            gs[g] = best;
        }
        __syncwarp();
        // the `keep` best groups are marked with +inf, then every other group's experts are closed
        for (int it = 0; it < keep; ++it) {
            float bv = -INFINITY;
            int bi = 0x7fffffff;
            for (int g = lane; g < groups; g += 32) {
                const float v = gs[g];
                if (v != INFINITY && (v > bv || bi == 0x7fffffff)) { bv = v; bi = g; }
            }
            warp_argmax(bv, bi);
            if (lane == 0 && bi != 0x7fffffff) gs[bi] = INFINITY;
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (gs[e / per] != INFINITY) c[e] = -INFINITY;
        __syncwarp();
    }
    for (int k = 0; k < top; ++k) {
        float bv = -INFINITY;
        int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float v = c[e];
            if (!isnan(v) && (v > bv)) { bv = v; bi = e; }
        }
        warp_argmax(bv, bi);
        if (bi == 0x7fffffff) {                 // fewer open experts than `top`: nothing more to choose
            if (lane == 0) { ids[(size_t)n * top + k] = -1; picked[(size_t)n * top + k] = 0.f; }
            continue;
        }
        if (lane == 0) {
            const float p = s[bi];
            weights[(size_t)n * E + bi] = p;
            ids[(size_t)n * top + k] = bi;
            picked[(size_t)n * top + k] = p;
            c[bi] = NAN;                         // taken
        }
        __syncwarp();
    }
}

// The router's product and the choice by its logits in one kernel, TT tokens a block.  A warp makes an
// output's logits for all of them: lane l takes elements 4 l .. 4 l + 3 of every 128, in order, one sum a lane joined in a fixed
// tree, so a token's logits do not depend on what else the step holds.  Then a warp per token picks the `top` largest
// of logit + bias (ties to the lower index) and writes the softmax over these.
struct RouterArgs {
    const void* x;             // [N, K] in T
    const float* router;       // [E, K]
    const float* bias;         // [E] or null
    float* weights;            // [N, E]
    int* ids;                  // [N, top]
    float* picked;             // [N, top]
    int N, E, K, top;
    int sigmoid, groups, keep; // sigmoid: choose and weigh by sigmoid scores, inside the `keep` best of `groups`
    float scale;
};

template <typename T, int TT>
__global__ void __launch_bounds__(TT == 1 ? 1024 : 256) moe_router_kernel(RouterArgs a) {
    sb::pdl_launch_dependents();
    extern __shared__ __align__(16) float rsm[];
    const int K = a.K, E = a.E, Kp = (K + 127) / 128 * 128;
    float* xs = rsm;                                         // [TT][Kp]
    float* zs = xs + TT * Kp;                                // [TT][2 E]: open logits, weights
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n0 = blockIdx.x * TT, warps = blockDim.x >> 5;
    sb::pdl_wait();
    const T* x = (const T*)a.x;
    constexpr int VEC = Vec16<T>::N;
    if (K % VEC == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0) {
        for (int i = threadIdx.x * VEC; i < TT * Kp; i += blockDim.x * VEC) {
            const int t = i / Kp, k = i - t * Kp;
            Vec16<T> v;
            const bool have = n0 + t < a.N && k < K;
            if (have) v.load(x + (size_t)(n0 + t) * K + k);
#pragma unroll
            for (int e = 0; e < VEC; ++e) xs[i + e] = have ? v.get(e) : 0.f;
        }
    } else {
        for (int i = threadIdx.x; i < TT * Kp; i += blockDim.x) {
            const int t = i / Kp, k = i - t * Kp;
            xs[i] = n0 + t < a.N && k < K ? to_float(x[(size_t)(n0 + t) * K + k]) : 0.f;
        }
    }
    __syncthreads();
    const bool wide = K % 4 == 0;
    for (int e = warp; e < E; e += warps) {
        const float* w = a.router + (size_t)e * K;
        float acc[TT];
#pragma unroll
        for (int t = 0; t < TT; ++t) acc[t] = 0.f;
#pragma unroll (TT == 1 ? 8 : 4)
        for (int k = lane * 4; k < Kp; k += 128) {
            float4 wv = make_float4(0.f, 0.f, 0.f, 0.f);
            if (wide) {
                if (k < K) wv = __ldg(reinterpret_cast<const float4*>(w + k));
            } else {
                if (k < K) wv.x = w[k];
                if (k + 1 < K) wv.y = w[k + 1];
                if (k + 2 < K) wv.z = w[k + 2];
                if (k + 3 < K) wv.w = w[k + 3];
            }
#pragma unroll
            for (int t = 0; t < TT; ++t) {
                const float4 xv = *reinterpret_cast<const float4*>(xs + t * Kp + k);
                acc[t] = fmaf(xv.x, wv.x, fmaf(xv.y, wv.y, fmaf(xv.z, wv.z, fmaf(xv.w, wv.w, acc[t]))));
            }
        }
        const float b = a.bias ? a.bias[e] : 0.f;
#pragma unroll
        for (int t = 0; t < TT; ++t) {
            const float z = warp_sum(acc[t]);
            if (lane == 0) {
                zs[t * 2 * E + e] = a.sigmoid ? 1.0f / (1.0f + expf(-(z + b))) : z + b;
                zs[t * 2 * E + E + e] = 0.f;
            }
        }
    }
    __syncthreads();
    for (int t = warp; t < TT; t += warps) {
        const int n = n0 + t;
        if (n >= a.N) break;
        float *c = zs + t * 2 * E, *w = c + E;
        float best = 0.f, sum = 0.f;
        if (a.sigmoid && a.keep < a.groups) {
            // w serves as scratch: w[g] = the group's score, then +inf for a group that stays
            const int per = E / a.groups;
            for (int g = lane; g < a.groups; g += 32) {
                float first = 0.f, second = 0.f;
                for (int e = g * per; e < (g + 1) * per; ++e) {
                    const float v = c[e];
                    if (v > first) { second = first; first = v; }
                    else if (v > second) second = v;
                }
                w[g] = first + second;
            }
            __syncwarp();
            for (int it = 0; it < a.keep; ++it) {
                float bv = -INFINITY;
                int bi = 0x7fffffff;
                for (int g = lane; g < a.groups; g += 32) {
                    const float v = w[g];
                    if (v != INFINITY && (v > bv || bi == 0x7fffffff)) { bv = v; bi = g; }
                }
                warp_argmax(bv, bi);
                if (lane == 0 && bi < a.groups) w[bi] = INFINITY;
                __syncwarp();
            }
            for (int e = lane; e < E; e += 32)
                if (w[e / per] != INFINITY) c[e] = -INFINITY;
            __syncwarp();
            for (int g = lane; g < a.groups; g += 32) w[g] = 0.f;
            __syncwarp();
        }
        for (int k = 0; k < a.top; ++k) {
            float bv = -INFINITY;
            int bi = 0x7fffffff;
            for (int e = lane; e < E; e += 32) {
                const float v = c[e];
                if (!isnan(v) && (v > bv || bi == 0x7fffffff)) { bv = v; bi = e; }
            }
            warp_argmax(bv, bi);
            if (k == 0) best = bv;
            const float p = a.sigmoid ? bv : expf(bv - best);
            sum += p;
            if (lane == 0 && bi < E) {
                a.ids[(size_t)n * a.top + k] = bi;
                w[bi] = p;
                c[bi] = NAN;                                 // taken
            }
            __syncwarp();
        }
        const float inv = a.sigmoid ? a.scale / (sum + 1e-20f) : 1.0f / sum;
        for (int e = lane; e < E; e += 32) a.weights[(size_t)n * E + e] = w[e] * inv;
        for (int k = lane; k < a.top; k += 32) a.picked[(size_t)n * a.top + k] = w[a.ids[(size_t)n * a.top + k]] * inv;
    }
}

template <typename T, int TT>
void launch_router(const RouterArgs& a, size_t smem, cudaStream_t stream) {
    static sb::OncePerDevice once;
    if (smem > 48 * 1024 && !once.flag()) {
        cudaFuncSetAttribute(moe_router_kernel<T, TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        once.flag() = true;
    }
    // one token: a warp per output as far as a block goes, so that its rows are on their way together
    const int warps = TT > 1 ? 8 : a.E < 8 ? 8 : a.E > 32 ? 32 : a.E;
    sb::launch(moe_router_kernel<T, TT>, dim3((a.N + TT - 1) / TT), dim3(32 * warps), smem, stream, a);
}

// Column f < experts * F belongs to expert f / F; the columns from there on to the shared expert, whose weight is
// one.  An expert that was not chosen is not read: its activations are zero.
struct MoeGluArgs {
    const void* in;            // [N, 2W] in T (gates, then values), or null
    const float* parts;        // [S, N, 2W]
    int S;
    size_t part_stride;
    const float* weights;      // [N, E_total]
    void* out;                 // [N, W] in T
    int W, E_total, experts, F;
    float limit, shared_limit, alpha, offset;
};

__device__ __forceinline__ float glu_clamped(float g, float u, float limit, float alpha, float offset) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-alpha * g)) * (u + offset);
}

template <typename T>
__global__ void __launch_bounds__(256) moe_glu_clamp_kernel(MoeGluArgs a, size_t total) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t n = i / a.W;
        const int f = (int)(i - n * a.W), e = f / a.F;
        const bool shared = e >= a.experts;
        const float w = shared ? 1.f : a.weights[n * a.E_total + e];
        float y = 0.f;
        if (w != 0.f) {
            const size_t at = n * 2 * a.W + f;
            float g = 0.f, u = 0.f;
            if (a.parts) {
                for (int s = 0; s < a.S; ++s) { g += a.parts[s * a.part_stride + at]; u += a.parts[s * a.part_stride + at + a.W]; }
            } else {
                g = to_float(((const T*)a.in)[at]);
                u = to_float(((const T*)a.in)[at + a.W]);
            }
            y = glu_clamped(g, u, shared ? a.shared_limit : a.limit, a.alpha, a.offset) * w;
        }
        ((T*)a.out)[i] = from_float<T>(y);
    }
}

// F and W multiples of the 16-byte vector: a thread takes one vector, whose elements share their expert.
template <typename T>
__global__ void __launch_bounds__(256) moe_glu_clamp_vec_kernel(MoeGluArgs a, size_t packs) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    constexpr int VEC = Vec16<T>::N;
    const int per_row = a.W / VEC;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < packs; i += (size_t)gridDim.x * blockDim.x) {
        const size_t n = i / per_row;
        const int f = (int)(i - n * per_row) * VEC, e = f / a.F;
        const bool shared = e >= a.experts;
        const float w = shared ? 1.f : a.weights[n * a.E_total + e];
        T* out = (T*)a.out + n * a.W + f;
        if (w == 0.f) {
            *reinterpret_cast<uint4*>(out) = make_uint4(0u, 0u, 0u, 0u);
            continue;
        }
        const float limit = shared ? a.shared_limit : a.limit;
        float g[VEC], u[VEC];
        if (a.parts) {
#pragma unroll
            for (int j = 0; j < VEC; ++j) g[j] = u[j] = 0.f;
            for (int s = 0; s < a.S; ++s) {
                const float* p = a.parts + s * a.part_stride + n * 2 * a.W + f;
#pragma unroll
                for (int j = 0; j < VEC; j += 4) {
                    const float4 x = *reinterpret_cast<const float4*>(p + j), y = *reinterpret_cast<const float4*>(p + a.W + j);
                    g[j] += x.x; g[j + 1] += x.y; g[j + 2] += x.z; g[j + 3] += x.w;
                    u[j] += y.x; u[j + 1] += y.y; u[j + 2] += y.z; u[j + 3] += y.w;
                }
            }
        } else {
            Vec16<T> gv, uv;
            gv.load((const T*)a.in + n * 2 * a.W + f);
            uv.load((const T*)a.in + n * 2 * a.W + a.W + f);
#pragma unroll
            for (int j = 0; j < VEC; ++j) { g[j] = gv.get(j); u[j] = uv.get(j); }
        }
        alignas(16) T y[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) y[j] = from_float<T>(glu_clamped(g[j], u[j], limit, a.alpha, a.offset) * w);
        *reinterpret_cast<uint4*>(out) = *reinterpret_cast<const uint4*>(y);
    }
}

// Units without a gate: relu squared, scaled.  VEC = 1 serves any shape; with VEC the 16-byte vector (F a multiple of
// it) a thread takes one vector, whose elements share their expert.  An expert that was not chosen is not read.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) moe_act_kernel(MoeGluArgs a, size_t items) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    const int per_row = a.W / VEC;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < items; i += (size_t)gridDim.x * blockDim.x) {
        const size_t n = i / per_row;
        const int f = (int)(i - n * per_row) * VEC;
        const float w = a.weights[n * a.E_total + f / a.F];
        T* out = (T*)a.out + n * a.W + f;
        float z[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) z[j] = 0.f;
        if (w != 0.f) {
            if (a.parts) {
                for (int s = 0; s < a.S; ++s) {
                    const float* p = a.parts + s * a.part_stride + n * a.W + f;
                    if constexpr (VEC == 1) {
                        z[0] += *p;
                    } else {
#pragma unroll
                        for (int j = 0; j < VEC; j += 4) {
                            const float4 x = *reinterpret_cast<const float4*>(p + j);
                            z[j] += x.x; z[j + 1] += x.y; z[j + 2] += x.z; z[j + 3] += x.w;
                        }
                    }
                }
            } else if constexpr (VEC == 1) {
                z[0] = to_float(((const T*)a.in)[n * a.W + f]);
            } else {
                Vec16<T> v;
                v.load((const T*)a.in + n * a.W + f);
#pragma unroll
                for (int j = 0; j < VEC; ++j) z[j] = v.get(j);
            }
        }
        alignas(16) T y[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
            const float p = fmaxf(z[j], 0.f);
            y[j] = from_float<T>(p * p * w);
        }
        if constexpr (VEC == 1) *out = y[0];
        else *reinterpret_cast<uint4*>(out) = *reinterpret_cast<const uint4*>(y);
    }
}

// A block per (token, four router outputs): the row of x goes to shared memory once (as float32), then each
// warp sums one output over K in a fixed order, whatever the batch holds: lane l takes elements l, l + 32,
// ..., eight loads in flight, four partial sums joined in a fixed tree.
template <typename T>
__global__ void __launch_bounds__(128) moe_logits_kernel(float* __restrict__ logits, const T* __restrict__ x,
                                                         const float* __restrict__ router, int E, int K) {
    sb::pdl_launch_dependents();
    extern __shared__ float xs[];
    const int n = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int e = blockIdx.y * 4 + warp;
    const float* w = router + (size_t)(e < E ? e : 0) * K;
    float wv[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) wv[j] = lane + 32 * j < K ? w[lane + 32 * j] : 0.f;     // weights: before the wait
    sb::pdl_wait();
    for (int k = threadIdx.x; k < K; k += blockDim.x) xs[k] = to_float(x[(size_t)n * K + k]);
    __syncthreads();
    if (e >= E) return;
    float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
    for (int k0 = 0; k0 < K; k0 += 256) {
        float nx[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {                       // the next eight are on their way while these are used
            const int k = k0 + 256 + lane + 32 * j;
            nx[j] = k < K ? w[k] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < 8; j += 4) {
            const int k = k0 + lane + 32 * j;
            a0 = fmaf(k < K ? xs[k] : 0.f, wv[j], a0);
            a1 = fmaf(k + 32 < K ? xs[k + 32] : 0.f, wv[j + 1], a1);
            a2 = fmaf(k + 64 < K ? xs[k + 64] : 0.f, wv[j + 2], a2);
            a3 = fmaf(k + 96 < K ? xs[k + 96] : 0.f, wv[j + 3], a3);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) wv[j] = nx[j];
    }
    const float total = warp_sum((a0 + a1) + (a2 + a3));
    if (lane == 0) logits[(size_t)n * E + e] = total;
}

template <typename T>
__global__ void __launch_bounds__(256) moe_scale_kernel(T* __restrict__ act, const float* __restrict__ weights,
                                                        int E_total, int experts, int F, size_t total) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    const size_t width = (size_t)experts * F;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t n = i / width;
        const int e = (int)((i - n * width) / F);
        const float w = weights[n * E_total + e];
        act[i] = from_float<T>(w == 0.f ? 0.f : to_float(act[i]) * w);
    }
}

// F a multiple of the 16-byte vector: a thread scales one vector, whose elements share their expert.
// An expert that was not chosen is not even read: its activations are overwritten with zeros.
template <typename T>
__global__ void __launch_bounds__(256) moe_scale_vec_kernel(T* __restrict__ act, const float* __restrict__ weights,
                                                            int E_total, int experts, int F, size_t total_vec) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    constexpr int VEC = Vec16<T>::N;
    const size_t width_vec = (size_t)experts * F / VEC;
    const int f_vec = F / VEC;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total_vec; i += (size_t)gridDim.x * blockDim.x) {
        const size_t n = i / width_vec;
        const int e = (int)((i - n * width_vec) / f_vec);
        const float w = weights[n * E_total + e];
        T* p = act + i * VEC;
        if (w == 0.f) {
            *reinterpret_cast<uint4*>(p) = make_uint4(0u, 0u, 0u, 0u);
            continue;
        }
        Vec16<T> v;
        v.load(p);
        alignas(16) T r[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) r[j] = from_float<T>(v.get(j) * w);
        *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(r);
    }
}

template <typename T>
__global__ void __launch_bounds__(256) moe_passthrough_kernel(float* __restrict__ slab, const T* __restrict__ x,
                                                              const float* __restrict__ weights, int E_total,
                                                              int first_identity, int d) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    const int n = blockIdx.x;
    float w = 0.f;
    for (int e = first_identity; e < E_total; ++e) w += weights[(size_t)n * E_total + e];
    for (int i = threadIdx.x; i < d; i += blockDim.x) slab[(size_t)n * d + i] = w * to_float(x[(size_t)n * d + i]);
}

// Routing by a table: token id t uses the experts table[t, 0..top-1] (distinct), each with weight 1 / top.
// Writes the dense weights [N, E] (zero where not chosen) that the scaling kernel reads.  A negative id -1 - j
// stands for feedback[j], a token that an earlier kernel on the stream wrote (as in the embedding).
__global__ void __launch_bounds__(128) moe_table_kernel(float* __restrict__ weights, const int* __restrict__ ids,
                                                        const int* __restrict__ feedback, const int* __restrict__ table,
                                                        int N, int E, int top, int V) {
    sb::pdl_launch_dependents();
    sb::pdl_wait();
    const int n = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (n >= N) return;
    int id = ids[n];
    if (id < 0 && feedback != nullptr) id = feedback[-1 - id];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);
    const int* row = table + (size_t)id * top;
    const float share = 1.0f / (float)top;
    for (int e = lane; e < E; e += 32) {
        float w = 0.f;
        for (int j = 0; j < top; ++j) w = row[j] == e ? share : w;
        weights[(size_t)n * E + e] = w;
    }
}

}  // namespace

extern "C" int sb_moe_table(float* weights, const int* ids, const int* feedback, const int* table, int N, int E,
                            int top, int V, cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && E > 0 && top >= 1 && top <= E && V > 0, "moe_table: bad sizes N=%d E=%d top=%d V=%d", N, E, top, V);
    if (N == 0) return 0;
    sb::launch(moe_table_kernel, dim3((N + 3) / 4), dim3(128), 0, stream, weights, ids, feedback, table, N, E, top, V);
    SB_LAUNCH_CHECK();
}

extern "C" int sb_moe_route(const float* logits, const float* correction, float* weights, int* ids, float* picked,
                            int N, int E, int groups, int keep, int top, cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && E > 0 && top >= 1 && top <= E, "moe_route: bad sizes N=%d E=%d top=%d", N, E, top);
    SB_REQUIRE(groups >= 1 && E % groups == 0 && keep >= 1 && keep <= groups,
               "moe_route: %d router outputs in %d groups of which %d stay", E, groups, keep);
    SB_REQUIRE(top <= keep * (E / groups), "moe_route: %d choices from %d open experts", top, keep * (E / groups));
    const size_t smem = (size_t)ROUTE_WARPS * (2 * E + groups) * sizeof(float);
    SB_REQUIRE(smem <= 48 * 1024, "moe_route: %d router outputs do not fit a block's shared memory", E);
    if (N == 0) return 0;
    sb::launch(moe_route_kernel, dim3((N + ROUTE_WARPS - 1) / ROUTE_WARPS), dim3(ROUTE_WARPS * 32), smem, stream,
               logits, correction, weights, ids, picked, N, E, groups, keep, top);
    SB_LAUNCH_CHECK();
}

// weights float32 [N, E]; ids int32 and picked float32 [N, top].
extern "C" int sb_moe_router(const void* x, const float* router, const float* bias, float* weights, int* ids, float* picked,
                             int N, int E, int K, int top, int sigmoid, int groups, int keep, float scale, int dtype,
                             cudaStream_t stream) {
    SB_REQUIRE(groups >= 1 && E % groups == 0 && keep >= 1 && keep <= groups && (sigmoid || groups == 1),
               "moe_router: %d outputs in %d groups of which %d stay", E, groups, keep);
    SB_REQUIRE(top <= keep * (E / groups), "moe_router: %d choices from %d open experts", top, keep * (E / groups));
    SB_REQUIRE(N >= 0 && E > 0 && K > 0 && top >= 1 && top <= E, "moe_router: bad sizes N=%d E=%d K=%d top=%d", N, E, K, top);
    const int Kp = (K + 127) / 128 * 128;
    auto need = [&](int tt) { return (size_t)tt * (Kp + 2 * E) * sizeof(float); };
    SB_REQUIRE(need(1) <= 200 * 1024, "moe_router: rows of %d values and %d outputs do not fit a block's shared memory", K, E);
    SB_REQUIRE(dtype == SB_F32 || dtype == SB_BF16, "moe_router: unknown dtype %d", dtype);
    if (N == 0) return 0;
    RouterArgs a;
    a.x = x; a.router = router; a.bias = bias; a.weights = weights; a.ids = ids; a.picked = picked; a.N = N; a.E = E; a.K = K;
    a.top = top; a.sigmoid = sigmoid; a.groups = groups; a.keep = keep; a.scale = scale;
    const bool many = N >= 512 && need(8) <= 100 * 1024;      // many tokens: a router row fetched once serves eight
    if (dtype == SB_F32) { if (many) launch_router<float, 8>(a, need(8), stream); else launch_router<float, 1>(a, need(1), stream); }
    else { if (many) launch_router<__nv_bfloat16, 8>(a, need(8), stream); else launch_router<__nv_bfloat16, 1>(a, need(1), stream); }
    SB_LAUNCH_CHECK();
}

// in [N, 2W] in the model dtype (or parts float32 [S, N, 2W]), W = experts * F + shared columns.
extern "C" int sb_moe_glu_clamp(void* out, const void* in, const float* parts, int S, long long part_stride,
                                const float* weights, int N, int W, int E_total, int experts, int F, float limit,
                                float shared_limit, float alpha, float offset, int dtype, cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && experts > 0 && experts <= E_total && F > 0 && W >= experts * F,
               "moe_glu_clamp: bad sizes N=%d experts=%d/%d F=%d W=%d", N, experts, E_total, F, W);
    SB_REQUIRE(limit > 0.f && shared_limit > 0.f, "moe_glu_clamp: clamps at %f and %f", limit, shared_limit);
    SB_REQUIRE((in != nullptr) != (parts != nullptr), "moe_glu_clamp: one input, a matrix or partial sums");
    if (N == 0) return 0;
    MoeGluArgs a;
    a.in = in; a.parts = parts; a.S = S; a.part_stride = (size_t)part_stride; a.weights = weights; a.out = out; a.W = W;
    a.E_total = E_total; a.experts = experts; a.F = F; a.limit = limit; a.shared_limit = shared_limit; a.alpha = alpha;
    a.offset = offset;
    const size_t total = (size_t)N * W;
    const int vec = dtype == SB_BF16 ? 8 : 4;
    const bool wide = F % vec == 0 && W % vec == 0 && part_stride % 4 == 0 &&
                      ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(parts) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    const size_t items = wide ? total / vec : total;
    const int blocks = (int)((items + 255) / 256 < 148 * 16 ? (items + 255) / 256 : 148 * 16);
    if (dtype == SB_F32) {
        if (wide) sb::launch(moe_glu_clamp_vec_kernel<float>, dim3(blocks), dim3(256), 0, stream, a, items);
        else sb::launch(moe_glu_clamp_kernel<float>, dim3(blocks), dim3(256), 0, stream, a, items);
    } else if (dtype == SB_BF16) {
        if (wide) sb::launch(moe_glu_clamp_vec_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, a, items);
        else sb::launch(moe_glu_clamp_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, a, items);
    } else {
        SB_REQUIRE(false, "moe_glu_clamp: unknown dtype %d", dtype);
    }
    SB_LAUNCH_CHECK();
}

// in [N, experts * F] in the model dtype (or parts float32 [S, N, experts * F]); weights float32 [N, E_total].
extern "C" int sb_moe_act(void* out, const void* in, const float* parts, int S, long long part_stride, const float* weights,
                          int N, int E_total, int experts, int F, int dtype, cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && experts > 0 && experts <= E_total && F > 0, "moe_act: bad sizes N=%d experts=%d/%d F=%d", N,
               experts, E_total, F);
    SB_REQUIRE((in != nullptr) != (parts != nullptr), "moe_act: one input, a matrix or partial sums");
    SB_REQUIRE(dtype == SB_F32 || dtype == SB_BF16, "moe_act: unknown dtype %d", dtype);
    if (N == 0) return 0;
    MoeGluArgs a = {};
    a.in = in; a.parts = parts; a.S = S; a.part_stride = (size_t)part_stride; a.weights = weights; a.out = out;
    a.W = experts * F; a.E_total = E_total; a.experts = experts; a.F = F;
    const size_t total = (size_t)N * a.W;
    const int vec = dtype == SB_BF16 ? 8 : 4;
    const bool wide = F % vec == 0 && part_stride % 4 == 0 &&
                      ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(parts) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    const size_t items = wide ? total / vec : total;
    const dim3 blocks((int)((items + 255) / 256 < 148 * 16 ? (items + 255) / 256 : 148 * 16));
    if (dtype == SB_F32) {
        if (wide) sb::launch(moe_act_kernel<float, 4>, blocks, dim3(256), 0, stream, a, items);
        else sb::launch(moe_act_kernel<float, 1>, blocks, dim3(256), 0, stream, a, items);
    } else {
        if (wide) sb::launch(moe_act_kernel<__nv_bfloat16, 8>, blocks, dim3(256), 0, stream, a, items);
        else sb::launch(moe_act_kernel<__nv_bfloat16, 1>, blocks, dim3(256), 0, stream, a, items);
    }
    SB_LAUNCH_CHECK();
}

// logits float32 [N, E] = x [N, K] (model dtype) times router [E, K] (float32), transposed.
extern "C" int sb_moe_logits(float* logits, const void* x, const float* router, int N, int E, int K, int dtype,
                             cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && E > 0 && K > 0, "moe_logits: bad sizes N=%d E=%d K=%d", N, E, K);
    const size_t smem = (size_t)K * sizeof(float);
    SB_REQUIRE(smem <= 160 * 1024, "moe_logits: rows of %d values do not fit a block's shared memory", K);
    SB_REQUIRE((E + 3) / 4 <= 65535 && N <= 2147483647, "moe_logits: too many router outputs");
    if (N == 0) return 0;
    static sb::OncePerDevice once_f, once_b;
    if (dtype == SB_F32) {
        if (smem > 48 * 1024 && !once_f.flag()) {
            cudaFuncSetAttribute(moe_logits_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
            once_f.flag() = true;
        }
        sb::launch(moe_logits_kernel<float>, dim3(N, (E + 3) / 4), dim3(128), smem, stream, logits, (const float*)x, router, E, K);
    } else if (dtype == SB_BF16) {
        if (smem > 48 * 1024 && !once_b.flag()) {
            cudaFuncSetAttribute(moe_logits_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
            once_b.flag() = true;
        }
        sb::launch(moe_logits_kernel<__nv_bfloat16>, dim3(N, (E + 3) / 4), dim3(128), smem, stream, logits, (const __nv_bfloat16*)x,
                   router, E, K);
    } else {
        SB_REQUIRE(false, "moe_logits: unknown dtype %d", dtype);
    }
    SB_LAUNCH_CHECK();
}

// act [N, experts*F] in the model dtype; weights float32 [N, E_total], the experts' first.
extern "C" int sb_moe_scale(void* act, const float* weights, int N, int E_total, int experts, int F, int dtype,
                            cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && experts > 0 && experts <= E_total && F > 0, "moe_scale: bad sizes N=%d experts=%d/%d F=%d", N,
               experts, E_total, F);
    if (N == 0) return 0;
    const size_t total = (size_t)N * experts * F;
    const int vec = dtype == SB_BF16 ? 8 : 4;
    if (F % vec == 0 && (reinterpret_cast<uintptr_t>(act) & 15) == 0 && (dtype == SB_F32 || dtype == SB_BF16)) {
        const size_t tv = total / vec;
        const int vblocks = (int)((tv + 255) / 256 < 148 * 16 ? (tv + 255) / 256 : 148 * 16);
        if (dtype == SB_F32)
            sb::launch(moe_scale_vec_kernel<float>, dim3(vblocks), dim3(256), 0, stream, (float*)act, weights, E_total,
                       experts, F, tv);
        else
            sb::launch(moe_scale_vec_kernel<__nv_bfloat16>, dim3(vblocks), dim3(256), 0, stream, (__nv_bfloat16*)act,
                       weights, E_total, experts, F, tv);
        SB_LAUNCH_CHECK();
    }
    const int blocks = (int)((total + 255) / 256 < 148 * 8 ? (total + 255) / 256 : 148 * 8);
    if (dtype == SB_F32)
        sb::launch(moe_scale_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)act, weights, E_total, experts, F, total);
    else if (dtype == SB_BF16)
        sb::launch(moe_scale_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (__nv_bfloat16*)act, weights,
                   E_total, experts, F, total);
    else
        SB_REQUIRE(false, "moe_scale: unknown dtype %d", dtype);
    SB_LAUNCH_CHECK();
}

// slab float32 [N, d]; x [N, d] in the model dtype.
extern "C" int sb_moe_passthrough(float* slab, const void* x, const float* weights, int N, int E_total,
                                  int first_identity, int d, int dtype, cudaStream_t stream) {
    SB_REQUIRE(N >= 0 && d > 0 && first_identity >= 0 && first_identity <= E_total, "moe_passthrough: bad sizes");
    if (N == 0) return 0;
    if (dtype == SB_F32)
        sb::launch(moe_passthrough_kernel<float>, dim3(N), dim3(256), 0, stream, slab, (const float*)x, weights, E_total,
                   first_identity, d);
    else if (dtype == SB_BF16)
        sb::launch(moe_passthrough_kernel<__nv_bfloat16>, dim3(N), dim3(256), 0, stream, slab, (const __nv_bfloat16*)x,
                   weights, E_total, first_identity, d);
    else
        SB_REQUIRE(false, "moe_passthrough: unknown dtype %d", dtype);
    SB_LAUNCH_CHECK();
}
