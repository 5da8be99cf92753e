// What may happen to an attention score between the product and the softmax, and which keys a query sees.
//
//   s <- s * scale ;  s <- cap * tanh(s / cap)  (cap > 0) ;  s <- s - slope_h * (i - j)  (slopes given)
//   keys j <= i, and of these: the last `window` (window > 0), or those of i's own chunk,
//   floor(j / chunk) = floor(i / chunk) (chunk > 0; chunks count from position 0 of the sequence), or all
#pragma once

#include "common.cuh"

namespace sb {

struct ScoreMap {
    float cap;              // 0: not capped
    const float* slopes;    // [Hq], not negative, or null
    int chunk;              // 0: no chunks

    __host__ __device__ bool maps_scores() const { return cap > 0.f || slopes != nullptr; }
};

// The first position that a query at `pos` sees.
__host__ __device__ __forceinline__ int first_visible(int pos, int window, int chunk) {
    if (chunk > 0) return pos - pos % chunk;
    return (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;
}

// One query row's constants of the map, for scores in units of log2 (softmax weights are 2^s then):
//   capped:   cap * tanh(z) = cap - 2 cap / (1 + e^{2z}), z = raw * scale / cap, in hardware ex2 and reciprocal.
//             Its absolute error is a few 1e-7 of the cap, whatever the score's size.
//   otherwise raw * scale.
// and then + slope * (j - i).
struct RowScores {
    float in, cap, slope, base;
    bool capped;

    __device__ __forceinline__ void set(const ScoreMap& m, float scale, int h) {
        constexpr float LOG2 = 1.4426950408889634f;
        capped = m.cap > 0.f;
        cap = m.cap * LOG2;
        in = capped ? scale / m.cap * (2.0f * LOG2) : scale * LOG2;
        slope = m.slopes != nullptr ? m.slopes[h] * LOG2 : 0.f;
        base = 0.f;
    }
    // the keys that follow are counted from one that is `ahead` = key position - query position away
    __device__ __forceinline__ void from(float ahead) { base = fmaf(slope, ahead, capped ? cap : 0.f); }

    __device__ __forceinline__ float plain(float raw, float offset) const { return fmaf(raw, in, fmaf(slope, offset, base)); }
    __device__ __forceinline__ float with_cap(float raw, float offset) const {
        float e, r;
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(raw * in));
        asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
        return fmaf(-2.0f * cap, r, fmaf(slope, offset, base));
    }
    __device__ __forceinline__ float operator()(float raw, float offset) const {
        return capped ? with_cap(raw, offset) : plain(raw, offset);
    }
};

}  // namespace sb
