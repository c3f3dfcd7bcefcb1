// What may happen to an attention score between the product and the softmax: a cap, c tanh(s / c),
// and a bias that falls with the distance between query and key, slope_h (i - j), taken off after
// the cap. The attention kernels are built with and without it (a template parameter), and the
// shaped ones hand their softmax scores in units of log2 e.
#pragma once

#include "common.cuh"

struct ScoreShape {
    // in: a raw product q . k times this is the tanh's argument (scale / cap); without a cap unused
    float inner = 0.f;
    // the cap times log2 e; 0: no cap
    float outer = 0.f;
    // scale * log2 e, for scores without a cap
    float plain = 0.f;
    // float32 [heads] or null: the slopes
    const float* slopes = nullptr;
    // With a cap a key so far back that its weight is below 2^-126 of the query's own is not read at
    // all: how many keys' worth of a slope of 1 that takes, (2 cap + 126 ln 2) (0: keep every key).
    float reach = 0.f;
};

static inline ScoreShape make_score_shape(float scale, float cap, const float* slopes) {
    constexpr float log2e = 1.4426950408889634f;
    ScoreShape shape;
    shape.plain = scale * log2e;
    if (cap > 0.f) {
        shape.inner = scale / cap;
        shape.outer = cap * log2e;
        if (slopes != nullptr) shape.reach = 2.f * cap + 126.f * 0.6931472f;
    }
    shape.slopes = slopes;
    return shape;
}

// The keys that a query of these heads reads, as a window (0: all). The weight of a key at distance d
// is at most exp(cap - slope d) while the query's own key has at least exp(-cap): beyond reach /
// slope their quotient is below the smallest normal number and the kernels' exponential gives 0.
__device__ __forceinline__ int shape_window(const ScoreShape& shape, int first_head, int heads) {
    if (shape.reach <= 0.f) return 0;
    float least = INFINITY;
    for (int h = 0; h < heads; ++h) least = fminf(least, shape.slopes[first_head + h]);
    if (!(least > 0.f)) return 0;
    const float keys = ceilf(shape.reach / least) + 1.f;
    return keys < 1e9f ? (int)keys : 0;
}

// tanh(t) = t P(t^2) for |t| <= 1: P of degree 5 fitted to the smallest largest relative error
// (6e-7) by reweighted least squares.
#define MLXONE_TANH_C0 0.9999994039535522f
#define MLXONE_TANH_C1 -0.3332904279232025f
#define MLXONE_TANH_C2 0.13281431794166565f
#define MLXONE_TANH_C3 -0.05160561203956604f
#define MLXONE_TANH_C4 0.016743037849664688f
#define MLXONE_TANH_C5 -0.0030670284759253263f

// ... and for |t| <= 1/2, of degree 3 (5.5e-7)
#define MLXONE_TANH_HALF_C0 0.999999463558197f
#define MLXONE_TANH_HALF_C1 -0.33326318860054016f
#define MLXONE_TANH_HALF_C2 0.13190296292304993f
#define MLXONE_TANH_HALF_C3 -0.04440220445394516f

__device__ __forceinline__ float tanh_small(float t) {
    const float x = t * t;
    float p = fmaf(x, MLXONE_TANH_C5, MLXONE_TANH_C4);
    p = fmaf(x, p, MLXONE_TANH_C3);
    p = fmaf(x, p, MLXONE_TANH_C2);
    p = fmaf(x, p, MLXONE_TANH_C1);
    p = fmaf(x, p, MLXONE_TANH_C0);
    return t * p;
}
// 1 - 2 / (1 + e^(2t)), for any t: absolute error of a few units of 2^-24
__device__ __forceinline__ float tanh_any(float t) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(t * 2.8853900817779268f));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
    return fmaf(-2.f, r, 1.f);
}

// Raw products of one thread -> scores in units of log2 e without the distance bias. All lanes of
// the warp come here together (they take the short way together).
template <int N>
__device__ __forceinline__ void shape_scores(float (&v)[N], const ScoreShape& shape) {
    if (shape.outer == 0.f) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] *= shape.plain;
        return;
    }
    float top = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) top = fmaxf(top, fabsf(v[i]));
    if (__any_sync(0xffffffffu, top * fabsf(shape.inner) > 1.f)) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = shape.outer * tanh_any(v[i] * shape.inner);
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = shape.outer * tanh_small(v[i] * shape.inner);
    }
}
