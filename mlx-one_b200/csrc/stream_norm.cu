// Norms of the 32-bit stream fused with what is added to it before: nothing, a plain output, or an
// output that is normed itself first (a norm behind a part as well as ahead of the next one).
//
//   residual[t] += delta_scale * delta[t]                  (post_kind 0)
//   residual[t] += norm(delta[t]; post_weight, post_bias)  (post_kind 1 or 2)
//   out[t] = norm(residual[t]; weight, bias)               (kind 1 or 2)
//
// kind 1: x / sqrt(mean(x^2) + eps) * weight. kind 2: (x - mean) / sqrt(variance + eps) * weight +
// bias, the variance being the mean of the squared deviations, taken in a second pass over the
// values in registers. All sums are 32-bit in an order fixed by the row length.
#include "common.cuh"

namespace {

struct StreamNorm {
    const float* post_weight;
    const float* post_bias;
    const float* weight;
    const float* bias;
    int post_kind, kind;
    float post_eps, eps, delta_scale;
};

template <typename T>
__device__ __forceinline__ void load4(const T* p, float (&v)[4]);
template <>
__device__ __forceinline__ void load4<float>(const float* p, float (&v)[4]) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
}
template <>
__device__ __forceinline__ void load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&x.x);
    const __nv_bfloat162 hi = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
    v[0] = __low2float(lo); v[1] = __high2float(lo);
    v[2] = __low2float(hi); v[3] = __high2float(hi);
}
template <typename T>
__device__ __forceinline__ void store4(T* p, const float (&v)[4]);
template <>
__device__ __forceinline__ void store4<float>(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <>
__device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]);
    const __nv_bfloat162 hi = __floats2bfloat162_rn(v[2], v[3]);
    uint2 x;
    x.x = *reinterpret_cast<const uint32_t*>(&lo);
    x.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = x;
}

// Sum over the threads that share a row: a warp, or the block (one barrier a sum: the warps' sums
// lie in a row of `scratch` of their own for each of a kernel's sums, and every warp adds them up).
template <bool WARP>
__device__ __forceinline__ float row_sum(float v, float* scratch) {
    v = warp_sum(v);
    if (WARP) return v;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    return warp_sum(lane < warps ? scratch[lane] : 0.f);
}

// The weight and bias of a norm at this thread's places: held in registers (few rows: they are asked for
// before the kernel ahead has finished) or read where they are used.
template <int VEC, bool HELD>
struct Affine {
    float w[HELD ? VEC : 1][4], b[HELD ? VEC : 1][4];
    const float* weight;
    const float* bias;
    int hidden, first, step;

    __device__ __forceinline__ Affine(const float* weight_, const float* bias_, int hidden_, int first_, int step_)
        : weight(weight_), bias(bias_), hidden(hidden_), first(first_), step(step_) {
        if (HELD)
#pragma unroll
            for (int j = 0; j < VEC; ++j) fetch(j, w[HELD ? j : 0], b[HELD ? j : 0]);
    }
    __device__ __forceinline__ void fetch(int j, float (&wj)[4], float (&bj)[4]) const {
#pragma unroll
        for (int i = 0; i < 4; ++i) wj[i] = bj[i] = 0.f;
        if (first + j * step >= hidden) return;
        if (weight != nullptr) load4<float>(weight + first + j * step, wj);
        if (bias != nullptr) load4<float>(bias + first + j * step, bj);
    }
    __device__ __forceinline__ void apply(int j, float (&v)[4], float inv) const {
        if (HELD) {
#pragma unroll
            for (int i = 0; i < 4; ++i) v[i] = fmaf(v[i] * inv, w[HELD ? j : 0][i], b[HELD ? j : 0][i]);
        } else {
            float wj[4], bj[4];
            fetch(j, wj, bj);
#pragma unroll
            for (int i = 0; i < 4; ++i) v[i] = fmaf(v[i] * inv, wj[i], bj[i]);
        }
    }
};

// Norms this thread's share of a row in place. `scratch`: two rows of 32 floats.
template <int VEC, bool WARP, bool HELD>
__device__ __forceinline__ void norm_row(float (&v)[VEC][4], int hidden, int first, int step, int kind,
                                         float eps, const Affine<VEC, HELD>& affine, float* scratch) {
    float mean = 0.f;
    if (kind == 2) {
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < VEC; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) sum += v[j][i];             // (values beyond the row are 0)
        mean = row_sum<WARP>(sum, scratch) / (float)hidden;
    }
    float squares = 0.f;
#pragma unroll
    for (int j = 0; j < VEC; ++j)
        if (first + j * step < hidden)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                v[j][i] -= mean;
                squares = fmaf(v[j][i], v[j][i], squares);
            }
    const float inv = 1.f / sqrtf(row_sum<WARP>(squares, scratch + 32) / (float)hidden + eps);
#pragma unroll
    for (int j = 0; j < VEC; ++j) affine.apply(j, v[j], inv);
}

// One row per block (WARP false) or per warp (WARP true), the row in registers: 4 VEC values a thread.
template <typename T, int VEC, bool WARP, bool HELD>
__global__ void __launch_bounds__(WARP ? 256 : HELD ? 1024 : 512)
stream_norm_kernel(float* __restrict__ residual, const T* __restrict__ delta, T* __restrict__ out,
                   int rows, int hidden, StreamNorm n) {
    __shared__ float scratch[4 * 32];
    griddep_launch();
    const int threads = WARP ? 32 : blockDim.x;
    const int row = WARP ? blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.x;
    const int first = (WARP ? (threadIdx.x & 31) : threadIdx.x) * 4, step = threads * 4;
    // the norms' weights do not depend on the kernel before this one
    const Affine<VEC, HELD> post(n.post_weight, n.post_bias, hidden, first, step);
    const Affine<VEC, HELD> next(n.weight, n.bias, hidden, first, step);
    griddep_wait();
    delta = settled(delta);
    if (row >= rows) return;                      // (whole warps; a block has one row)
    const size_t base = (size_t)row * hidden;
    float x[VEC][4], y[VEC][4];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
#pragma unroll
        for (int i = 0; i < 4; ++i) x[j][i] = y[j][i] = 0.f;
        if (first + j * step < hidden) {
            load4<float>(residual + base + first + j * step, x[j]);
            if (delta != nullptr) load4<T>(delta + base + first + j * step, y[j]);
        }
    }
    if (delta != nullptr) {
        float factor = n.delta_scale;
        if (n.post_kind != 0) {
            norm_row<VEC, WARP, HELD>(y, hidden, first, step, n.post_kind, n.post_eps, post, scratch);
            factor = 1.f;
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j)
            if (first + j * step < hidden) {
#pragma unroll
                for (int i = 0; i < 4; ++i) x[j][i] = fmaf(factor, y[j][i], x[j][i]);
                store4<float>(residual + base + first + j * step, x[j]);
            }
    }
    norm_row<VEC, WARP, HELD>(x, hidden, first, step, n.kind, n.eps, next, scratch + 64);
#pragma unroll
    for (int j = 0; j < VEC; ++j)
        if (first + j * step < hidden) store4<T>(out + base + first + j * step, x[j]);
}

// Any row length: one block per row, the values read again for every pass.
template <typename T>
__global__ void stream_norm_any_kernel(float* __restrict__ residual, const T* __restrict__ delta,
                                       T* __restrict__ out, int hidden, StreamNorm n) {
    __shared__ float scratch[33];
    griddep_launch();
    griddep_wait();
    delta = settled(delta);
    const size_t base = (size_t)blockIdx.x * hidden;
    auto moments = [&](auto value, int kind, float eps, float& mean) {
        float sum = 0.f;
        mean = 0.f;
        if (kind == 2) {
            for (int c = threadIdx.x; c < hidden; c += blockDim.x) sum += value(c);
            mean = block_sum(sum, scratch) / (float)hidden;
        }
        float squares = 0.f;
        for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
            const float d = value(c) - mean;
            squares = fmaf(d, d, squares);
        }
        return 1.f / sqrtf(block_sum(squares, scratch) / (float)hidden + eps);
    };
    float mean;
    if (delta != nullptr && n.post_kind == 0) {
        for (int c = threadIdx.x; c < hidden; c += blockDim.x)
            residual[base + c] = fmaf(n.delta_scale, to_float<T>(delta[base + c]), residual[base + c]);
    } else if (delta != nullptr) {
        const float inv = moments([&](int c) { return to_float<T>(delta[base + c]); }, n.post_kind,
                                  n.post_eps, mean);
        for (int c = threadIdx.x; c < hidden; c += blockDim.x)
            residual[base + c] += fmaf((to_float<T>(delta[base + c]) - mean) * inv, n.post_weight[c],
                                       n.post_bias != nullptr ? n.post_bias[c] : 0.f);
    }
    // (a thread reads back only what it wrote itself)
    const float inv = moments([&](int c) { return residual[base + c]; }, n.kind, n.eps, mean);
    for (int c = threadIdx.x; c < hidden; c += blockDim.x)
        out[base + c] = from_float<T>(fmaf((residual[base + c] - mean) * inv, n.weight[c],
                                           n.bias != nullptr ? n.bias[c] : 0.f));
}

template <typename T>
cudaError_t launch(float* residual, const void* delta, void* out, int rows, int hidden,
                   const StreamNorm& n, cudaStream_t stream) {
    auto aligned16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool aligned = hidden % 4 == 0 && aligned16(residual) && aligned16(delta) && aligned16(out) &&
                         aligned16(n.weight) && aligned16(n.bias) && aligned16(n.post_weight) &&
                         aligned16(n.post_bias);
    const T* d = (const T*)delta;
    T* o = (T*)out;
#define ROWS(VEC, HELD)                                                                             \
    launch_kernel(stream_norm_kernel<T, VEC, false, HELD>, dim3(rows), dim3(threads), 0, stream,    \
                  true, residual, d, o, rows, hidden, n)
#define WARPS(VEC)                                                                                  \
    launch_kernel(stream_norm_kernel<T, VEC, true, false>, dim3((rows + 7) / 8), dim3(256), 0,      \
                  stream, true, residual, d, o, rows, hidden, n)
    if (aligned && rows >= 1536 && hidden <= 512) {
        if (hidden <= 256) return WARPS(2);
        return WARPS(4);
    }
    if (aligned && hidden <= 8192) {
        // many rows: fewer threads a row and more rows at a time; few rows: as many threads as there are
        const int quads = hidden / 4;
        const bool many = rows >= 592 && quads > 64;
        const int each = many && quads > 1024 ? 4 : many || quads > 1024 ? 2 : 1;
        const int threads = ((quads + each - 1) / each + 31) / 32 * 32;
        if (each == 1) return ROWS(1, true);
        if (each == 2) return many ? ROWS(2, false) : ROWS(2, true);
        return ROWS(4, false);
    }
#undef ROWS
#undef WARPS
    const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
    return launch_kernel(stream_norm_any_kernel<T>, dim3(rows), dim3(threads), 0, stream, true, residual,
                         d, o, hidden, n);
}

}  // namespace

// See the head of this file. delta may be null. post_bias and bias may be null (kind 1 has none).
MLXONE_API int mlxone_stream_norm(float* residual, const void* delta, float delta_scale,
                                  const float* post_weight, const float* post_bias, int post_kind,
                                  float post_eps, const float* weight, const float* bias, int kind,
                                  float eps, void* out, int rows, int hidden, int dtype,
                                  cudaStream_t stream) {
    if (rows == 0) return 0;
    MLXONE_REQUIRE(rows > 0 && hidden > 0, "stream_norm: bad sizes");
    MLXONE_REQUIRE((kind == 1 || kind == 2) && post_kind >= 0 && post_kind <= 2,
                   "stream_norm: unknown norm %d or %d", kind, post_kind);
    MLXONE_REQUIRE(weight != nullptr && (post_kind == 0 || (post_weight != nullptr && delta != nullptr)),
                   "stream_norm: a norm has a weight");
    StreamNorm n{post_weight, post_bias, weight, bias, post_kind, kind, post_eps, eps, delta_scale};
    const cudaError_t err = dtype == MLXONE_BF16
                                ? launch<__nv_bfloat16>(residual, delta, out, rows, hidden, n, stream)
                                : launch<float>(residual, delta, out, rows, hidden, n, stream);
    if (err != cudaSuccess) {
        mlxone_set_error("stream_norm: launch failed: %s", cudaGetErrorString(err));
        return 2;
    }
    MLXONE_LAUNCH_CHECK("stream_norm");
    return 0;
}
