// Parallel residual streams (hyper-connections).
//
// A token has n streams X_1 .. X_n of `hidden` 32-bit values. A sublayer reads u = sum_s read[s]
// X_s, and its output y is written back as X_t <- sum_s mix[s, t] X_s + out[t] y, all streams at
// once from the old ones. read_streams stands between two sublayers: it writes the last one's
// output into the streams, reads the next one's input from them and norms it (root mean square,
// 32-bit), so every stream passes through the GPU once per sublayer. Before the first write
// there is one stream that stands for all n (n_in = 1); the write then makes n of it.
// sum_streams: what follows the last layer, the wanted rows' streams added up, with the pending
// write folded into one weight per stream.
#include "common.cuh"

namespace {

constexpr int MAX_STREAMS = 16;

template <typename T> struct Four;
template <> struct Four<float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
};
template <> struct Four<__nv_bfloat16> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.y));
        v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]);
        const __nv_bfloat162 hi = __floats2bfloat162_rn(v[2], v[3]);
        uint2 x;
        x.x = *reinterpret_cast<const uint32_t*>(&lo);
        x.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = x;
    }
};

// The weights of one write and read, in shared memory: mix [n_in][n_out], out [n_out], read.
struct Weights {
    float mix[MAX_STREAMS * MAX_STREAMS], out[MAX_STREAMS], read[MAX_STREAMS];
};

__device__ __forceinline__ void stage_weights(Weights& to, const float* mix, const float* out,
                                              const float* read, int n_in, int n_out, bool update) {
    if (update) {
        for (int i = threadIdx.x; i < n_in * n_out; i += blockDim.x) to.mix[i] = mix[i];
        for (int i = threadIdx.x; i < n_out; i += blockDim.x) to.out[i] = out[i];
    }
    for (int i = threadIdx.x; i < n_out; i += blockDim.x) to.read[i] = read[i];
}

// One block per token, four neighbouring values a thread and pass (hidden <= 4 * blockDim.x *
// PASSES, a multiple of 4). y null: nothing is pending, the streams stay (n_out = n_in).
// `after` may be `before` (n_out = n_in): a thread reads all its values before it writes any.
template <typename T, int S, int PASSES>
__global__ void __launch_bounds__(1024)
read_streams_kernel(const float* before, float* after, const T* __restrict__ y,
                    const float* __restrict__ mix, const float* __restrict__ out,
                    const float* __restrict__ read, const float* __restrict__ norm_weight,
                    T* __restrict__ normed, int n_in, int n_out, int hidden, float eps) {
    __shared__ Weights w;
    __shared__ float scratch[33];
    griddep_launch();
    // (weights do not depend on the kernel before this one)
    stage_weights(w, mix, out, read, n_in, n_out, y != nullptr);
    float scale[PASSES][4];
#pragma unroll
    for (int pass = 0; pass < PASSES; ++pass) {
        const int c = (pass * blockDim.x + threadIdx.x) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) scale[pass][i] = 0.f;
        if (c < hidden) Four<float>::load(norm_weight + c, scale[pass]);
    }
    __syncthreads();
    griddep_wait();
    before = settled(before);
    y = settled(y);
    const size_t t = blockIdx.x;
    float x[PASSES][S][4], add[PASSES][4], u[PASSES][4];
#pragma unroll
    for (int pass = 0; pass < PASSES; ++pass) {
        const int c = (pass * blockDim.x + threadIdx.x) * 4;
        const bool live = c < hidden;
#pragma unroll
        for (int s = 0; s < S; ++s) {
#pragma unroll
            for (int i = 0; i < 4; ++i) x[pass][s][i] = 0.f;
            if (live && s < n_in) Four<float>::load(before + (t * n_in + s) * hidden + c, x[pass][s]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) add[pass][i] = u[pass][i] = 0.f;
        if (live && y != nullptr) Four<T>::load(y + t * hidden + c, add[pass]);
    }
    float squares = 0.f;
#pragma unroll
    for (int pass = 0; pass < PASSES; ++pass) {
        const int c = (pass * blockDim.x + threadIdx.x) * 4;
        if (y != nullptr) {
#pragma unroll
            for (int to = 0; to < S; ++to) {
                if (to >= n_out) break;
                float v[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) v[i] = w.out[to] * add[pass][i];
#pragma unroll
                for (int s = 0; s < S; ++s) {
                    if (s >= n_in) break;
                    const float factor = w.mix[s * n_out + to];
#pragma unroll
                    for (int i = 0; i < 4; ++i) v[i] = fmaf(factor, x[pass][s][i], v[i]);
                }
                if (c < hidden) Four<float>::store(after + (t * n_out + to) * hidden + c, v);
#pragma unroll
                for (int i = 0; i < 4; ++i) u[pass][i] = fmaf(w.read[to], v[i], u[pass][i]);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) {
                if (s >= n_in) break;
#pragma unroll
                for (int i = 0; i < 4; ++i) u[pass][i] = fmaf(w.read[s], x[pass][s][i], u[pass][i]);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) squares = fmaf(u[pass][i], u[pass][i], squares);
    }
    const float inv = rsqrtf(block_sum(squares, scratch) / (float)hidden + eps);
#pragma unroll
    for (int pass = 0; pass < PASSES; ++pass) {
        const int c = (pass * blockDim.x + threadIdx.x) * 4;
        if (c >= hidden) continue;
        float v[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = u[pass][i] * inv * scale[pass][i];
        Four<T>::store(normed + t * hidden + c, v);
    }
}

// The same for any width and up to MAX_STREAMS streams (also rows that would fill more registers
// than a thread has): a value a thread and turn, u in dynamic shared memory [hidden].
template <typename T>
__global__ void __launch_bounds__(256)
read_streams_any_kernel(const float* before, float* after, const T* __restrict__ y,
                        const float* __restrict__ mix, const float* __restrict__ out,
                        const float* __restrict__ read, const float* __restrict__ norm_weight,
                        T* __restrict__ normed, int n_in, int n_out, int hidden, float eps) {
    extern __shared__ float u[];
    __shared__ Weights w;
    __shared__ float scratch[33];
    griddep_launch();
    stage_weights(w, mix, out, read, n_in, n_out, y != nullptr);
    __syncthreads();
    griddep_wait();
    before = settled(before);
    y = settled(y);
    const size_t t = blockIdx.x;
    float squares = 0.f;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        float x[MAX_STREAMS];
        float sum = 0.f;
#pragma unroll
        for (int s = 0; s < MAX_STREAMS; ++s) x[s] = s < n_in ? before[(t * n_in + s) * hidden + c] : 0.f;
        if (y != nullptr) {
            const float add = to_float<T>(y[t * hidden + c]);
            for (int to = 0; to < n_out; ++to) {
                float v = w.out[to] * add;
#pragma unroll
                for (int s = 0; s < MAX_STREAMS; ++s)
                    if (s < n_in) v = fmaf(w.mix[s * n_out + to], x[s], v);
                after[(t * n_out + to) * hidden + c] = v;
                sum = fmaf(w.read[to], v, sum);
            }
        } else {
#pragma unroll
            for (int s = 0; s < MAX_STREAMS; ++s)
                if (s < n_in) sum = fmaf(w.read[s], x[s], sum);
        }
        u[c] = sum;
        squares = fmaf(sum, sum, squares);
    }
    const float inv = rsqrtf(block_sum(squares, scratch) / (float)hidden + eps);
    for (int c = threadIdx.x; c < hidden; c += blockDim.x)
        normed[t * hidden + c] = from_float<T>(u[c] * inv * norm_weight[c]);
}

// out[i, :] = sum_s (sum_t mix[s, t]) X_s + (sum_t out[t]) y of token rows[i] (rows null: token i)
template <typename T>
__global__ void __launch_bounds__(256)
sum_streams_kernel(const float* __restrict__ streams, const T* __restrict__ y,
                   const float* __restrict__ mix, const float* __restrict__ out,
                   const int* __restrict__ rows, float* __restrict__ total, int n_in, int n_out,
                   int hidden, int tokens, int wide) {
    __shared__ float factor[MAX_STREAMS + 1];
    griddep_launch();
    if (threadIdx.x <= n_in) {
        const int s = threadIdx.x;
        float sum = 0.f;
        if (y == nullptr) sum = s < n_in ? 1.f : 0.f;
        else for (int to = 0; to < n_out; ++to) sum += s < n_in ? mix[s * n_out + to] : out[to];
        factor[s] = sum;
    }
    __syncthreads();
    griddep_wait();
    streams = settled(streams);
    y = settled(y);
    rows = settled(rows);
    const int i = blockIdx.x;
    const int t = rows != nullptr ? rows[i] : i;
    if (t < 0 || t >= tokens) return;
    if (wide) {
        // four values a load, the streams' loads on their way together
        for (int c = threadIdx.x * 4; c < hidden; c += blockDim.x * 4) {
            float sum[4] = {0.f, 0.f, 0.f, 0.f};
            if (y != nullptr) {
                Four<T>::load(y + (size_t)t * hidden + c, sum);
#pragma unroll
                for (int k = 0; k < 4; ++k) sum[k] *= factor[n_in];
            }
#pragma unroll 4
            for (int s = 0; s < n_in; ++s) {
                float x[4];
                Four<float>::load(streams + ((size_t)t * n_in + s) * hidden + c, x);
#pragma unroll
                for (int k = 0; k < 4; ++k) sum[k] = fmaf(factor[s], x[k], sum[k]);
            }
            Four<float>::store(total + (size_t)i * hidden + c, sum);
        }
        return;
    }
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
        float sum = y != nullptr ? factor[n_in] * to_float<T>(y[(size_t)t * hidden + c]) : 0.f;
        for (int s = 0; s < n_in; ++s)
            sum = fmaf(factor[s], streams[((size_t)t * n_in + s) * hidden + c], sum);
        total[(size_t)i * hidden + c] = sum;
    }
}

template <typename T>
int launch_read(const float* before, float* after, const void* y, const float* mix, const float* out,
                const float* read, const float* norm_weight, void* normed, int tokens, int n_in,
                int n_out, int hidden, float eps, cudaStream_t stream) {
    const auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const int streams = n_in > n_out ? n_in : n_out;
    const bool four = hidden % 4 == 0 && aligned(before) && aligned(after) && aligned(y) &&
                      aligned(norm_weight) && aligned(normed);
    // (the block's shape follows the width alone, so a token's sums never change order)
    const int quads = hidden / 4;
    const int passes = quads <= 1024 ? 1 : 2;
    if (four && (streams <= 4 || (streams <= 8 && passes == 1)) && quads <= 2048) {
        const int per_pass = (quads + passes - 1) / passes;
        const int threads = (per_pass + 31) / 32 * 32;
#define READ(S, PASSES)                                                                          \
    launch_kernel(read_streams_kernel<T, S, PASSES>, dim3(tokens), dim3(threads), 0, stream, true, \
                  before, after, (const T*)y, mix, out, read, norm_weight, (T*)normed, n_in, n_out, \
                  hidden, eps)
#define READ_PASSES(S)                   \
    do {                                 \
        if (passes == 1) READ(S, 1);     \
        else READ(S, 2);                 \
    } while (0)
        if (streams == 1) READ_PASSES(1);
        else if (streams == 2) READ_PASSES(2);
        else if (streams == 3) READ_PASSES(3);
        else if (streams == 4) READ_PASSES(4);
        else READ(8, 1);
#undef READ_PASSES
#undef READ
    } else {
        const size_t shared = (size_t)hidden * sizeof(float);
        MLXONE_REQUIRE(shared <= 200 * 1024, "read_streams: rows of %d values do not fit", hidden);
        if (shared > 40 * 1024)
            cudaFuncSetAttribute(read_streams_any_kernel<T>,
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
        launch_kernel(read_streams_any_kernel<T>, dim3(tokens), dim3(256), shared, stream, true,
                      before, after, (const T*)y, mix, out, read, norm_weight, (T*)normed, n_in,
                      n_out, hidden, eps);
    }
    MLXONE_LAUNCH_CHECK("read_streams");
    return 0;
}

}  // namespace

MLXONE_API int mlxone_read_streams_max() { return MAX_STREAMS; }

// before [tokens, n_in, hidden], after [tokens, n_out, hidden] (unused without y), y and normed
// [tokens, hidden] in the compute type; mix [n_in, n_out], out [n_out], read [n_out] (n_in = n_out
// without y).
MLXONE_API int mlxone_read_streams(const float* before, float* after, const void* y,
                                   const float* mix, const float* out, const float* read,
                                   const float* norm_weight, void* normed, int tokens, int n_in,
                                   int n_out, int hidden, float eps, int dtype, cudaStream_t stream) {
    if (tokens == 0) return 0;
    MLXONE_REQUIRE(tokens > 0 && hidden > 0 && n_in >= 1 && n_out >= 1 && n_in <= MAX_STREAMS &&
                       n_out <= MAX_STREAMS, "read_streams: 1 to %d streams", MAX_STREAMS);
    MLXONE_REQUIRE(y != nullptr || n_in == n_out, "read_streams: nothing is written");
    MLXONE_REQUIRE(before != after || n_in == n_out, "read_streams: in place with other streams");
    return dtype == MLXONE_BF16
        ? launch_read<__nv_bfloat16>(before, after, y, mix, out, read, norm_weight, normed, tokens,
                                     n_in, n_out, hidden, eps, stream)
        : launch_read<float>(before, after, y, mix, out, read, norm_weight, normed, tokens, n_in,
                             n_out, hidden, eps, stream);
}

MLXONE_API int mlxone_sum_streams(const float* streams, const void* y, const float* mix,
                                  const float* out, const int* rows, float* total, int count,
                                  int tokens, int n_in, int n_out, int hidden, int dtype,
                                  cudaStream_t stream) {
    if (count == 0) return 0;
    MLXONE_REQUIRE(count > 0 && tokens > 0 && hidden > 0 && n_in >= 1 && n_in <= MAX_STREAMS &&
                       n_out >= 1 && n_out <= MAX_STREAMS, "sum_streams: 1 to %d streams", MAX_STREAMS);
    const auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const int wide = hidden % 4 == 0 && aligned(streams) && aligned(y) && aligned(total);
    if (dtype == MLXONE_BF16)
        launch_kernel(sum_streams_kernel<__nv_bfloat16>, dim3(count), dim3(256), 0, stream, true,
                      streams, (const __nv_bfloat16*)y, mix, out, rows, total, n_in, n_out, hidden,
                      tokens, wide);
    else
        launch_kernel(sum_streams_kernel<float>, dim3(count), dim3(256), 0, stream, true, streams,
                      (const float*)y, mix, out, rows, total, n_in, n_out, hidden, tokens, wide);
    MLXONE_LAUNCH_CHECK("sum_streams");
    return 0;
}
