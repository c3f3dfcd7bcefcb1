// Attention over one latent row per token, and attention with two score maps per head: the
// steps around the attention kernels.
//
// latent_prepare: from the fused input product of a latent-attention mixer to the queries'
// rotated parts and the token's row [latent | rotated shared key part] in its request's pages;
// also in two steps, for queries that come out of a latent of their own (latent_rows: the page's
// row and the queries' latent, normed; latent_queries: the rotated parts).
// sigmoid_gate: values * sigmoid(gate). differential_combine: o = a1 - mix * a2 per head, divided
// by its root mean square, times a factor.
#include "common.cuh"

namespace {

// One block per token; every source has rows of its own stride. q_source (null: this part is left
// out): heads * (head_dim + rot_dim) query values, head by head, the rotated part last; queries
// [tokens, heads, latent + rot_dim]: only the last rot_dim values of every head are written here
// (the first `latent` are another product's output). small_source (null: left out): `rank` values,
// of which small [tokens, rank] gets the normed ones (times small_weight). down_source (null: left
// out): latent + rot_dim values of the down product. The page row [latent + rot_dim] gets the latent divided by its root mean square
// times `norm_weight`, and the rotated shared key part. Rotation: the first `rotary_dim` values
// of a rotated part; pair i is (2i, 2i + 1) if `neighbours`, else (i, i + rotary_dim / 2); cosine
// and sine are multiplied by `amplitude`.
// Dynamic shared memory: rotary_dim floats (cosines and sines).
template <typename T>
__global__ void __launch_bounds__(512)
latent_prepare_kernel(const T* __restrict__ q_source, int ld_q, T* __restrict__ queries,
                      const T* __restrict__ small_source, int ld_small,
                      const float* __restrict__ small_weight, T* __restrict__ small, int rank,
                      const T* __restrict__ down_source, int ld_down,
                      const float* __restrict__ norm_weight, float eps,
                      const float* __restrict__ inv_freq, int rotary_dim, float amplitude,
                      int neighbours,
                      const int* __restrict__ positions, const int* __restrict__ token_request,
                      T* __restrict__ pages, const int* __restrict__ block_table, int table_width,
                      int page_size, int heads, int head_dim, int rot_dim, int latent, int write,
                      int* __restrict__ error_flag) {
    extern __shared__ float shared[];
    __shared__ float scratch[33];
    griddep_launch();
    griddep_wait();
    q_source = settled(q_source);
    small_source = settled(small_source);
    down_source = settled(down_source);
    const int t = blockIdx.x;
    // (two blocks a token: the second has the queries' latent, the first the rest)
    if (gridDim.y == 2 && blockIdx.y == 0) small_source = nullptr;
    if (gridDim.y == 2 && blockIdx.y == 1) {
        q_source = nullptr;
        down_source = nullptr;
        rotary_dim = 0;
    }
    const int position = positions[t];
    const int half = rotary_dim / 2;
    float* cosines = shared;
    float* sines = shared + half;
    for (int j = threadIdx.x; j < half; j += blockDim.x) {
        float sine, cosine;
        sincosf((float)position * inv_freq[j], &sine, &cosine);
        sines[j] = sine * amplitude;
        cosines[j] = cosine * amplitude;
    }
    __syncthreads();
    const int per_head = head_dim + rot_dim;
    const int row = latent + rot_dim;
    // value e of a rotated part that starts at `part`
    auto rotated = [&](const T* part, int e) -> float {
        const float v = to_float<T>(part[e]);
        if (e >= rotary_dim) return v;
        int pair, other;
        bool first;
        if (neighbours) {
            pair = e >> 1; first = (e & 1) == 0; other = e ^ 1;
        } else {
            first = e < half; pair = first ? e : e - half; other = first ? e + half : e - half;
        }
        const float w = to_float<T>(part[other]);
        // (u, v) -> (u cos - v sin, v cos + u sin)
        return first ? v * cosines[pair] - w * sines[pair] : v * cosines[pair] + w * sines[pair];
    };
    if (q_source != nullptr) {
        const T* source = q_source + (size_t)t * ld_q;
#pragma unroll 4
        for (int i = threadIdx.x; i < heads * rot_dim; i += blockDim.x) {
            const int head = i / rot_dim, e = i % rot_dim;
            queries[((size_t)t * heads + head) * row + latent + e] =
                from_float<T>(rotated(source + (size_t)head * per_head + head_dim, e));
        }
    }
    if (small_source != nullptr) {
        const T* source = small_source + (size_t)t * ld_small;
        float squares = 0.f;
        for (int e = threadIdx.x; e < rank; e += blockDim.x) {
            const float v = to_float<T>(source[e]);
            squares = fmaf(v, v, squares);
        }
        squares = block_sum(squares, scratch);
        const float inv = rsqrtf(squares / (float)rank + eps);
        for (int e = threadIdx.x; e < rank; e += blockDim.x)
            small[(size_t)t * rank + e] = from_float<T>(to_float<T>(source[e]) * inv * small_weight[e]);
    }
    if (!write || down_source == nullptr) return;
    const int r = token_request[t];
    const int block = position / page_size;
    const int page = block < table_width ? block_table[(size_t)r * table_width + block] : -1;
    if (page < 0) {
        if (threadIdx.x == 0) atomicExch(error_flag, 2);
        return;
    }
    T* dst = pages + ((size_t)page * page_size + position % page_size) * row;
    const T* down = down_source + (size_t)t * ld_down;
    float squares = 0.f;
    for (int e = threadIdx.x; e < latent; e += blockDim.x) {
        const float v = to_float<T>(down[e]);
        squares = fmaf(v, v, squares);
    }
    squares = block_sum(squares, scratch);
    const float inv = rsqrtf(squares / (float)latent + eps);
    for (int e = threadIdx.x; e < latent; e += blockDim.x)
        dst[e] = from_float<T>(to_float<T>(down[e]) * inv * norm_weight[e]);
    for (int e = threadIdx.x; e < rot_dim; e += blockDim.x)
        dst[latent + e] = from_float<T>(rotated(down + latent, e));
}

// Few tokens: the queries against the latents in one kernel. Grid (heads, tiles of 64 latent columns
// + 1): queries[t, h, n] = up_k[h, n, :] . q[t, h, :head_dim] for the tile's columns n, two threads
// a column with half of the products each, the matrix's rows asked for before the wait; the last
// block of a head rotates its queries' rotated parts. head_dim a multiple of 16 up to 128, at most
// TOKENS tokens.
constexpr int ABSORB_COLUMNS = 64, ABSORB_PIECES = 8;

template <int TOKENS>
__global__ void __launch_bounds__(2 * ABSORB_COLUMNS)
latent_absorb_kernel(const __nv_bfloat16* __restrict__ q, int ld, const __nv_bfloat16* __restrict__ up_k,
                     __nv_bfloat16* __restrict__ queries, const float* __restrict__ inv_freq,
                     int rotary_dim, float amplitude, int neighbours, const int* __restrict__ positions,
                     int tokens, int heads, int head_dim, int rot_dim, int latent) {
    using T = __nv_bfloat16;
    __shared__ __align__(16) float staged[TOKENS * (128 + 8)];
    griddep_launch();
    const int h = blockIdx.x, row = latent + rot_dim;
    const T* source = q + (size_t)h * (head_dim + rot_dim);
    if (blockIdx.y == gridDim.y - 1) {
        griddep_wait();
        source = settled(source);
        const int half = rotary_dim / 2, rest = rot_dim - rotary_dim;
        for (int i = threadIdx.x; i < tokens * (half + rest); i += blockDim.x) {
            const int t = i / (half + rest), pair = i - t * (half + rest);
            const T* part = source + (size_t)t * ld + head_dim;
            T* to = queries + ((size_t)t * heads + h) * row + latent;
            if (pair >= half) {
                to[half + pair] = part[half + pair];              // = rotary_dim + (pair - half)
                continue;
            }
            float sine, cosine;
            sincosf((float)positions[t] * inv_freq[pair], &sine, &cosine);
            sine *= amplitude;
            cosine *= amplitude;
            const int first = neighbours ? 2 * pair : pair, second = neighbours ? first + 1 : pair + half;
            const float u = to_float<T>(part[first]), v = to_float<T>(part[second]);
            to[first] = from_float<T>(u * cosine - v * sine);
            to[second] = from_float<T>(v * cosine + u * sine);
        }
        return;
    }
    const int side = threadIdx.x & 1, n = blockIdx.y * ABSORB_COLUMNS + (threadIdx.x >> 1);
    const int halved = head_dim / 2, pieces = halved / 8, stride = halved + 4;
    uint4 held[ABSORB_PIECES];
#pragma unroll
    for (int i = 0; i < ABSORB_PIECES; ++i) {
        held[i] = make_uint4(0u, 0u, 0u, 0u);
        if (i < pieces && n < latent)
            held[i] = *reinterpret_cast<const uint4*>(up_k + ((size_t)h * latent + n) * head_dim +
                                                      side * halved + i * 8);
    }
    griddep_wait();
    source = settled(source);
    for (int i = threadIdx.x; i < TOKENS * head_dim; i += blockDim.x) {
        const int t = i / head_dim, e = i - t * head_dim;
        staged[t * 2 * stride + (e < halved ? e : e + 4)] = t < tokens ? to_float<T>(source[(size_t)t * ld + e]) : 0.f;
    }
    __syncthreads();
    float sum[TOKENS];
#pragma unroll
    for (int t = 0; t < TOKENS; ++t) sum[t] = 0.f;
#pragma unroll
    for (int i = 0; i < ABSORB_PIECES; ++i) {
        if (i >= pieces) break;
        const T* w = reinterpret_cast<const T*>(&held[i]);
        float weight[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) weight[k] = to_float<T>(w[k]);
#pragma unroll
        for (int t = 0; t < TOKENS; ++t) {
            const float* x = staged + t * 2 * stride + side * stride + i * 8;
            const float4 lo = *reinterpret_cast<const float4*>(x), hi = *reinterpret_cast<const float4*>(x + 4);
            sum[t] = fmaf(weight[0], lo.x, sum[t]); sum[t] = fmaf(weight[1], lo.y, sum[t]);
            sum[t] = fmaf(weight[2], lo.z, sum[t]); sum[t] = fmaf(weight[3], lo.w, sum[t]);
            sum[t] = fmaf(weight[4], hi.x, sum[t]); sum[t] = fmaf(weight[5], hi.y, sum[t]);
            sum[t] = fmaf(weight[6], hi.z, sum[t]); sum[t] = fmaf(weight[7], hi.w, sum[t]);
        }
    }
#pragma unroll
    for (int t = 0; t < TOKENS; ++t) {
        sum[t] += __shfl_xor_sync(0xffffffffu, sum[t], 1);
        if (t < tokens && n < latent && (t & 1) == side)
            queries[((size_t)t * heads + h) * row + n] = from_float<T>(sum[t]);
    }
}

// out[t, c] = values[t, c] * sigmoid(gate[t * ld_gate + c])
template <typename T>
__global__ void sigmoid_gate_kernel(const T* __restrict__ values, const T* __restrict__ gate,
                                    int ld_gate, T* __restrict__ out, int width, long long total) {
    griddep_launch();
    griddep_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const long long t = i / width;
    const int c = (int)(i % width);
    const float g = to_float<T>(gate[t * ld_gate + c]);
    out[i] = from_float<T>(to_float<T>(values[i]) / (1.f + expf(-g)));
}

// The same for bfloat16 rows whose width and strides are multiples of 8: 16 bytes per thread.
__global__ void sigmoid_gate_wide_kernel(const __nv_bfloat16* __restrict__ values,
                                         const __nv_bfloat16* __restrict__ gate, int ld_gate,
                                         __nv_bfloat16* __restrict__ out, int width,
                                         long long groups) {
    griddep_launch();
    griddep_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= groups) return;
    const int per_row = width >> 3;
    const long long t = i / per_row;
    const int c = (int)(i - t * per_row) << 3;
    const uint4 v = *reinterpret_cast<const uint4*>(values + t * width + c);
    const uint4 g = *reinterpret_cast<const uint4*>(gate + t * ld_gate + c);
    const __nv_bfloat162* vs = reinterpret_cast<const __nv_bfloat162*>(&v);
    const __nv_bfloat162* gs = reinterpret_cast<const __nv_bfloat162*>(&g);
    uint4 result;
    __nv_bfloat162* rs = reinterpret_cast<__nv_bfloat162*>(&result);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const float2 a = __bfloat1622float2(vs[j]), b = __bfloat1622float2(gs[j]);
        rs[j] = __floats2bfloat162_rn(a.x / (1.f + expf(-b.x)), a.y / (1.f + expf(-b.y)));
    }
    *reinterpret_cast<uint4*>(out + t * width + c) = result;
}

// maps [tokens, 2 * heads, row_dim]: head h of map m is row m * heads + h, its first value_dim
// values count. out [tokens, heads * value_dim]: o = a1 - mix * a2, o * rsqrt(mean(o^2) + eps) *
// factor. One warp per (token, head).
constexpr int COMBINE_WARPS = 4;
constexpr int COMBINE_MAX = 512 / 32;

template <typename T>
__global__ void __launch_bounds__(COMBINE_WARPS * 32)
differential_combine_kernel(const T* __restrict__ maps, T* __restrict__ out, long long items,
                            int heads, int row_dim, int value_dim, float mix, float eps,
                            float factor) {
    griddep_launch();
    griddep_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * COMBINE_WARPS + warp;
    if (item >= items) return;
    const long long t = item / heads;
    const int head = (int)(item % heads);
    const T* first = maps + ((size_t)t * 2 * heads + head) * row_dim;
    const T* second = first + (size_t)heads * row_dim;
    float o[COMBINE_MAX];
    float squares = 0.f;
#pragma unroll
    for (int i = 0; i < COMBINE_MAX; ++i) {
        const int e = lane + 32 * i;
        o[i] = 0.f;
        if (e < value_dim) {
            o[i] = to_float<T>(first[e]) - mix * to_float<T>(second[e]);
            squares = fmaf(o[i], o[i], squares);
        }
    }
    squares = warp_sum(squares);
    const float inv = rsqrtf(squares / (float)value_dim + eps) * factor;
    T* dst = out + ((size_t)t * heads + head) * value_dim;
#pragma unroll
    for (int i = 0; i < COMBINE_MAX; ++i) {
        const int e = lane + 32 * i;
        if (e < value_dim) dst[e] = from_float<T>(o[i] * inv);
    }
}

// The heads' outputs times a sigmoid gate: values [tokens, heads, row_dim], of which the first
// value_dim of a row count, -> out [tokens, heads * value_dim]; the gate has one number per value
// (rows [heads * value_dim]) or, with `per_head`, one per head (rows [heads]); its rows may be a
// slice of wider rows.
template <typename T>
__global__ void gate_heads_kernel(const T* __restrict__ values, const T* __restrict__ gate, int ld_gate,
                                  T* __restrict__ out, int heads, int row_dim, int value_dim,
                                  int per_head, long long total) {
    griddep_launch();
    griddep_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int width = heads * value_dim;
    const long long t = i / width;
    const int c = (int)(i - t * width);
    const int head = c / value_dim, e = c - head * value_dim;
    const float g = to_float<T>(gate[t * ld_gate + (per_head ? head : c)]);
    const float v = to_float<T>(values[(t * heads + head) * row_dim + e]);
    // (16-bit storage: the hardware's exponential and reciprocal, far inside its rounding)
    out[i] = from_float<T>(sizeof(T) == 2 ? v * __frcp_rn(1.f + __expf(-g)) : v / (1.f + expf(-g)));
}

}  // namespace

// q_source, small_source, down_source: null leaves a part out (see the kernel).
MLXONE_API int mlxone_latent_prepare(const void* q_source, int ld_q, void* queries,
                                     const void* small_source, int ld_small,
                                     const float* small_weight, void* small, int rank,
                                     const void* down_source, int ld_down,
                                     const float* norm_weight, float eps, const float* inv_freq,
                                     int rotary_dim, float amplitude, int neighbours,
                                     const int* positions, const int* token_request, void* pages,
                                     const int* block_table, int table_width, int page_size,
                                     int tokens, int heads, int head_dim, int rot_dim, int latent,
                                     int write, int dtype, int* error_flag, cudaStream_t stream) {
    if (tokens == 0) return 0;
    MLXONE_REQUIRE(tokens > 0 && heads > 0 && head_dim >= 0 && rot_dim >= 0 && latent > 0,
                   "latent_prepare: bad sizes");
    MLXONE_REQUIRE((q_source == nullptr || ld_q >= heads * (head_dim + rot_dim)) &&
                       (down_source == nullptr || ld_down >= latent + rot_dim) &&
                       (small_source == nullptr || (rank > 0 && ld_small >= rank)),
                   "latent_prepare: rows of %d, %d, %d values are too short", ld_q, ld_small, ld_down);
    if (inv_freq == nullptr) rotary_dim = 0;
    MLXONE_REQUIRE(rotary_dim >= 0 && rotary_dim % 2 == 0 && rotary_dim <= rot_dim,
                   "latent_prepare: %d rotated dimensions in a part of %d", rotary_dim, rot_dim);
    const size_t shared = (size_t)rotary_dim * sizeof(float);
    // (the block's size follows the model's sizes alone, so a token's sums never change order)
    int most = latent;
    if (q_source != nullptr && heads * rot_dim > most) most = heads * rot_dim;
    if (small_source != nullptr && rank > most) most = rank;
    const int threads = most >= 2048 ? 512 : most >= 512 ? 256 : 128;
#define PREPARE(T)                                                                              \
    launch_kernel(latent_prepare_kernel<T>, dim3(tokens, small_source != nullptr ? 2 : 1),      \
                  dim3(threads), shared, stream, true,                                          \
                  (const T*)q_source, ld_q, (T*)queries, (const T*)small_source, ld_small,      \
                  small_weight, (T*)small, rank, (const T*)down_source, ld_down, norm_weight, eps, \
                  inv_freq, rotary_dim, amplitude, neighbours, positions, token_request, (T*)pages, \
                  block_table, table_width, page_size, heads, head_dim, rot_dim, latent, write, \
                  error_flag)
    if (dtype == MLXONE_BF16) PREPARE(__nv_bfloat16);
    else PREPARE(float);
#undef PREPARE
    MLXONE_LAUNCH_CHECK("latent_prepare");
    return 0;
}

// 1 if latent_absorb takes `tokens` tokens of heads with head_dim unrotated values.
MLXONE_API int mlxone_latent_absorb_fits(int tokens, int head_dim) {
    return tokens >= 1 && tokens <= 16 && head_dim % 16 == 0 && head_dim >= 16 &&
           head_dim <= 16 * ABSORB_PIECES;
}

// q [tokens, heads * (head_dim + rot_dim)] bfloat16 with rows `ld` apart; up_k [heads, latent,
// head_dim]; queries [tokens, heads, latent + rot_dim].
MLXONE_API int mlxone_latent_absorb(const void* q, int ld, const void* up_k, void* queries,
                                    const float* inv_freq, int rotary_dim, float amplitude,
                                    int neighbours, const int* positions, int tokens, int heads,
                                    int head_dim, int rot_dim, int latent, cudaStream_t stream) {
    if (tokens == 0) return 0;
    if (inv_freq == nullptr) rotary_dim = 0;
    MLXONE_REQUIRE(mlxone_latent_absorb_fits(tokens, head_dim) && heads > 0 && latent > 0 && rot_dim >= 0 &&
                       ld >= heads * (head_dim + rot_dim), "latent_absorb: bad sizes");
    MLXONE_REQUIRE((reinterpret_cast<uintptr_t>(up_k) & 15) == 0, "latent_absorb: up_k is not aligned");
    MLXONE_REQUIRE(rotary_dim >= 0 && rotary_dim % 2 == 0 && rotary_dim <= rot_dim,
                   "latent_absorb: %d rotated dimensions in a part of %d", rotary_dim, rot_dim);
    const dim3 grid(heads, (latent + ABSORB_COLUMNS - 1) / ABSORB_COLUMNS + 1);
#define ABSORB(TOKENS)                                                                              \
    launch_kernel(latent_absorb_kernel<TOKENS>, grid, dim3(2 * ABSORB_COLUMNS), 0, stream, true,    \
                  (const __nv_bfloat16*)q, ld, (const __nv_bfloat16*)up_k, (__nv_bfloat16*)queries, \
                  inv_freq, rotary_dim, amplitude, neighbours, positions, tokens, heads, head_dim,  \
                  rot_dim, latent)
    if (tokens <= 4) ABSORB(4);
    else if (tokens <= 8) ABSORB(8);
    else ABSORB(16);
#undef ABSORB
    MLXONE_LAUNCH_CHECK("latent_absorb");
    return 0;
}

MLXONE_API int mlxone_sigmoid_gate(const void* values, const void* gate, int ld_gate, void* out,
                                   int rows, int width, int dtype, cudaStream_t stream) {
    if (rows == 0 || width == 0) return 0;
    MLXONE_REQUIRE(rows > 0 && width > 0 && ld_gate >= width, "sigmoid_gate: bad sizes");
    const long long total = (long long)rows * width;
    const auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (dtype == MLXONE_BF16 && width % 8 == 0 && ld_gate % 8 == 0 && aligned(values) &&
        aligned(gate) && aligned(out)) {
        using T = __nv_bfloat16;
        launch_kernel(sigmoid_gate_wide_kernel, dim3(ceil_div_host(total / 8, 256)), dim3(256), 0,
                      stream, true, (const T*)values, (const T*)gate, ld_gate, (T*)out, width,
                      total / 8);
    } else if (dtype == MLXONE_BF16) {
        using T = __nv_bfloat16;
        launch_kernel(sigmoid_gate_kernel<T>, dim3(ceil_div_host(total, 256)), dim3(256), 0, stream,
                      true, (const T*)values, (const T*)gate, ld_gate, (T*)out, width, total);
    } else {
        using T = float;
        launch_kernel(sigmoid_gate_kernel<T>, dim3(ceil_div_host(total, 256)), dim3(256), 0, stream,
                      true, (const T*)values, (const T*)gate, ld_gate, (T*)out, width, total);
    }
    MLXONE_LAUNCH_CHECK("sigmoid_gate");
    return 0;
}

MLXONE_API int mlxone_differential_combine(const void* maps, void* out, int tokens, int heads,
                                           int row_dim, int value_dim, float mix, float eps,
                                           float factor, int dtype, cudaStream_t stream) {
    if (tokens == 0) return 0;
    MLXONE_REQUIRE(tokens > 0 && heads > 0 && value_dim > 0 && value_dim <= row_dim &&
                       value_dim <= COMBINE_MAX * 32,
                   "differential_combine: values of %d in rows of %d", value_dim, row_dim);
    const long long items = (long long)tokens * heads;
    const dim3 grid(ceil_div_host(items, COMBINE_WARPS));
    if (dtype == MLXONE_BF16) {
        using T = __nv_bfloat16;
        launch_kernel(differential_combine_kernel<T>, grid, dim3(COMBINE_WARPS * 32), 0, stream,
                      true, (const T*)maps, (T*)out, items, heads, row_dim, value_dim, mix, eps,
                      factor);
    } else {
        using T = float;
        launch_kernel(differential_combine_kernel<T>, grid, dim3(COMBINE_WARPS * 32), 0, stream,
                      true, (const T*)maps, (T*)out, items, heads, row_dim, value_dim, mix, eps,
                      factor);
    }
    MLXONE_LAUNCH_CHECK("differential_combine");
    return 0;
}

MLXONE_API int mlxone_gate_heads(const void* values, const void* gate, int ld_gate, void* out,
                                 int tokens, int heads, int row_dim, int value_dim, int per_head,
                                 int dtype, cudaStream_t stream) {
    if (tokens == 0) return 0;
    MLXONE_REQUIRE(heads > 0 && value_dim > 0 && value_dim <= row_dim,
                   "gate_heads: values of %d in rows of %d", value_dim, row_dim);
    const long long total = (long long)tokens * heads * value_dim;
    if (dtype == MLXONE_BF16) {
        using T = __nv_bfloat16;
        launch_kernel(gate_heads_kernel<T>, dim3(ceil_div_host(total, 256)), dim3(256), 0, stream,
                      true, (const T*)values, (const T*)gate, ld_gate, (T*)out, heads, row_dim,
                      value_dim, per_head, total);
    } else {
        using T = float;
        launch_kernel(gate_heads_kernel<T>, dim3(ceil_div_host(total, 256)), dim3(256), 0, stream,
                      true, (const T*)values, (const T*)gate, ld_gate, (T*)out, heads, row_dim,
                      value_dim, per_head, total);
    }
    MLXONE_LAUNCH_CHECK("gate_heads");
    return 0;
}
