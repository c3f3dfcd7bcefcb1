// Per-head RMSNorm of queries and keys, rotary position encoding, and the write of keys and
// values into the request's pages.
//
// qkv[t] = [q heads | k heads | v heads], each head of head_dim values. One warp handles one
// (token, head): it norms q or k over head_dim in 32-bit (if a norm weight is given), rotates
// the first rotary_dim dimensions by position * inv_freq (pairs j and j + rotary_dim/2, the
// non-interleaved form; angles in 32-bit), writes q to q_out[t, head, :] and k, v to
// kv[0 or 1, page, kv_head, position % page_size, :] with page = block_table[request,
// position / page_size].
#include "common.cuh"

namespace {

constexpr int WARPS = 8;
constexpr int MAX_HEAD_DIM = 512;

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
qk_prep_kernel(const T* __restrict__ qkv, const float* __restrict__ q_weight,
               const float* __restrict__ k_weight, float eps, const float* __restrict__ inv_freq,
               int rotary_dim, const int* __restrict__ positions,
               const int* __restrict__ token_request, T* __restrict__ q_out,
               T* __restrict__ kv, const int* __restrict__ block_table, int table_width,
               int page_size, long long kv_half, int tokens, int heads, int kv_heads,
               int head_dim, int write_kv, int* __restrict__ error_flag) {
    extern __shared__ float shared[];
    griddep_launch();
    griddep_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slots_per_token = heads + 2 * kv_heads;
    const long long item = (long long)blockIdx.x * WARPS + warp;
    if (item >= (long long)tokens * slots_per_token) return;
    const int t = (int)(item / slots_per_token);
    const int slot = (int)(item % slots_per_token);
    float* values = shared + warp * head_dim;

    const T* src = qkv + (size_t)t * slots_per_token * head_dim + (size_t)slot * head_dim;
    const bool is_q = slot < heads;
    const bool is_k = !is_q && slot < heads + kv_heads;
    if (!is_q && !write_kv) return;

    float sum = 0.f;
    for (int e = lane; e < head_dim; e += 32) {
        const float v = to_float<T>(src[e]);
        values[e] = v;
        sum += v * v;
    }
    const int position = positions[t];
    if (is_q || is_k) {
        const float* weight = is_q ? q_weight : k_weight;
        if (weight != nullptr) {
            sum = warp_sum(sum);
            const float inv = rsqrtf(sum / (float)head_dim + eps);
            for (int e = lane; e < head_dim; e += 32) values[e] = values[e] * inv * weight[e];
        }
        __syncwarp();
        if (inv_freq != nullptr) {
            const int half = rotary_dim / 2;
            for (int j = lane; j < half; j += 32) {
                const float angle = (float)position * inv_freq[j];
                float sine, cosine;
                sincosf(angle, &sine, &cosine);
                const float a = values[j], b = values[j + half];
                values[j] = a * cosine - b * sine;
                values[j + half] = b * cosine + a * sine;
            }
        }
    }
    __syncwarp();

    T* dst;
    if (is_q) {
        dst = q_out + ((size_t)t * heads + slot) * head_dim;
    } else {
        const int kv_head = is_k ? slot - heads : slot - heads - kv_heads;
        const int r = token_request[t];
        const int block = position / page_size;
        const int page = block < table_width ? block_table[(size_t)r * table_width + block] : -1;
        if (page < 0) {
            if (lane == 0) atomicExch(error_flag, 2);
            return;
        }
        dst = kv + (is_k ? 0 : kv_half) +
              (((size_t)page * kv_heads + kv_head) * page_size + position % page_size) * head_dim;
    }
    for (int e = lane; e < head_dim; e += 32) dst[e] = from_float<T>(values[e]);
}

// bfloat16 with a head size of 32, 64, 128 or 256 that is rotated as a whole (or not at all):
// a lane keeps HD/32 neighbouring values of the head in registers, its rotation partner sits 16
// lanes away, and the angles are computed once per token, not once per head. One block per
// token; its warps take the token's heads in turn.
template <int HD>
__global__ void __launch_bounds__(WARPS * 32)
qk_prep_wide_kernel(const __nv_bfloat16* __restrict__ qkv, const float* __restrict__ q_weight,
                    const float* __restrict__ k_weight, float eps,
                    const float* __restrict__ inv_freq, const int* __restrict__ positions,
                    const int* __restrict__ token_request, __nv_bfloat16* __restrict__ q_out,
                    __nv_bfloat16* __restrict__ kv, const int* __restrict__ block_table,
                    int table_width, int page_size, long long kv_half, int heads, int kv_heads,
                    int write_kv, int* __restrict__ error_flag) {
    using T = __nv_bfloat16;
    constexpr int E = HD / 32;
    griddep_launch();
    griddep_wait();
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slots = heads + 2 * kv_heads;
    const int e0 = E * lane;
    // AHEAD of the warp's heads at a time: their loads are issued together, the first ones
    // before anything that waits for the token's position or page
    constexpr int AHEAD = 6;
    const T* row = qkv + (size_t)t * slots * HD;
    float held[AHEAD][E];
    auto load_heads = [&](int base) {
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) {
            const int slot = base + a * WARPS;
            if (slot >= slots) continue;
            const T* src = row + (size_t)slot * HD + e0;
            if (E == 1) {
                held[a][0] = __bfloat162float(src[0]);
            } else {
#pragma unroll
                for (int i = 0; i < E; i += 2) {
                    const __nv_bfloat162 pair = *reinterpret_cast<const __nv_bfloat162*>(src + i);
                    held[a][i] = __low2float(pair);
                    held[a][i + 1] = __high2float(pair);
                }
            }
        }
    };
    load_heads(warp);
    const int position = positions[t];
    float cosine[E], sine[E], q_scale[E], k_scale[E];
#pragma unroll
    for (int i = 0; i < E; ++i) {
        cosine[i] = 1.f;
        sine[i] = 0.f;
        if (inv_freq != nullptr) {
            const float angle = (float)position * inv_freq[(e0 + i) % (HD / 2)];
            sincosf(angle, &sine[i], &cosine[i]);
            if (lane < 16) sine[i] = -sine[i];       // first half: a cos - b sin
        }
        q_scale[i] = q_weight ? q_weight[e0 + i] : 1.f;
        k_scale[i] = k_weight ? k_weight[e0 + i] : 1.f;
    }
    // where this token's keys and values go
    T* page_base = nullptr;
    if (write_kv) {
        const int r = token_request[t];
        const int block = position / page_size;
        const int page = block < table_width ? block_table[(size_t)r * table_width + block] : -1;
        if (page < 0) {
            if (threadIdx.x == 0) atomicExch(error_flag, 2);
        } else {
            page_base = kv + ((size_t)page * kv_heads * page_size + position % page_size) * HD;
        }
    }
    for (int base = warp; base < slots; base += AHEAD * WARPS) {
        if (base != warp) load_heads(base);
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) {
            const int slot = base + a * WARPS;
            if (slot >= slots) continue;
            const bool is_q = slot < heads;
            const bool is_k = !is_q && slot < heads + kv_heads;
            if (!is_q && page_base == nullptr) continue;
            float (&v)[E] = held[a];
            if (is_q || is_k) {
                const float* scale = is_q ? q_scale : k_scale;
                if ((is_q ? q_weight : k_weight) != nullptr) {
                    float sum = 0.f;
#pragma unroll
                    for (int i = 0; i < E; ++i) sum += v[i] * v[i];
                    sum = warp_sum(sum);
                    const float inv = rsqrtf(sum / (float)HD + eps);
#pragma unroll
                    for (int i = 0; i < E; ++i) v[i] = v[i] * inv * scale[i];
                }
                if (inv_freq != nullptr) {
#pragma unroll
                    for (int i = 0; i < E; ++i) {
                        const float partner = __shfl_xor_sync(0xffffffffu, v[i], 16);
                        v[i] = v[i] * cosine[i] + partner * sine[i];
                    }
                }
            }
            T* dst;
            if (is_q) {
                dst = q_out + ((size_t)t * heads + slot) * HD + e0;
            } else {
                const int kv_head = is_k ? slot - heads : slot - heads - kv_heads;
                dst = page_base + (is_k ? 0 : kv_half) + (size_t)kv_head * page_size * HD + e0;
            }
            if (E == 1) {
                dst[0] = __float2bfloat16_rn(v[0]);
            } else {
#pragma unroll
                for (int i = 0; i < E; i += 2)
                    *reinterpret_cast<__nv_bfloat162*>(dst + i) = __floats2bfloat162_rn(v[i], v[i + 1]);
            }
        }
    }
}

// The general form: queries and keys of ``head_dim`` values, values of ``value_dim``, all
// written into rows of ``row_dim`` >= both (zeros behind the shorter ones), so that keys and
// values share one page geometry. qkv[t] = [heads x head_dim | kv_heads x head_dim | kv_heads x
// value_dim], rows ``ld`` values apart (a slice of a wider product). The rotation multiplies
// cosine and sine by ``amplitude``. norm_mode 0: no norm;
// 1: RMSNorm with the given weights before the rotation; 2: division by the root mean square
// (over head_dim, eps inside the root) after the rotation, no weight; 3: RMSNorm over all query heads'
// values at once, and over all key heads', with weights of those sizes, before the rotation (every
// block of a token works the two sums out). One warp per (token, head). `extra`: a factor on the
// queries that grows with the position, and values mixed with another layer's.
struct PrepExtra {
    float coef = 0.f;               // queries times 1 + coef ln(floor((p + 1) / every) + 1); 0: as they are
    double every = 1.0;
    const void* first = nullptr;    // v <- (1 - mix) v + mix first[t, :]; rows `first_ld` values apart
    int first_ld = 0;
    float mix = 0.f;
};

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
qk_prep_general_kernel(const T* __restrict__ qkv, const float* __restrict__ q_weight,
                       const float* __restrict__ k_weight, float eps,
                       const float* __restrict__ inv_freq, int rotary_dim, float amplitude,
                       int norm_mode, const int* __restrict__ positions,
                       const int* __restrict__ token_request, T* __restrict__ q_out,
                       T* __restrict__ kv, const int* __restrict__ block_table, int table_width,
                       int page_size, long long kv_half, int tokens, int heads, int kv_heads,
                       int head_dim, int value_dim, int row_dim, int write_kv, int ld,
                       int* __restrict__ error_flag, PrepExtra extra) {
    // Blocks (token, part): the angles' cosines and sines are worked out once for the block's
    // heads (rotary_dim / 2 of each, scaled), then its warps take their share of the token's
    // heads in turn: a warp has one head in a step of few tokens, two in a large one.
    extern __shared__ float shared[];
    float* cosines = shared;
    float* sines = shared + rotary_dim / 2;
    griddep_launch();
    griddep_wait();
    qkv = settled(qkv);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slots_per_token = heads + 2 * kv_heads;
    const int t = blockIdx.x;
    const int position = positions[t];
    const int half = rotary_dim / 2;
    if (inv_freq != nullptr) {
        for (int j = threadIdx.x; j < half; j += blockDim.x) {
            float sine, cosine;
            sincosf((float)position * inv_freq[j], &sine, &cosine);
            sines[j] = sine * amplitude;
            cosines[j] = cosine * amplitude;
        }
    }
    float whole[2] = {1.f, 1.f};               // 1 / rms of all queries, of all keys
    if (norm_mode == 3) {
        __shared__ float scratch[33];
        const T* row = qkv + (size_t)t * ld;
        for (int part = 0; part < 2; ++part) {
            const int first = part == 0 ? 0 : heads * head_dim;
            const int count = (part == 0 ? heads : kv_heads) * head_dim;
            float sum = 0.f;
            for (int e = threadIdx.x; e < count; e += blockDim.x) {
                const float v = to_float<T>(row[first + e]);
                sum = fmaf(v, v, sum);
            }
            whole[part] = rsqrtf(block_sum(sum, scratch) / (float)count + eps);
        }
    }
    float warmth = 1.f;
    if (extra.coef != 0.f)
        warmth = fmaf(extra.coef, logf((float)(floor((double)(position + 1) / extra.every) + 1.0)), 1.f);
    __syncthreads();
    // where this token's keys and values go
    T* page_base = nullptr;
    if (write_kv) {
        const int r = token_request[t];
        const int block = position / page_size;
        const int page = block < table_width ? block_table[(size_t)r * table_width + block] : -1;
        if (page < 0) {
            if (threadIdx.x == 0) atomicExch(error_flag, 2);
        } else {
            page_base = kv + ((size_t)page * kv_heads * page_size + position % page_size) * row_dim;
        }
    }
    float* values = shared + rotary_dim + warp * row_dim;
    for (int slot = warp + WARPS * blockIdx.y; slot < slots_per_token; slot += WARPS * gridDim.y) {
        const bool is_q = slot < heads;
        const bool is_k = !is_q && slot < heads + kv_heads;
        if (!is_q && page_base == nullptr) continue;
        const int size = (is_q || is_k) ? head_dim : value_dim;
        const T* src = qkv + (size_t)t * ld +
                       (is_q || is_k ? (size_t)slot * head_dim
                                     : (size_t)(heads + kv_heads) * head_dim +
                                           (size_t)(slot - heads - kv_heads) * value_dim);
        float sum = 0.f;
        for (int e = lane; e < row_dim; e += 32) {
            const float v = e < size ? to_float<T>(src[e]) : 0.f;
            values[e] = v;
            sum += v * v;
        }
        if (is_q || is_k) {
            const float* weight = is_q ? q_weight : k_weight;
            if (norm_mode == 1) {
                sum = warp_sum(sum);
                const float inv = rsqrtf(sum / (float)head_dim + eps);
                for (int e = lane; e < head_dim; e += 32)
                    values[e] = values[e] * inv * (weight ? weight[e] : 1.f);
            } else if (norm_mode == 3) {
                const int first = (is_q ? slot : slot - heads) * head_dim;
                const float inv = is_q ? whole[0] : whole[1];
                for (int e = lane; e < head_dim; e += 32) values[e] = values[e] * inv * weight[first + e];
            }
            if (is_q && warmth != 1.f)          // (a factor on the row: before or after the rotation alike)
                for (int e = lane; e < head_dim; e += 32) values[e] *= warmth;
            __syncwarp();
            float squares = 0.f;
            if (inv_freq != nullptr) {
                for (int j = lane; j < half; j += 32) {
                    const float a = values[j], b = values[j + half];
                    const float first = a * cosines[j] - b * sines[j];
                    const float second = b * cosines[j] + a * sines[j];
                    values[j] = first;
                    values[j + half] = second;
                }
            }
            __syncwarp();
            if (norm_mode == 2) {
                for (int e = lane; e < head_dim; e += 32) squares = fmaf(values[e], values[e], squares);
                squares = warp_sum(squares);
                const float inv = 1.f / sqrtf(squares / (float)head_dim + eps);
                for (int e = lane; e < head_dim; e += 32) values[e] *= inv;
            }
        } else if (extra.first != nullptr) {
            const T* first = static_cast<const T*>(extra.first) + (size_t)t * extra.first_ld +
                             (size_t)(slot - heads - kv_heads) * value_dim;
            for (int e = lane; e < value_dim; e += 32)
                values[e] = fmaf(extra.mix, to_float<T>(first[e]), (1.f - extra.mix) * values[e]);
        }
        __syncwarp();
        T* dst;
        if (is_q) {
            dst = q_out + ((size_t)t * heads + slot) * row_dim;
        } else {
            const int kv_head = is_k ? slot - heads : slot - heads - kv_heads;
            dst = page_base + (is_k ? 0 : kv_half) + (size_t)kv_head * page_size * row_dim;
        }
        for (int e = lane; e < row_dim; e += 32) dst[e] = from_float<T>(values[e]);
        __syncwarp();
    }
}

// Norm mode 3 without a rotation, for bfloat16 rows whose heads are multiples of 8 values: one block per
// token, the whole row in registers (C pieces of 16 bytes a thread), one pass over memory.
template <int C>
__global__ void __launch_bounds__(C == 4 ? 768 : 1024)
qk_prep_rows_kernel(const __nv_bfloat16* __restrict__ qkv, const float* __restrict__ q_weight,
                    const float* __restrict__ k_weight, float eps, const int* __restrict__ positions,
                    const int* __restrict__ token_request, __nv_bfloat16* __restrict__ q_out,
                    __nv_bfloat16* __restrict__ kv, const int* __restrict__ block_table, int table_width,
                    int page_size, long long kv_half, int heads, int kv_heads, int head_dim,
                    int value_dim, int row_dim, int write_kv, int ld, int* __restrict__ error_flag,
                    PrepExtra extra) {
    using T = __nv_bfloat16;
    __shared__ float sums[2][32];
    griddep_launch();
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int q_size = heads * head_dim, k_size = kv_heads * head_dim, v_size = kv_heads * value_dim;
    const int pieces = (q_size + k_size + v_size) / 8;
    griddep_wait();
    const T* row = settled(qkv) + (size_t)t * ld;
    const T* first = extra.first == nullptr ? nullptr
        : settled(static_cast<const T*>(extra.first)) + (size_t)t * extra.first_ld;
    uint4 raw[C], other[C];
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int at = (c * blockDim.x + threadIdx.x) * 8;
        raw[c] = other[c] = make_uint4(0u, 0u, 0u, 0u);
        if (at < pieces * 8) {
            raw[c] = *reinterpret_cast<const uint4*>(row + at);
            if (first != nullptr && at >= q_size + k_size)
                other[c] = *reinterpret_cast<const uint4*>(first + at - q_size - k_size);
        }
    }
    const int position = positions[t];
    T* page_base = nullptr;
    if (write_kv) {
        const int block = position / page_size;
        const int page = block < table_width
                             ? block_table[(size_t)token_request[t] * table_width + block] : -1;
        if (page >= 0)
            page_base = kv + ((size_t)page * kv_heads * page_size + position % page_size) * row_dim;
        else if (threadIdx.x == 0)
            atomicExch(error_flag, 2);
    }
    float warmth = 1.f;
    if (extra.coef != 0.f)
        warmth = fmaf(extra.coef, logf((float)(floor((double)(position + 1) / extra.every) + 1.0)), 1.f);
    float squares[2] = {0.f, 0.f};
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int at = (c * blockDim.x + threadIdx.x) * 8;
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw[c]);
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float a = __low2float(p[i]), b = __high2float(p[i]);
            sum = fmaf(a, a, fmaf(b, b, sum));
        }
        if (at < q_size) squares[0] += sum;
        else if (at < q_size + k_size) squares[1] += sum;
    }
    const int warps = blockDim.x >> 5;
#pragma unroll
    for (int part = 0; part < 2; ++part) {
        squares[part] = warp_sum(squares[part]);
        if (lane == 0) sums[part][warp] = squares[part];
    }
    __syncthreads();
    const float q_inv = rsqrtf(warp_sum(lane < warps ? sums[0][lane] : 0.f) / (float)q_size + eps) * warmth;
    const float k_inv = rsqrtf(warp_sum(lane < warps ? sums[1][lane] : 0.f) / (float)k_size + eps);
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int at = (c * blockDim.x + threadIdx.x) * 8;
        if (at >= pieces * 8) continue;
        const bool is_q = at < q_size, is_k = !is_q && at < q_size + k_size;
        if (!is_q && page_base == nullptr) continue;
        const int within = is_q ? at : is_k ? at - q_size : at - q_size - k_size;
        const int size = is_q || is_k ? head_dim : value_dim;
        const int head = within / size, place = within - head * size;
        __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&raw[c]);
        const __nv_bfloat162* o = reinterpret_cast<const __nv_bfloat162*>(&other[c]);
        if (is_q || is_k) {
            const float* weight = (is_q ? q_weight : k_weight) + within;
            const float4 lo = *reinterpret_cast<const float4*>(weight), hi = *reinterpret_cast<const float4*>(weight + 4);
            const float w[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
            const float inv = is_q ? q_inv : k_inv;
#pragma unroll
            for (int i = 0; i < 4; ++i)
                p[i] = __floats2bfloat162_rn(__low2float(p[i]) * inv * w[2 * i],
                                             __high2float(p[i]) * inv * w[2 * i + 1]);
        } else if (first != nullptr) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
                p[i] = __floats2bfloat162_rn(
                    fmaf(extra.mix, __low2float(o[i]), (1.f - extra.mix) * __low2float(p[i])),
                    fmaf(extra.mix, __high2float(o[i]), (1.f - extra.mix) * __high2float(p[i])));
        }
        T* dst = is_q ? q_out + ((size_t)t * heads + head) * row_dim
                      : page_base + (is_k ? 0 : kv_half) + (size_t)head * page_size * row_dim;
        *reinterpret_cast<uint4*>(dst + place) = raw[c];
    }
    // the zeros behind rows that are shorter than the pages'
    const int q_pad = (row_dim - head_dim) / 8, v_pad = (row_dim - value_dim) / 8;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    for (int i = threadIdx.x; i < (heads + kv_heads) * q_pad; i += blockDim.x) {
        const int head = i / q_pad, place = head_dim + (i - head * q_pad) * 8;
        if (head < heads)
            *reinterpret_cast<uint4*>(q_out + ((size_t)t * heads + head) * row_dim + place) = zero;
        else if (page_base != nullptr)
            *reinterpret_cast<uint4*>(page_base + (size_t)(head - heads) * page_size * row_dim + place) = zero;
    }
    if (page_base != nullptr)
        for (int i = threadIdx.x; i < kv_heads * v_pad; i += blockDim.x) {
            const int head = i / v_pad, place = value_dim + (i - head * v_pad) * 8;
            *reinterpret_cast<uint4*>(page_base + kv_half + (size_t)head * page_size * row_dim + place) = zero;
        }
}

template <int HD>
static void launch_qk_prep_wide(const void* qkv, const float* q_weight, const float* k_weight,
                                float eps, const float* inv_freq, const int* positions,
                                const int* token_request, void* q_out, void* kv,
                                const int* block_table, int table_width, int page_size,
                                long long kv_half, int tokens, int heads, int kv_heads,
                                int write_kv, int* error_flag, cudaStream_t stream) {
    using T = __nv_bfloat16;
    launch_kernel(qk_prep_wide_kernel<HD>, dim3(tokens), dim3(WARPS * 32), 0, stream, true,
                  (const T*)qkv, q_weight, k_weight, eps, inv_freq, positions, token_request,
                  (T*)q_out, (T*)kv, block_table, table_width, page_size, kv_half, heads, kv_heads,
                  write_kv, error_flag);
}

}  // namespace

MLXONE_API int mlxone_qk_prep(const void* qkv, const float* q_weight, const float* k_weight,
                              float eps, const float* inv_freq, int rotary_dim,
                              const int* positions, const int* token_request, void* q_out,
                              void* kv, const int* block_table, int table_width, int page_size,
                              int pages, int tokens, int heads, int kv_heads, int head_dim,
                              int write_kv, int dtype, int* error_flag, cudaStream_t stream) {
    if (tokens == 0) return 0;
    MLXONE_REQUIRE(tokens > 0 && heads > 0 && kv_heads > 0, "qk_prep: bad sizes");
    MLXONE_REQUIRE(head_dim >= 2 && head_dim <= MAX_HEAD_DIM,
                   "qk_prep: head size %d is not in 2..%d", head_dim, MAX_HEAD_DIM);
    MLXONE_REQUIRE(inv_freq == nullptr ||
                       (rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= head_dim),
                   "qk_prep: rotary size %d must be even and at most the head size %d", rotary_dim,
                   head_dim);
    MLXONE_REQUIRE(page_size > 0 && pages > 0 && table_width > 0, "qk_prep: bad page geometry");
    const long long items = (long long)tokens * (heads + 2 * kv_heads);
    const int blocks = ceil_div_host(items, WARPS);
    const size_t shared = (size_t)WARPS * head_dim * sizeof(float);
    const long long kv_half = (long long)pages * kv_heads * page_size * head_dim;
    const bool whole = inv_freq == nullptr || rotary_dim == head_dim;
    if (dtype == MLXONE_BF16 && whole &&
        (head_dim == 32 || head_dim == 64 || head_dim == 128 || head_dim == 256)) {
#define WIDE(HD)                                                                                 \
    launch_qk_prep_wide<HD>(qkv, q_weight, k_weight, eps, inv_freq, positions, token_request,   \
                            q_out, kv, block_table, table_width, page_size, kv_half, tokens,    \
                            heads, kv_heads, write_kv, error_flag, stream)
        if (head_dim == 32) WIDE(32);
        else if (head_dim == 64) WIDE(64);
        else if (head_dim == 128) WIDE(128);
        else WIDE(256);
#undef WIDE
    } else if (dtype == MLXONE_BF16) {
        using T = __nv_bfloat16;
        launch_kernel(qk_prep_kernel<T>, dim3(blocks), dim3(WARPS * 32), shared, stream, true, (const T*)qkv, q_weight, k_weight, eps, inv_freq, rotary_dim, positions,
            token_request, (T*)q_out, (T*)kv, block_table, table_width, page_size, kv_half,
            tokens, heads, kv_heads, head_dim, write_kv, error_flag);
    } else {
        using T = float;
        launch_kernel(qk_prep_kernel<T>, dim3(blocks), dim3(WARPS * 32), shared, stream, true, (const T*)qkv, q_weight, k_weight, eps, inv_freq, rotary_dim, positions,
            token_request, (T*)q_out, (T*)kv, block_table, table_width, page_size, kv_half,
            tokens, heads, kv_heads, head_dim, write_kv, error_flag);
    }
    MLXONE_LAUNCH_CHECK("qk_prep");
    return 0;
}

static int qk_prep_general(const void* qkv, const float* q_weight, const float* k_weight,
                           float eps, const float* inv_freq, int rotary_dim,
                           float amplitude, int norm_mode, const int* positions,
                           const int* token_request, void* q_out, void* kv,
                           const int* block_table, int table_width, int page_size,
                           int pages, int tokens, int heads, int kv_heads, int head_dim,
                           int value_dim, int row_dim, int write_kv, int ld, int dtype,
                           int* error_flag, PrepExtra extra, cudaStream_t stream) {
    if (tokens == 0) return 0;
    MLXONE_REQUIRE(tokens > 0 && heads > 0 && kv_heads > 0, "qk_prep: bad sizes");
    MLXONE_REQUIRE(head_dim >= 1 && value_dim >= 1 && row_dim >= head_dim && row_dim >= value_dim &&
                       row_dim <= MAX_HEAD_DIM,
                   "qk_prep: head sizes %d and %d do not fit rows of %d (at most %d)", head_dim,
                   value_dim, row_dim, MAX_HEAD_DIM);
    MLXONE_REQUIRE(inv_freq == nullptr ||
                       (rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= head_dim),
                   "qk_prep: rotary size %d must be even and at most the head size %d", rotary_dim,
                   head_dim);
    MLXONE_REQUIRE(norm_mode >= 0 && norm_mode <= 3, "qk_prep: unknown norm mode %d", norm_mode);
    MLXONE_REQUIRE(norm_mode != 3 || (q_weight != nullptr && k_weight != nullptr),
                   "qk_prep: a norm over whole rows has weights");
    MLXONE_REQUIRE(extra.every > 0.0 && (extra.first == nullptr || extra.first_ld >= kv_heads * value_dim),
                   "qk_prep: bad temperature or value rows");
    MLXONE_REQUIRE(ld >= (heads + kv_heads) * head_dim + kv_heads * value_dim,
                   "qk_prep: rows %d apart are shorter than their heads", ld);
    MLXONE_REQUIRE(page_size > 0 && pages > 0 && table_width > 0, "qk_prep: bad page geometry");
    const int slots = heads + 2 * kv_heads;
    const int parts = tokens < 64 ? ceil_div_host(slots, WARPS) : ceil_div_host(slots, 2 * WARPS);
    const dim3 blocks(tokens, parts < 1 ? 1 : parts);
    const size_t shared = (size_t)(rotary_dim + WARPS * row_dim) * sizeof(float);
    const long long kv_half = (long long)pages * kv_heads * page_size * row_dim;
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const int pieces = ((heads + kv_heads) * head_dim + kv_heads * value_dim) / 8;
    if (dtype == MLXONE_BF16 && norm_mode == 3 && inv_freq == nullptr && head_dim % 8 == 0 &&
        value_dim % 8 == 0 && row_dim % 8 == 0 && ld % 8 == 0 && pieces <= 3072 && aligned(qkv) &&
        aligned(q_out) && aligned(kv) && aligned(q_weight) && aligned(k_weight) && aligned(extra.first) &&
        extra.first_ld % 8 == 0) {
        const int each = pieces > 2048 ? 4 : tokens >= 256 || pieces > 1024 ? 2 : 1;
        const int threads = (ceil_div_host(pieces, each) + 31) / 32 * 32;
        auto kernel = each == 4 ? qk_prep_rows_kernel<4> : each == 2 ? qk_prep_rows_kernel<2>
                                                                     : qk_prep_rows_kernel<1>;
        launch_kernel(kernel, dim3(tokens), dim3(threads), 0, stream, true, (const __nv_bfloat16*)qkv,
                      q_weight, k_weight, eps, positions, token_request, (__nv_bfloat16*)q_out,
                      (__nv_bfloat16*)kv, block_table, table_width, page_size, kv_half, heads, kv_heads,
                      head_dim, value_dim, row_dim, write_kv, ld, error_flag, extra);
        MLXONE_LAUNCH_CHECK("qk_prep_rows");
        return 0;
    }
    if (dtype == MLXONE_BF16) {
        using T = __nv_bfloat16;
        launch_kernel(qk_prep_general_kernel<T>, blocks, dim3(WARPS * 32), shared, stream, true,
                      (const T*)qkv, q_weight, k_weight, eps, inv_freq, rotary_dim, amplitude,
                      norm_mode, positions, token_request, (T*)q_out, (T*)kv, block_table,
                      table_width, page_size, kv_half, tokens, heads, kv_heads, head_dim, value_dim,
                      row_dim, write_kv, ld, error_flag, extra);
    } else {
        using T = float;
        launch_kernel(qk_prep_general_kernel<T>, blocks, dim3(WARPS * 32), shared, stream, true,
                      (const T*)qkv, q_weight, k_weight, eps, inv_freq, rotary_dim, amplitude,
                      norm_mode, positions, token_request, (T*)q_out, (T*)kv, block_table,
                      table_width, page_size, kv_half, tokens, heads, kv_heads, head_dim, value_dim,
                      row_dim, write_kv, ld, error_flag, extra);
    }
    MLXONE_LAUNCH_CHECK("qk_prep_general");
    return 0;
}

MLXONE_API int mlxone_qk_prep_general(const void* qkv, const float* q_weight, const float* k_weight,
                                      float eps, const float* inv_freq, int rotary_dim,
                                      float amplitude, int norm_mode, const int* positions,
                                      const int* token_request, void* q_out, void* kv,
                                      const int* block_table, int table_width, int page_size,
                                      int pages, int tokens, int heads, int kv_heads, int head_dim,
                                      int value_dim, int row_dim, int write_kv, int ld, int dtype,
                                      int* error_flag, cudaStream_t stream) {
    return qk_prep_general(qkv, q_weight, k_weight, eps, inv_freq, rotary_dim, amplitude, norm_mode,
                           positions, token_request, q_out, kv, block_table, table_width, page_size,
                           pages, tokens, heads, kv_heads, head_dim, value_dim, row_dim, write_kv, ld,
                           dtype, error_flag, PrepExtra(), stream);
}

// ... with queries times 1 + coef ln(floor((p + 1) / every) + 1) (coef 0: as they are), and values
// (1 - mix) v + mix first[t, :] (first: rows of kv_heads * value_dim values, `first_ld` apart; null: as
// they are).
MLXONE_API int mlxone_qk_prep_mixed(const void* qkv, const float* q_weight, const float* k_weight,
                                    float eps, const float* inv_freq, int rotary_dim,
                                    float amplitude, int norm_mode, float coef, double every,
                                    const void* first, int first_ld, float mix, const int* positions,
                                    const int* token_request, void* q_out, void* kv,
                                    const int* block_table, int table_width, int page_size, int pages,
                                    int tokens, int heads, int kv_heads, int head_dim, int value_dim,
                                    int row_dim, int write_kv, int ld, int dtype, int* error_flag,
                                    cudaStream_t stream) {
    PrepExtra extra;
    extra.coef = coef; extra.every = every;
    extra.first = first; extra.first_ld = first_ld; extra.mix = mix;
    return qk_prep_general(qkv, q_weight, k_weight, eps, inv_freq, rotary_dim, amplitude, norm_mode,
                           positions, token_request, q_out, kv, block_table, table_width, page_size,
                           pages, tokens, heads, kv_heads, head_dim, value_dim, row_dim, write_kv, ld,
                           dtype, error_flag, extra, stream);
}
