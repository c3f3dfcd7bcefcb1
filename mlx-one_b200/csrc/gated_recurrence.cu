// A gated linear recurrence per channel (the recurrence of Griffin's real-gated linear recurrent
// unit). Per token and channel, from the 32-bit outputs z_r, z_i of the gates' block-diagonal product:
//   r = sigmoid(z_r + bias_r), i = sigmoid(z_i + bias_i), log a = rate * r     (rate <= 0)
//   S = a S + sqrt(1 - a^2) i u;  out = S * gelu_tanh(y)
// S is 32-bit, one number per channel in the request's slot. u and y are rows of the compute dtype.
//
// A prompt's portion is cut into chunks of L tokens that run side by side. Three kernels: `build`
// walks every chunk from S = 0 and leaves the product of its decays and its last S; `chain` brings the
// state from chunk to chunk (eight runs of a request's chunks side by side, joined in shared memory)
// and leaves every chunk's starting state and the request's last one; `walk` goes over the tokens
// again from the starting states and writes the outputs. Portions of one chunk need `walk` only. A step
// of few single tokens is one kernel, the gates' product included.
#include "common.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float fast_inverse(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float fast_root(float x) {
    float y;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// The functions of one token and channel. For 32-bit storage CUDA's own; for 16-bit storage the
// hardware's exponential, reciprocal and root (a few units of 2^-24), and 1 - e^x as a Taylor sum
// where the difference would cancel.
template <typename T>
struct Math {
    static __device__ __forceinline__ float sigmoid(float z) { return fast_inverse(1.f + fast_exp2(-LOG2E * z)); }
    static __device__ __forceinline__ void decay(float log_a, float& a, float& rest) {
        a = fast_exp2(LOG2E * log_a);
        const float x = 2.f * log_a;
        // (1 - e^x) / -x up to x^7 / 8! for -0.35 <= x <= 0: relative error below 2e-8
        float p = fmaf(x, 1.f / 40320.f, 1.f / 5040.f);
        p = fmaf(x, p, 1.f / 720.f);
        p = fmaf(x, p, 1.f / 120.f);
        p = fmaf(x, p, 1.f / 24.f);
        p = fmaf(x, p, 1.f / 6.f);
        p = fmaf(x, p, 0.5f);
        p = fmaf(x, p, 1.f);
        rest = fast_root(x > -0.35f ? -x * p : fmaf(-a, a, 1.f));
    }
    static __device__ __forceinline__ float gelu(float z) {
        // 0.5 (1 + tanh(v)) = sigmoid(2 v)
        return z * sigmoid(1.5957691216057308f * fmaf(0.044715f * z * z, z, z));
    }
};
template <>
struct Math<float> {
    static __device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
    static __device__ __forceinline__ void decay(float log_a, float& a, float& rest) {
        a = expf(log_a);
        rest = sqrtf(-expm1f(2.f * log_a));
    }
    static __device__ __forceinline__ float gelu(float z) { return mlxone_activate(z, MLXONE_ACT_GELU_TANH); }
};

// V (1 or 2) neighbouring values of a row.
template <int V>
__device__ __forceinline__ void load_values(const float* p, float (&v)[V]) {
    if (V == 2) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        v[0] = x.x; v[V - 1] = x.y;
    } else {
        v[0] = *p;
    }
}
template <int V>
__device__ __forceinline__ void load_values(const __nv_bfloat16* p, float (&v)[V]) {
    if (V == 2) {
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(p);
        v[0] = __low2float(x); v[V - 1] = __high2float(x);
    } else {
        v[0] = __bfloat162float(*p);
    }
}
template <int V>
__device__ __forceinline__ void store_values(float* p, const float (&v)[V]) {
    if (V == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[V - 1]);
    else *p = v[0];
}
template <int V>
__device__ __forceinline__ void store_values(__nv_bfloat16* p, const float (&v)[V]) {
    if (V == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[V - 1]);
    else *p = __float2bfloat16_rn(v[0]);
}

struct Operands {
    const void* u;              // [tokens, width]
    const void* y;              // [tokens, width], rows y_ld apart
    int y_ld;
    const float* z;             // the gates' products: token t, part b, row m at t z_token + b z_block + m
    long long z_token, z_block;
    const float* gate_bias;     // [blocks, 2 part]: r's, then i's
    const float* rate;          // [width]
    float* state;               // [slots, width]
    const int* slots;
    const int* request_start;
    void* out;                  // [tokens, width]
    int requests, width, part, chunk, write;
};

// The request and the tokens [first, last) of chunk `index`, the requests' chunks counted through;
// false: there is none (the grid is sized by an upper bound). Also the request's first chunk.
__device__ __forceinline__ bool find_chunk(const Operands& o, int index, int& request, int& first, int& last) {
    __shared__ int found[3];
    if (threadIdx.x == 0) {
        int left = index;
        found[0] = -1;
        for (int r = 0; r < o.requests; ++r) {
            const int from = o.request_start[r], count = o.request_start[r + 1] - from;
            const int chunks = (count + o.chunk - 1) / o.chunk;
            if (left < chunks) {
                found[0] = r;
                found[1] = from + left * o.chunk;
                found[2] = min(from + (left + 1) * o.chunk, from + count);
                break;
            }
            left -= chunks;
        }
    }
    __syncthreads();
    request = found[0]; first = found[1]; last = found[2];
    return request >= 0;
}

// WRITE false: `build`; true: `walk`. carry [chunks, 2, width]: build leaves (product of decays, last
// S from zero); walk starts from carry[chunk][0] (chain has put the starting state there), or, with
// `alone`, from the request's slot, where it then leaves the last state.
template <typename T, int V, bool WALK>
__global__ void __launch_bounds__(128)
gated_recurrence_kernel(Operands o, float* __restrict__ carry, int alone) {
    griddep_launch();
    griddep_wait();
    int request, first, last;
    if (!find_chunk(o, blockIdx.y, request, first, last)) return;
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (c >= o.width) return;
    const int block = c / o.part, within = c - block * o.part;      // (V divides a part)
    float bias_r[V], bias_i[V], rate[V], s[V], product[V];
    load_values<V>(o.gate_bias + (size_t)block * 2 * o.part + within, bias_r);
    load_values<V>(o.gate_bias + (size_t)block * 2 * o.part + o.part + within, bias_i);
    load_values<V>(o.rate + c, rate);
    float* slot = o.state + (size_t)o.slots[request] * o.width + c;
    float* mine = carry == nullptr ? nullptr : carry + (size_t)blockIdx.y * 2 * o.width + c;
#pragma unroll
    for (int i = 0; i < V; ++i) { s[i] = 0.f; product[i] = 1.f; }
    if (WALK) load_values<V>(alone ? slot : mine, s);
    const T* u_row = static_cast<const T*>(o.u) + c;
    const T* y_row = static_cast<const T*>(o.y) + c;
    T* out_row = static_cast<T*>(o.out) + c;
    const float* z_row = o.z + (size_t)block * o.z_block + within;
    // the operands of the next AHEAD tokens are on their way while the current ones are worked on
    constexpr int AHEAD = 4;
    struct Group { float u[AHEAD][V], y[AHEAD][V], zr[AHEAD][V], zi[AHEAD][V]; };
    auto fetch = [&](Group& g, int t0) {
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            const int t = min(t0 + k, last - 1);
            load_values<V>(z_row + (size_t)t * o.z_token, g.zr[k]);
            load_values<V>(z_row + (size_t)t * o.z_token + o.part, g.zi[k]);
            load_values<V>(u_row + (size_t)t * o.width, g.u[k]);
            if (WALK) load_values<V>(y_row + (size_t)t * o.y_ld, g.y[k]);
        }
    };
    auto work = [&](const Group& g, int t0) {
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            if (t0 + k >= last) break;
            float result[V];
#pragma unroll
            for (int i = 0; i < V; ++i) {
                const float r = Math<T>::sigmoid(g.zr[k][i] + bias_r[i]);
                const float gate = Math<T>::sigmoid(g.zi[k][i] + bias_i[i]);
                float a, rest;
                Math<T>::decay(rate[i] * r, a, rest);
                s[i] = fmaf(a, s[i], rest * gate * g.u[k][i]);
                if (WALK) result[i] = s[i] * Math<T>::gelu(g.y[k][i]);
                else product[i] *= a;
            }
            if (WALK) store_values<V>(out_row + (size_t)(t0 + k) * o.width, result);
        }
    };
    Group even, odd;
    fetch(even, first);
    for (int t0 = first; t0 < last; t0 += 2 * AHEAD) {
        fetch(odd, t0 + AHEAD);
        work(even, t0);
        fetch(even, t0 + 2 * AHEAD);
        work(odd, t0 + AHEAD);
    }
    if (!WALK) {
        store_values<V>(mine, product);
        store_values<V>(mine + o.width, s);
    } else if (alone && o.write) {
        store_values<V>(slot, s);
    }
}

// Per request and channel: the starting state of every chunk (into carry[chunk][0]) and the last one
// (into the slot). A block has 32 channels; its RUNS warps take equal runs of the request's chunks:
// each joins its own chunks, the runs are joined in shared memory, then each goes over its chunks
// again from its starting state.
constexpr int RUNS = 8;
__global__ void __launch_bounds__(RUNS * 32)
gated_recurrence_chain_kernel(Operands o, float* __restrict__ carry) {
    __shared__ float decays[RUNS][32], lasts[RUNS][32];
    __shared__ int place[2];
    griddep_launch();
    griddep_wait();
    const int request = blockIdx.y, lane = threadIdx.x & 31, run = threadIdx.x >> 5;
    if (threadIdx.x == 0) {
        int before = 0, mine = 0;
        for (int r = 0; r <= request; ++r) {
            before += mine;
            mine = (o.request_start[r + 1] - o.request_start[r] + o.chunk - 1) / o.chunk;
        }
        place[0] = before;
        place[1] = mine;
    }
    __syncthreads();
    const int c = blockIdx.x * 32 + lane, chunks = place[1];
    const bool live = c < o.width;
    const int share = (chunks + RUNS - 1) / RUNS;
    const int from = min(run * share, chunks), to = min(from + share, chunks);
    float* rows = carry + (size_t)place[0] * 2 * o.width + c;
    const size_t step = 2 * (size_t)o.width;
    float* slot = o.state + (size_t)o.slots[request] * o.width + c;
    float a = 1.f, s = 0.f, now = 0.f;
    if (live) {
        now = *slot;                     // (written after the barrier, by the last run)
#pragma unroll 8
        for (int k = from; k < to; ++k) {
            const float d = rows[k * step];
            s = fmaf(d, s, rows[k * step + o.width]);
            a *= d;
        }
    }
    decays[run][lane] = a;
    lasts[run][lane] = s;
    __syncthreads();
    if (!live) return;
    for (int before = 0; before < run; ++before) now = fmaf(decays[before][lane], now, lasts[before][lane]);
#pragma unroll 8
    for (int k = from; k < to; ++k) {
        const float d = rows[k * step], last = rows[k * step + o.width];
        rows[k * step] = now;
        now = fmaf(d, now, last);
    }
    if (run == RUNS - 1 && o.write) *slot = now;
}

// A step of few single tokens: request i's token is token i. A warp has four channels, so eight rows of
// the gates' matrices, eight values of a row a lane, against four tokens at a time; the 32 sums are
// brought to one a lane (31 shuffles), and the lanes of r finish their channel and token.
__device__ __forceinline__ void load_eight(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load_eight(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 x = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&x);
#pragma unroll
    for (int i = 0; i < 4; ++i) { v[2 * i] = __low2float(pairs[i]); v[2 * i + 1] = __high2float(pairs[i]); }
}

constexpr int STEP_WARPS = 4;
template <typename T>
__global__ void __launch_bounds__(STEP_WARPS * 32)
gated_recurrence_step_kernel(Operands o, const T* __restrict__ gates, int tokens) {
    griddep_launch();
    const int lane = threadIdx.x & 31;
    const int c0 = (blockIdx.x * STEP_WARPS + (threadIdx.x >> 5)) * 4;
    if (c0 >= o.width) return;
    const int block = c0 / o.part, within = c0 - block * o.part;
    const T* rows = gates + ((size_t)block * 2 * o.part + within) * o.part;
    const int token_of = lane >> 3, channel = (lane >> 1) & 3, gate = lane & 1;
    // what depends on constants only is asked for ahead of the wait, the first weights among it
    const float bias = o.gate_bias[(size_t)block * 2 * o.part + gate * o.part + within + channel];
    const float rate = o.rate[c0 + channel];
    float w[8][8];
    auto weights = [&](int k) {
#pragma unroll
        for (int r = 0; r < 8; ++r) {
#pragma unroll
            for (int i = 0; i < 8; ++i) w[r][i] = 0.f;
            if (k < o.part) load_eight(rows + ((size_t)(r & 1) * o.part + (r >> 1)) * o.part + k, w[r]);
        }
    };
    weights(lane * 8);
    const bool one_pass = o.part <= 256;
    griddep_wait();
    const T* u = settled(static_cast<const T*>(o.u));
    const T* y = settled(static_cast<const T*>(o.y));
    for (int t0 = 0; t0 < tokens; t0 += 4) {
        const int t = t0 + token_of;
        const bool mine = gate == 0 && t < tokens;
        // the finishing lane's own operands are on their way during the product
        float* slot = nullptr;
        float state = 0.f, own = 0.f, other = 0.f;
        if (mine) {
            slot = o.state + (size_t)o.slots[t] * o.width + c0 + channel;
            state = *slot;
            own = to_float<T>(u[(size_t)t * o.width + c0 + channel]);
            other = to_float<T>(y[(size_t)t * o.y_ld + c0 + channel]);
        }
        float sums[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) sums[i] = 0.f;
        for (int k = lane * 8; k < o.part; k += 256) {
            if (!one_pass) weights(k);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                float x[8];
                load_eight(u + (size_t)min(t0 + q, tokens - 1) * o.width + (size_t)block * o.part + k, x);
#pragma unroll
                for (int r = 0; r < 8; ++r)
#pragma unroll
                    for (int i = 0; i < 8; ++i) sums[q * 8 + r] = fmaf(w[r][i], x[i], sums[q * 8 + r]);
            }
        }
        // lane l ends with the whole of sums[l]
#pragma unroll
        for (int offset = 16; offset > 0; offset >>= 1) {
            const bool upper = (lane & offset) != 0;
#pragma unroll
            for (int i = 0; i < offset; ++i) {
                const float keep = upper ? sums[i + offset] : sums[i];
                const float give = upper ? sums[i] : sums[i + offset];
                sums[i] = keep + __shfl_xor_sync(0xffffffffu, give, offset);
            }
        }
        const float opened = Math<T>::sigmoid(sums[0] + bias);
        const float input = __shfl_xor_sync(0xffffffffu, opened, 1);     // (r's lanes get i)
        if (mine) {
            float a, rest;
            Math<T>::decay(rate * opened, a, rest);
            state = fmaf(a, state, rest * input * own);
            if (o.write) *slot = state;
            static_cast<T*>(o.out)[(size_t)t * o.width + c0 + channel] =
                from_float<T>(state * Math<T>::gelu(other));
        }
    }
}

int chunk_length(int tokens, int max_portion) {
    if (max_portion <= 32) return 32;
    return tokens <= 4096 ? 16 : 32;
}

template <typename T>
void run(const Operands& o, float* carry, int tokens, int max_portion, cudaStream_t stream) {
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool pairs = o.part % 2 == 0 && o.y_ld % 2 == 0 && o.z_token % 2 == 0 && o.z_block % 2 == 0 &&
                      aligned(o.u) && (reinterpret_cast<uintptr_t>(o.y) & (sizeof(T) * 2 - 1)) == 0 &&
                      aligned(o.z) && aligned(o.gate_bias) && aligned(o.rate) && aligned(o.state) &&
                      aligned(o.out);
    const bool alone = max_portion <= o.chunk;
    const int chunks = alone ? o.requests : ceil_div_host(tokens, o.chunk) + o.requests;
    const int columns = pairs ? 2 : 1;
    const dim3 grid(ceil_div_host(o.width, 128 * columns), chunks);
    if (!alone) {
        if (pairs) launch_kernel(gated_recurrence_kernel<T, 2, false>, grid, dim3(128), 0, stream, true, o, carry, 0);
        else launch_kernel(gated_recurrence_kernel<T, 1, false>, grid, dim3(128), 0, stream, true, o, carry, 0);
        launch_kernel(gated_recurrence_chain_kernel, dim3(ceil_div_host(o.width, 32), o.requests),
                      dim3(RUNS * 32), 0, stream, true, o, carry);
    }
    if (pairs)
        launch_kernel(gated_recurrence_kernel<T, 2, true>, grid, dim3(128), 0, stream, true, o, carry, alone ? 1 : 0);
    else
        launch_kernel(gated_recurrence_kernel<T, 1, true>, grid, dim3(128), 0, stream, true, o, carry, alone ? 1 : 0);
}

}  // namespace

// Floats of scratch for mlxone_gated_recurrence (0: none is needed).
MLXONE_API long long mlxone_gated_recurrence_scratch(int tokens, int requests, int max_portion, int width) {
    const int chunk = chunk_length(tokens, max_portion);
    if (max_portion <= chunk) return 0;
    return (long long)(ceil_div_host(tokens, chunk) + requests) * 2 * width;
}

// See the head of this file. z: the gates' products in 32-bit, token t, part b, row m (r's rows, then
// i's) at z[t * z_token + b * z_block + m]. `max_portion` bounds the tokens a request brings.
MLXONE_API int mlxone_gated_recurrence(const void* u, const void* y, int y_ld, const float* z,
                                       long long z_token, long long z_block, const float* gate_bias,
                                       const float* rate, float* state, const int* slots,
                                       const int* request_start, float* carry, void* out, int tokens,
                                       int requests, int max_portion, int width, int blocks, int write,
                                       int dtype, cudaStream_t stream) {
    if (tokens == 0) return 0;
    MLXONE_REQUIRE(tokens > 0 && requests > 0 && max_portion > 0 && width > 0 && blocks > 0 &&
                       width % blocks == 0 && y_ld >= width, "gated_recurrence: bad sizes");
    Operands o{u, y, y_ld, z, z_token, z_block, gate_bias, rate, state, slots, request_start, out,
               requests, width, width / blocks, chunk_length(tokens, max_portion), write};
    MLXONE_REQUIRE(max_portion <= o.chunk || carry != nullptr, "gated_recurrence: a scratch buffer is needed");
    MLXONE_REQUIRE(ceil_div_host(tokens, o.chunk) + requests <= 65535, "gated_recurrence: too many chunks");
    if (dtype == MLXONE_BF16) run<__nv_bfloat16>(o, carry, tokens, max_portion, stream);
    else run<float>(o, carry, tokens, max_portion, stream);
    MLXONE_LAUNCH_CHECK("gated_recurrence");
    return 0;
}

// 1 if mlxone_gated_recurrence_step takes a step of `tokens` single tokens with parts of this size.
MLXONE_API int mlxone_gated_recurrence_step_fits(int tokens, int part) {
    return tokens >= 1 && tokens <= 16 && part % 8 == 0 ? 1 : 0;
}

// A step of single tokens, the gates' product included: gates [blocks, 2 part, part] in the compute
// dtype (r's rows, then i's). Token i is request i's.
MLXONE_API int mlxone_gated_recurrence_step(const void* u, const void* y, int y_ld, const void* gates,
                                            const float* gate_bias, const float* rate, float* state,
                                            const int* slots, void* out, int tokens, int width,
                                            int blocks, int write, int dtype, cudaStream_t stream) {
    if (tokens == 0) return 0;
    MLXONE_REQUIRE(width > 0 && blocks > 0 && width % blocks == 0 && y_ld >= width &&
                       mlxone_gated_recurrence_step_fits(tokens, width / blocks),
                   "gated_recurrence_step: bad sizes");
    MLXONE_REQUIRE((reinterpret_cast<uintptr_t>(u) & 15) == 0 && (reinterpret_cast<uintptr_t>(gates) & 15) == 0,
                   "gated_recurrence_step: operands must be 16-byte aligned");
    Operands o{u, y, y_ld, nullptr, 0, 0, gate_bias, rate, state, slots, nullptr, out,
               tokens, width, width / blocks, 1, write};
    const dim3 grid(ceil_div_host(width, 4 * STEP_WARPS));
    if (dtype == MLXONE_BF16)
        launch_kernel(gated_recurrence_step_kernel<__nv_bfloat16>, grid, dim3(STEP_WARPS * 32), 0, stream,
                      true, o, (const __nv_bfloat16*)gates, tokens);
    else
        launch_kernel(gated_recurrence_step_kernel<float>, grid, dim3(STEP_WARPS * 32), 0, stream, true, o,
                      (const float*)gates, tokens);
    MLXONE_LAUNCH_CHECK("gated_recurrence_step");
    return 0;
}
