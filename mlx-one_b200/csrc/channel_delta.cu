// The gated delta rule with a decay per head and key channel, over a ragged batch, with
// per-request state in 32-bit slots.
//
// projected[t] (rows `ld` values apart) = [q: G x D | k: G x D | v: H x V | beta: H | ...] (G
// query/key heads of D values, H value heads of V values; value head h reads query/key head h / (H
// / G)). The first C = 2 G D + H V channels pass a causal convolution over the last `taps` tokens
// of the request (conv [C, taps], last column the current token's) and silu. A slot's layout (S
// [H, D, V], then a ring of the convolution's inputs) is that of the rule with one decay per head.
//
// Per token and head, with the token's decays g [D] on the rows of S:
//   S = g * S;  u = beta (v - S^T k);  S = S + k u^T;  o = S^T q.
// Eight tokens are worked on together. With c_j = g_1 ... g_j (the products of the eight tokens'
// decays, per channel) and S_0 the state before the eight,
//   S_j = c_j * S_0 + sum_(i<=j) (g_(i+1) ... g_j * k_i) u_i^T, so with
//   a_j = S_0^T (c_j * k_j), b_j = S_0^T (c_j * q_j), K_ij = sum_d k_i k_j g_(i+1) ... g_j and Q_ij
//   likewise with q_j:
//   u_j = beta_j (v_j - a_j - sum_(i<j) K_ij u_i),  o_j = b_j + sum_(i<=j) Q_ij u_i.
// The u_j solve a triangular system whose inverse M (with the betas) does not depend on S:
//   u = M (v - a).
//
// A step with portions runs three kernels:
//   prepare  per (eight tokens, query/key head): convolutions + silu, unit lengths (q also times
//            D^-1/2), decays; c_j * k_j, c_j * q_j, g_(j+1) ... g_8 * k_j, c_8, M and Q.
//   scan     per (request, value head, tile of columns of S): a column of S depends on no other
//            column. A thread keeps PER rows of two columns, LANES threads share the rows
//            (products on pairs of rows, two multiply-adds an instruction); the sums over the rows
//            of all eight tokens and both columns are taken together (each exchange of the butterfly halves what a lane carries), u, o and the update follow.
//            The operands of the next 16 tokens travel to shared memory (cp.async) while the
//            current 16 are worked on. Extra blocks write the convolution's inputs into the ring.
//   finish   per (token, head): o / rms(o) * weight * sigmoid(gate), in the compute type.
// A step of single tokens runs one kernel, a block per (request, value head), which also takes
// the products of the decay's and the gate's second matrices (their rows for this head are asked
// for before the wait for the projection).
#include "delta_common.cuh"

namespace {

constexpr int GROUP = 8;             // tokens worked on together
constexpr int PREP_THREADS = 128;
constexpr int SCAN_THREADS = 256;
constexpr int CHUNK = 16;            // tokens whose operands are staged in shared memory together
constexpr int COLS = 2;              // columns of S per thread of the scan
constexpr int PAIRS = GROUP * COLS;
constexpr int SOLVE = 2 * GROUP * GROUP;    // M, then Q, both [GROUP][GROUP]
constexpr int STEP_LANES = 4;        // single-token kernel: lanes that share a column of S
constexpr int STEP_MAX_COLUMNS = 128;
constexpr int STEP_ROWS = 16;        // rows of the second matrices that a warp holds in registers

// Two 32-bit numbers in one register pair.
using Pair = unsigned long long;
__device__ __forceinline__ Pair pair_of(float lo, float hi) {
    Pair p;
    asm("mov.b64 %0, {%1, %2};" : "=l"(p) : "f"(lo), "f"(hi));
    return p;
}
__device__ __forceinline__ void halves(Pair p, float& lo, float& hi) {
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(p));
}
__device__ __forceinline__ Pair pair_fma(Pair a, Pair b, Pair c) {
    Pair d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ Pair pair_mul(Pair a, Pair b) {
    Pair d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// Sums of N values over groups of LANES lanes: each exchange halves the values a lane carries.
// Afterwards v[i] of lane l (within its group) is the sum of value l * (N / LANES) + i; where N <
// LANES every value ends up in LANES / N neighbouring lanes.
template <int N, int LANES>
__device__ __forceinline__ void reduce_many(float (&v)[N], int lane) {
    constexpr int STEPS = LANES == 32 ? 5 : LANES == 16 ? 4 : 3;
#pragma unroll
    for (int step = 0; step < STEPS; ++step) {
        const int across = LANES >> (step + 1), left = N >> step;
        if (left > 1) {
            const bool upper = (lane & across) != 0;
#pragma unroll
            for (int i = 0; i < left / 2; ++i) {
                const float keep = upper ? v[i + left / 2] : v[i];
                const float give = upper ? v[i] : v[i + left / 2];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, give, across);
            }
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], across);
        }
    }
}

// Which request and which of its groups of eight tokens block number `block` has: groups are
// counted request by request. False: there are fewer groups.
__device__ __forceinline__ bool find_group(const int* request_start, int requests, int block,
                                           int& request, int& index) {
    const int lane = threadIdx.x & 31;
    int before = 0;
    for (int base = 0; base < requests; base += 32) {
        const int r = base + lane;
        int count = 0;
        if (r < requests) count = (request_start[r + 1] - request_start[r] + GROUP - 1) / GROUP;
        int through = count;
#pragma unroll
        for (int step = 1; step < 32; step <<= 1) {
            const int other = __shfl_up_sync(0xffffffffu, through, step);
            if (lane >= step) through += other;
        }
        const unsigned hit = __ballot_sync(0xffffffffu, before + through > block);
        if (hit != 0u) {
            const int who = __ffs(hit) - 1;
            const int skipped = __shfl_sync(0xffffffffu, through - count, who);
            request = base + who;
            index = (block - before - skipped) * GROUP;
            return true;
        }
        before += __shfl_sync(0xffffffffu, through, 31);
    }
    return false;
}

// Convolution + silu of channel c for the `count` tokens from t0 on (place `index` of the portion).
template <typename T, int TAPS>
__device__ __forceinline__ void convolve(const T* projected, int ld, const float* ring,
                                         const float* conv, int channels, int taps, int t0,
                                         int index, int position, int count, int c,
                                         float (&y)[GROUP]) {
    if (TAPS > 0) {
        float in[GROUP + TAPS - 1], w[TAPS > 0 ? TAPS : 1];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = conv[(size_t)c * TAPS + j];
        if (index >= TAPS - 1 && count == GROUP) {
            // all inputs are rows of this step: one round trip for all of them
            const T* row = projected + (size_t)(t0 - (TAPS - 1)) * ld + c;
#pragma unroll
            for (int i = 0; i < GROUP + TAPS - 1; ++i) in[i] = to_float<T>(row[(size_t)i * ld]);
        } else {
#pragma unroll
            for (int i = 0; i < GROUP + TAPS - 1; ++i) {
                const int place = i - (TAPS - 1);
                in[i] = place < count
                    ? conv_input<T>(projected, ld, ring, channels, TAPS, t0, index, position, -place, c)
                    : 0.f;
            }
        }
#pragma unroll
        for (int j = 0; j < GROUP; ++j) {
            float sum = 0.f;
#pragma unroll
            for (int k = 0; k < TAPS; ++k) sum = fmaf(w[k], in[j + k], sum);
            y[j] = silu(sum);
        }
    } else {
#pragma unroll
        for (int j = 0; j < GROUP; ++j) {
            float sum = 0.f;
            if (j < count)
                for (int k = 0; k < taps; ++k)
                    sum = fmaf(conv[(size_t)c * taps + k],
                               conv_input<T>(projected, ld, ring, channels, taps, t0 + j, index + j,
                                             position + j, taps - 1 - k, c), sum);
            y[j] = silu(sum);
        }
    }
}

// ------------------------------------------------------------------ prepare
// Grid (groups of eight tokens, G). steps [tokens, H, D]: the decay's second product. Results:
// kc, qc, ks [tokens, H, D] (c_j * k_j, c_j * q_j, g_(j+1) ... g_8 * k_j), v [tokens, H, V]; at the
// group's first token: cum [tokens, H, D] (c_8) and solve [tokens, H, SOLVE] (M and Q, row j: what
// token j takes of token i). Dynamic shared memory: q and k [GROUP][D].
template <typename T, int TAPS>
__global__ void __launch_bounds__(PREP_THREADS, 4)
channel_prepare_kernel(const T* __restrict__ projected, const float* __restrict__ steps,
                       const float* __restrict__ conv, const float* __restrict__ a_log,
                       const float* __restrict__ dt_bias, const float* __restrict__ state,
                       const int* __restrict__ slots, const int* __restrict__ request_start,
                       const int* __restrict__ history, float* __restrict__ kc,
                       float* __restrict__ qc, float* __restrict__ ks, float* __restrict__ v_out,
                       float* __restrict__ cum, float* __restrict__ solve, DeltaSizes sizes,
                       int requests, float unit_eps, int ld) {
    constexpr int WARPS = PREP_THREADS / 32;
    extern __shared__ float rows[];
    __shared__ float sums[WARPS][64];
    __shared__ float beta[GROUP];
    griddep_wait();
    projected = settled(projected);
    steps = settled(steps);
    state = settled(state);
    int r, index;
    if (!find_group(request_start, requests, blockIdx.x, r, index)) return;
    const int g = blockIdx.y;
    const int G = sizes.kv_heads, D = sizes.key_dim, H = sizes.heads, V = sizes.value_dim;
    const int taps = sizes.taps, channels = sizes.channels(), qk = sizes.qk();
    const int t0 = request_start[r] + index;
    const int count = min(GROUP, request_start[r + 1] - t0);
    const int position = history[r] + index;
    const float* ring = state + (size_t)slots[r] * sizes.state() + sizes.matrices();
    float* qs = rows;
    float* keys = rows + GROUP * D;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    for (int i = threadIdx.x; i < 2 * D; i += PREP_THREADS) {
        const bool is_key = i >= D;
        const int e = is_key ? i - D : i;
        float y[GROUP];
        convolve<T, TAPS>(projected, ld, ring, conv, channels, taps, t0, index, position, count,
                          (is_key ? qk : 0) + g * D + e, y);
        float* to = is_key ? keys : qs;
#pragma unroll
        for (int j = 0; j < GROUP; ++j) to[j * D + e] = j < count ? y[j] : 0.f;
    }
    __syncthreads();
    // unit lengths: a warp per row
    for (int row = warp; row < 2 * GROUP; row += WARPS) {
        float* x = rows + row * D;
        float squares = 0.f;
        for (int e = lane; e < D; e += 32) squares = fmaf(x[e], x[e], squares);
        squares = warp_sum(squares);
        const float factor = (row < GROUP ? rsqrtf((float)D) : 1.f) / sqrtf(squares + unit_eps);
        for (int e = lane; e < D; e += 32) x[e] *= factor;
    }
    __syncthreads();

    const int share = H / G;
    for (int h = g * share; h < (g + 1) * share; ++h) {
        const float rate = -expf(a_log[h]);
        // K_ij (i < j) and Q_ij (i <= j), this thread's channels: 28 + 36 sums
        float part[64];
#pragma unroll
        for (int i = 0; i < 64; ++i) part[i] = 0.f;
        for (int d = threadIdx.x; d < D; d += PREP_THREADS) {
            float decay[GROUP], k[GROUP], q[GROUP];
            const float bias = dt_bias[h * D + d];
#pragma unroll
            for (int j = 0; j < GROUP; ++j)
                decay[j] = steps[((size_t)(t0 + min(j, count - 1)) * H + h) * D + d];
#pragma unroll
            for (int j = 0; j < GROUP; ++j) {
                k[j] = keys[j * D + d];
                q[j] = qs[j * D + d];
                decay[j] = j < count ? expf(rate * softplus(decay[j] + bias)) : 1.f;
            }
            float before = 1.f;
#pragma unroll
            for (int j = 0; j < GROUP; ++j) {
                before *= decay[j];
                if (j < count) {
                    const size_t at = ((size_t)(t0 + j) * H + h) * D + d;
                    kc[at] = before * k[j];
                    qc[at] = before * q[j];
                }
            }
            cum[((size_t)t0 * H + h) * D + d] = before;
            float after = 1.f;
#pragma unroll
            for (int j = GROUP - 1; j >= 0; --j) {
                if (j < count) ks[((size_t)(t0 + j) * H + h) * D + d] = after * k[j];
                after *= decay[j];
            }
            int at_k = 0, at_q = 28;
#pragma unroll
            for (int i = 0; i < GROUP; ++i) {
                float carried = k[i];
                part[at_q] = fmaf(carried, q[i], part[at_q]);
                ++at_q;
#pragma unroll
                for (int j = i + 1; j < GROUP; ++j) {
                    carried *= decay[j];
                    part[at_k] = fmaf(carried, k[j], part[at_k]);
                    part[at_q] = fmaf(carried, q[j], part[at_q]);
                    ++at_k;
                    ++at_q;
                }
            }
        }
        reduce_many<64, 32>(part, lane);
        sums[warp][2 * lane] = part[0];
        sums[warp][2 * lane + 1] = part[1];
        if (threadIdx.x < GROUP)
            beta[threadIdx.x] = threadIdx.x < count
                ? sigmoid(to_float<T>(projected[(size_t)(t0 + threadIdx.x) * ld + channels + h])) : 0.f;
        __syncthreads();
        if (threadIdx.x < 64) {
            float all = 0.f;
#pragma unroll
            for (int w = 0; w < WARPS; ++w) all += sums[w][threadIdx.x];
            sums[0][threadIdx.x] = all;
        }
        __syncthreads();
        float* to = solve + ((size_t)t0 * H + h) * SOLVE;
        // value number of K_ij, i < j, and of Q_ij, i <= j
        auto number_k = [](int i, int j) { return i * (2 * GROUP - 1 - i) / 2 + (j - i - 1); };
        auto number_q = [](int i, int j) { return 28 + i * (2 * GROUP + 1 - i) / 2 + (j - i); };
        if (threadIdx.x < GROUP) {
            // column i of M: M_ii = beta_i, M_ji = -beta_j sum_(i<=l<j) K_lj M_li
            const int i = threadIdx.x;
            float column[GROUP];
#pragma unroll
            for (int j = 0; j < GROUP; ++j) {
                float sum = 0.f;
#pragma unroll
                for (int l = 0; l < j; ++l)
                    if (l >= i) sum = fmaf(sums[0][number_k(l, j)], column[l], sum);
                column[j] = j < i ? 0.f : j == i ? beta[j] : -beta[j] * sum;
                to[j * GROUP + i] = column[j];
            }
        } else if (threadIdx.x >= 64) {
            const int item = threadIdx.x - 64, j = item / GROUP, i = item % GROUP;
            to[GROUP * GROUP + item] = i <= j ? sums[0][number_q(i, j)] : 0.f;
        }
        // this head's values
        for (int e = threadIdx.x; e < V; e += PREP_THREADS) {
            float y[GROUP];
            convolve<T, TAPS>(projected, ld, ring, conv, channels, taps, t0, index, position, count,
                              2 * qk + h * V + e, y);
#pragma unroll
            for (int j = 0; j < GROUP; ++j)
                if (j < count) v_out[((size_t)(t0 + j) * H + h) * V + e] = y[j];
        }
        __syncthreads();
    }
    // (the scan's blocks would only wait beside this kernel's if they were let in earlier)
    griddep_launch();
}

// ------------------------------------------------------------------ scan
// Grid (column tiles, H + 1, requests); blocks with blockIdx.y == H write the convolution's
// inputs into the ring. Lane l of LANES keeps rows l * PER .. of COLS columns. Dynamic shared
// memory: two buffers of kc, qc, ks [CHUNK][ROWS], cum [CHUNK / GROUP][ROWS], solve [CHUNK /
// GROUP][SOLVE], v [CHUNK][COLUMNS]; then per group of lanes v - a and u, [COLS][GROUP] each.
template <int PER, int LANES>
struct ScanShape {
    static constexpr int ROWS = PER * LANES;
    static constexpr int TEAMS = SCAN_THREADS / LANES;       // groups of lanes
    static constexpr int COLUMNS = TEAMS * COLS;             // columns of S per block
    static constexpr int BUFFER = 3 * CHUNK * ROWS + (CHUNK / GROUP) * (ROWS + SOLVE) + CHUNK * COLUMNS;
    static constexpr int TOTAL = 2 * BUFFER + TEAMS * 2 * PAIRS;
};

template <typename T, int PER, int LANES>
__global__ void __launch_bounds__(SCAN_THREADS, 1)
channel_scan_kernel(const float* __restrict__ kc, const float* __restrict__ qc,
                    const float* __restrict__ ks, const float* __restrict__ v_in,
                    const float* __restrict__ cum, const float* __restrict__ solve,
                    const T* __restrict__ projected, float* __restrict__ state,
                    const int* __restrict__ slots, const int* __restrict__ request_start,
                    const int* __restrict__ history, float* __restrict__ out, DeltaSizes sizes,
                    int write, int ld) {
    using Shape = ScanShape<PER, LANES>;
    constexpr int ROWS = Shape::ROWS, COLUMNS = Shape::COLUMNS, BUFFER = Shape::BUFFER;
    // What a lane holds after the sums: with 32 lanes one of the 32 values, a of (column, token)
    // pair l in the lower half of the warp and b of pair l - 16 in the upper; with fewer lanes a and
    // b of OWN pairs.
    constexpr bool SPLIT = LANES == 2 * PAIRS;
    constexpr int OWN = SPLIT ? 1 : PAIRS / LANES;
    extern __shared__ __align__(16) float staged[];
    griddep_wait();
    kc = settled(kc);
    qc = settled(qc);
    ks = settled(ks);
    v_in = settled(v_in);
    cum = settled(cum);
    solve = settled(solve);
    projected = settled(projected);
    state = settled(state);
    const int r = blockIdx.z;
    const int first = request_start[r], last = request_start[r + 1];
    const int H = sizes.heads, D = sizes.key_dim, V = sizes.value_dim;
    float* slot = state + (size_t)slots[r] * sizes.state();
    if (blockIdx.y == H) {
        // the inputs of the portion's last positions (at most taps of them) go into the ring
        griddep_launch();
        if (!write) return;
        const int channels = sizes.channels(), taps = sizes.taps;
        const int n = last - first, kept = min(n, taps);
        float* ring = slot + sizes.matrices();
        for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < channels;
             c += gridDim.x * blockDim.x)
            for (int index = n - kept; index < n; ++index)
                ring[(size_t)((history[r] + index) % taps) * channels + c] =
                    to_float<T>(projected[(size_t)(first + index) * ld + c]);
        return;
    }
    const int h = blockIdx.y;
    const int lane = threadIdx.x & (LANES - 1), team = threadIdx.x / LANES;
    const int column0 = blockIdx.x * COLUMNS + team * COLS;
    float* matrix = slot + (size_t)h * D * V;
    Pair S[COLS][PER / 2];                            // rows 2 e and 2 e + 1 of this lane's
    auto stored = [&](int c, int e) {
        const int row = lane * PER + e;
        return column0 + c < V && row < D ? matrix[(size_t)row * V + column0 + c] : 0.f;
    };
#pragma unroll
    for (int e = 0; e < PER; e += 2)
#pragma unroll
        for (int c = 0; c < COLS; ++c) S[c][e / 2] = pair_of(stored(c, e), stored(c, e + 1));
    const bool quads = D % 4 == 0 && ((reinterpret_cast<uintptr_t>(kc) | reinterpret_cast<uintptr_t>(qc) |
                                       reinterpret_cast<uintptr_t>(ks) | reinterpret_cast<uintptr_t>(cum)) & 15) == 0;
    const bool value_quads = V % 4 == 0 && (reinterpret_cast<uintptr_t>(v_in) & 15) == 0;
    // rows behind D, columns behind V and places behind the portion's end stay finite
    for (int i = threadIdx.x; i < Shape::TOTAL; i += SCAN_THREADS) staged[i] = 0.f;
    __syncthreads();
    float* own = staged + 2 * BUFFER + team * 2 * PAIRS;
    auto copy_row = [&](float* to, const float* from, bool wide, int values, int place, int places) {
        if (wide) {
            for (int i = place * 4; i < values; i += places * 4) copy_async_16(to + i, from + i);
        } else {
            for (int i = place; i < values; i += places) copy_async_4(to + i, from + i);
        }
    };
    auto fetch = [&](int base, int buffer) {
        const int count = min(CHUNK, last - base);
        float* at = staged + buffer * BUFFER;
        const int warp = threadIdx.x >> 5, in_warp = threadIdx.x & 31;
        for (int t = warp; t < count; t += SCAN_THREADS / 32) {
            const size_t from = ((size_t)(base + t) * H + h) * D;
            copy_row(at + t * ROWS, kc + from, quads, D, in_warp, 32);
            copy_row(at + (CHUNK + t) * ROWS, qc + from, quads, D, in_warp, 32);
            copy_row(at + (2 * CHUNK + t) * ROWS, ks + from, quads, D, in_warp, 32);
        }
        at += 3 * CHUNK * ROWS;
        for (int group = warp; group * GROUP < count; group += SCAN_THREADS / 32) {
            const size_t from = (size_t)(base + group * GROUP) * H + h;
            copy_row(at + group * ROWS, cum + from * D, quads, D, in_warp, 32);
            copy_row(at + (CHUNK / GROUP) * ROWS + group * SOLVE, solve + from * SOLVE, true, SOLVE,
                     in_warp, 32);
        }
        at += (CHUNK / GROUP) * (ROWS + SOLVE);
        const int wide = min(COLUMNS, V - (int)blockIdx.x * COLUMNS);
        constexpr int LANES_A_ROW = COLUMNS / 4;
        for (int t = threadIdx.x / LANES_A_ROW; t < count; t += SCAN_THREADS / LANES_A_ROW)
            copy_row(at + t * COLUMNS, v_in + ((size_t)(base + t) * H + h) * V + blockIdx.x * COLUMNS,
                     value_quads, wide, threadIdx.x % LANES_A_ROW, LANES_A_ROW);
        copy_commit();
    };
    if (first < last) fetch(first, 0);
    int buffer = 0;
    for (int base = first; base < last; base += CHUNK, buffer ^= 1) {
        const int count = min(CHUNK, last - base);
        if (base + CHUNK < last) {
            fetch(base + CHUNK, buffer ^ 1);
            copy_wait_for<1>();
        } else {
            copy_wait_for<0>();
        }
        __syncthreads();
        const float* kcs = staged + buffer * BUFFER;
        const float* qcs = kcs + CHUNK * ROWS;
        const float* kss = qcs + CHUNK * ROWS;
        const float* cums = kss + CHUNK * ROWS;
        const float* solves = cums + (CHUNK / GROUP) * ROWS;
        const float* vs = solves + (CHUNK / GROUP) * SOLVE;
        for (int t0 = 0; t0 < count; t0 += GROUP) {
            // a and b of every (column, token) pair c * GROUP + j
            float sum[2 * PAIRS];
#pragma unroll
            for (int j = 0; j < GROUP; ++j) {
                Pair a[COLS], b[COLS];
#pragma unroll
                for (int e = 0; e < PER; e += 4) {
                    const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(kcs + (t0 + j) * ROWS + lane * PER + e);
                    const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(qcs + (t0 + j) * ROWS + lane * PER + e);
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        a[c] = e == 0 ? pair_mul(S[c][0], k4.x) : pair_fma(S[c][e / 2], k4.x, a[c]);
                        b[c] = e == 0 ? pair_mul(S[c][0], q4.x) : pair_fma(S[c][e / 2], q4.x, b[c]);
                        a[c] = pair_fma(S[c][e / 2 + 1], k4.y, a[c]);
                        b[c] = pair_fma(S[c][e / 2 + 1], q4.y, b[c]);
                    }
                }
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    const int pair = c * GROUP + j;
                    float lo, hi;
                    halves(a[c], lo, hi);
                    sum[SPLIT ? pair : 2 * pair] = lo + hi;
                    halves(b[c], lo, hi);
                    sum[SPLIT ? PAIRS + pair : 2 * pair + 1] = lo + hi;
                }
            }
            reduce_many<2 * PAIRS, LANES>(sum, lane);
            const float* solve_group = solves + (t0 / GROUP) * SOLVE;
            const int first_pair = SPLIT ? lane % PAIRS : lane * OWN;
#pragma unroll
            for (int i = 0; i < OWN; ++i) {
                const int pair = first_pair + i, c = pair / GROUP, j = pair % GROUP;
                if (!SPLIT || lane < PAIRS)
                    own[pair] = vs[(t0 + j) * COLUMNS + team * COLS + c] - sum[2 * i];
            }
            __syncwarp();
#pragma unroll
            for (int i = 0; i < OWN; ++i) {
                const int pair = first_pair + i, c = pair / GROUP, j = pair % GROUP;
                float u = 0.f;
#pragma unroll
                for (int l = 0; l < GROUP; l += 4) {
                    const float4 m = *reinterpret_cast<const float4*>(solve_group + j * GROUP + l);
                    const float4 w = *reinterpret_cast<const float4*>(own + c * GROUP + l);
                    u = fmaf(m.x, w.x, u); u = fmaf(m.y, w.y, u);
                    u = fmaf(m.z, w.z, u); u = fmaf(m.w, w.w, u);
                }
                if (!SPLIT || lane < PAIRS) own[PAIRS + pair] = u;
            }
            __syncwarp();
#pragma unroll
            for (int i = 0; i < OWN; ++i) {
                const int pair = first_pair + i, c = pair / GROUP, j = pair % GROUP;
                float o = sum[SPLIT ? 0 : 2 * i + 1];
#pragma unroll
                for (int l = 0; l < GROUP; l += 4) {
                    const float4 m = *reinterpret_cast<const float4*>(solve_group + GROUP * GROUP + j * GROUP + l);
                    const float4 w = *reinterpret_cast<const float4*>(own + PAIRS + c * GROUP + l);
                    o = fmaf(m.x, w.x, o); o = fmaf(m.y, w.y, o);
                    o = fmaf(m.z, w.z, o); o = fmaf(m.w, w.w, o);
                }
                if ((!SPLIT || lane >= PAIRS) && t0 + j < count && column0 + c < V)
                    out[((size_t)(base + t0 + j) * H + h) * V + column0 + c] = o;
            }
            // S = c_8 * S + sum_j (g_(j+1) ... g_8 * k_j) u_j
#pragma unroll
            for (int e = 0; e < PER; e += 4) {
                const ulonglong2 c4 = *reinterpret_cast<const ulonglong2*>(cums + (t0 / GROUP) * ROWS + lane * PER + e);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    S[c][e / 2] = pair_mul(S[c][e / 2], c4.x);
                    S[c][e / 2 + 1] = pair_mul(S[c][e / 2 + 1], c4.y);
                }
            }
#pragma unroll
            for (int j = 0; j < GROUP; j += 4) {
                Pair u[COLS][4];
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    const float4 w = *reinterpret_cast<const float4*>(own + PAIRS + c * GROUP + j);
                    u[c][0] = pair_of(w.x, w.x); u[c][1] = pair_of(w.y, w.y);
                    u[c][2] = pair_of(w.z, w.z); u[c][3] = pair_of(w.w, w.w);
                }
#pragma unroll
                for (int step = 0; step < 4; ++step) {
#pragma unroll
                    for (int e = 0; e < PER; e += 4) {
                        const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(kss + (t0 + j + step) * ROWS + lane * PER + e);
#pragma unroll
                        for (int c = 0; c < COLS; ++c) {
                            S[c][e / 2] = pair_fma(k4.x, u[c][step], S[c][e / 2]);
                            S[c][e / 2 + 1] = pair_fma(k4.y, u[c][step], S[c][e / 2 + 1]);
                        }
                    }
                }
            }
            __syncwarp();         // (v - a is written again by the next group)
        }
        __syncthreads();          // the buffer is fetched into again two rounds on
    }
    griddep_launch();
    if (write) {
#pragma unroll
        for (int e = 0; e < PER; e += 2)
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
                const int row = lane * PER + e;
                float lo, hi;
                halves(S[c][e / 2], lo, hi);
                if (column0 + c < V && row < D) matrix[(size_t)row * V + column0 + c] = lo;
                if (column0 + c < V && row + 1 < D) matrix[(size_t)(row + 1) * V + column0 + c] = hi;
            }
    }
}

// ------------------------------------------------------------------ a step of single tokens
// One block per (value head, request); request r brings token r. Threads: STEP_LANES per column
// of S. decay_up [H * D, decay_rank] and gate_up [H * V, gate_rank] in the compute type, their
// inner rows at columns decay_at and gate_at of the projection. `held`: every warp's rows of the
// two matrices fit into its registers (16-bit, ranks of at most 128 that are multiples of 4).
// Dynamic shared memory: q, k, decays [ROWS each], v, o, gate [V each], the inner rows, scalars.
template <typename T>
__device__ __forceinline__ float row_product(const T* w, const float* x, int n, int lane) {
    float sum = 0.f;
    for (int e = lane; e < n; e += 32) sum = fmaf(to_float<T>(w[e]), x[e], sum);
    return warp_sum(sum);
}

template <typename T, int PER>
__global__ void __launch_bounds__(STEP_LANES * STEP_MAX_COLUMNS)
channel_step_kernel(const T* __restrict__ projected, const T* __restrict__ decay_up, int decay_at,
                    int decay_rank, const T* __restrict__ gate_up, int gate_at, int gate_rank,
                    const float* __restrict__ conv, const float* __restrict__ a_log,
                    const float* __restrict__ dt_bias, const float* __restrict__ norm_weight,
                    float eps, float unit_eps, float* __restrict__ state,
                    const int* __restrict__ slots, const int* __restrict__ history,
                    T* __restrict__ mixed, DeltaSizes sizes, int write, int ld, int held) {
    constexpr int LANES = STEP_LANES;
    constexpr int ROWS = PER * LANES;
    extern __shared__ __align__(16) float staged[];
    const int H = sizes.heads, G = sizes.kv_heads, D = sizes.key_dim, V = sizes.value_dim;
    const int taps = sizes.taps, channels = sizes.channels();
    float* qs = staged;
    float* keys = qs + ROWS;
    float* decays = keys + ROWS;
    float* inner_decay = decays + ROWS;                       // 16-byte aligned: ROWS % 4 == 0
    float* inner_gate = inner_decay + (decay_rank + 3) / 4 * 4;
    float* vs = inner_gate + (gate_rank + 3) / 4 * 4;
    float* os = vs + V;
    float* gates = os + V;
    float* scalars = gates + V;              // k.q, beta, 1 / rms(o)
    griddep_launch();
    const int h = blockIdx.x, r = blockIdx.y, g = h / (H / G);
    const int lane = threadIdx.x & (LANES - 1), column = threadIdx.x / LANES;
    const bool live = column < V;
    const int warp = threadIdx.x >> 5, in_warp = threadIdx.x & 31, warps = blockDim.x >> 5;
    // weights, and the head's matrix, which an earlier step wrote: their loads start before the
    // wait for the kernel that writes this step's projection
    float* slot = state + (size_t)slots[r] * sizes.state();
    float* matrix = slot + (size_t)h * D * V;
    float S[PER];
#pragma unroll
    for (int e = 0; e < PER; ++e) {
        const int row = (e / 4) * (4 * LANES) + lane * 4 + e % 4;
        S[e] = live && row < D ? matrix[(size_t)row * V + column] : 0.f;
    }
    // row `item` of the two matrices' rows of this head: the decay's D, then the gate's V
    uint2 weights[STEP_ROWS];
    if (held) {
#pragma unroll
        for (int i = 0; i < STEP_ROWS; ++i) {
            const int item = warp + i * warps;
            weights[i] = make_uint2(0u, 0u);
            const bool is_decay = item < D;
            const int rank = is_decay ? decay_rank : gate_rank;
            if (item < D + V && in_warp * 4 < rank)
                weights[i] = *reinterpret_cast<const uint2*>(
                    (is_decay ? decay_up + ((size_t)h * D + item) * rank
                              : gate_up + ((size_t)h * V + item - D) * rank) + in_warp * 4);
        }
    }
    for (int i = threadIdx.x; i < 3 * ROWS; i += blockDim.x) qs[i] = 0.f;      // q, k, decays, padded
    __syncthreads();
    griddep_wait();
    projected = settled(projected);
    const int position = history[r];
    float* ring = settled(slot + sizes.matrices());
    const T* row_in = projected + (size_t)r * ld;
    for (int i = threadIdx.x; i < decay_rank; i += blockDim.x)
        inner_decay[i] = to_float<T>(row_in[decay_at + i]);
    for (int i = threadIdx.x; i < gate_rank; i += blockDim.x)
        inner_gate[i] = to_float<T>(row_in[gate_at + i]);
    // convolution + silu of this block's channels: its key head's q and k, its own v
    const bool owner = h % (H / G) == 0;         // writes the key head's inputs into the ring
    for (int i = threadIdx.x; i < 2 * D + V; i += blockDim.x) {
        const int c = i < D ? g * D + i : (i < 2 * D ? sizes.qk() + g * D + (i - D)
                                                     : 2 * sizes.qk() + h * V + (i - 2 * D));
        const float now = to_float<T>(row_in[c]);
        float y = conv[(size_t)c * taps + taps - 1] * now;
        for (int j = 0; j + 1 < taps; ++j) {
            const int before = position - (taps - 1 - j);
            if (before >= 0)
                y = fmaf(conv[(size_t)c * taps + j], ring[(size_t)(before % taps) * channels + c], y);
        }
        if (write && (i >= 2 * D || owner)) ring[(size_t)(position % taps) * channels + c] = now;
        const float value = silu(y);
        if (i < D) qs[i] = value;
        else if (i < 2 * D) keys[i - D] = value;
        else vs[i - 2 * D] = value;
    }
    __syncthreads();
    // the decays and the gate: the second matrices' products with the inner rows
    const float rate = -expf(a_log[h]);
    auto finish = [&](int item, float value) {
        if (item < D) decays[item] = expf(rate * softplus(value + dt_bias[h * D + item]));
        else gates[item - D] = sigmoid(value);
    };
    if (held) {
        float product[STEP_ROWS];
        const float4 x_decay = in_warp * 4 < decay_rank
            ? *reinterpret_cast<const float4*>(inner_decay + in_warp * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 x_gate = in_warp * 4 < gate_rank
            ? *reinterpret_cast<const float4*>(inner_gate + in_warp * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < STEP_ROWS; ++i) {
            const float4 x = warp + i * warps < D ? x_decay : x_gate;
            const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&weights[i].x));
            const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&weights[i].y));
            product[i] = fmaf(lo.x, x.x, fmaf(lo.y, x.y, fmaf(hi.x, x.z, hi.y * x.w)));
        }
        reduce_many<STEP_ROWS, 32>(product, in_warp);         // row in_warp / 2 of this warp's
        const int item = warp + (in_warp >> 1) * warps;
        if ((in_warp & 1) == 0 && item < D + V) finish(item, product[0]);
    } else {
        for (int item = warp; item < D + V; item += warps) {
            const float value = item < D
                ? row_product<T>(decay_up + ((size_t)h * D + item) * decay_rank, inner_decay, decay_rank, in_warp)
                : row_product<T>(gate_up + ((size_t)h * V + item - D) * gate_rank, inner_gate, gate_rank, in_warp);
            if (in_warp == 0) finish(item, value);
        }
    }
    if (warp == 0) {
        float qq = 0.f, kk = 0.f;
        for (int e = in_warp; e < D; e += 32) {
            qq = fmaf(qs[e], qs[e], qq);
            kk = fmaf(keys[e], keys[e], kk);
        }
        qq = warp_sum(qq);
        kk = warp_sum(kk);
        const float q_scale = rsqrtf((float)D) / sqrtf(qq + unit_eps);
        const float k_scale = 1.f / sqrtf(kk + unit_eps);
        float dot = 0.f;
        for (int e = in_warp; e < D; e += 32) {
            const float qv = qs[e] * q_scale, kv = keys[e] * k_scale;
            qs[e] = qv;
            keys[e] = kv;
            dot = fmaf(qv, kv, dot);
        }
        dot = warp_sum(dot);
        if (in_warp == 0) {
            scalars[0] = dot;
            scalars[1] = sigmoid(to_float<T>(row_in[channels + h]));
        }
    }
    __syncthreads();
    {
        float wk[4] = {0.f, 0.f, 0.f, 0.f}, wq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int e = 0; e < PER; e += 4) {
            const int at = (e / 4) * (4 * LANES) + lane * 4;
            const float4 k4 = *reinterpret_cast<const float4*>(keys + at);
            const float4 q4 = *reinterpret_cast<const float4*>(qs + at);
            const float4 d4 = *reinterpret_cast<const float4*>(decays + at);
            S[e] *= d4.x; S[e + 1] *= d4.y; S[e + 2] *= d4.z; S[e + 3] *= d4.w;
            wk[0] = fmaf(S[e], k4.x, wk[0]); wq[0] = fmaf(S[e], q4.x, wq[0]);
            wk[1] = fmaf(S[e + 1], k4.y, wk[1]); wq[1] = fmaf(S[e + 1], q4.y, wq[1]);
            wk[2] = fmaf(S[e + 2], k4.z, wk[2]); wq[2] = fmaf(S[e + 2], q4.z, wq[2]);
            wk[3] = fmaf(S[e + 3], k4.w, wk[3]); wq[3] = fmaf(S[e + 3], q4.w, wq[3]);
        }
        float with_k = (wk[0] + wk[1]) + (wk[2] + wk[3]);
        float with_q = (wq[0] + wq[1]) + (wq[2] + wq[3]);
#pragma unroll
        for (int across = 1; across < LANES; across <<= 1) {
            with_k += __shfl_xor_sync(0xffffffffu, with_k, across);
            with_q += __shfl_xor_sync(0xffffffffu, with_q, across);
        }
        const float u = scalars[1] * ((live ? vs[column] : 0.f) - with_k);
        if (write && live) {
#pragma unroll
            for (int e = 0; e < PER; ++e) {
                const int row = (e / 4) * (4 * LANES) + lane * 4 + e % 4;
                if (row < D) matrix[(size_t)row * V + column] = fmaf(keys[row], u, S[e]);
            }
        }
        if (live && lane == 0) os[column] = fmaf(u, scalars[0], with_q);
    }
    __syncthreads();
    if (warp == 0) {
        float sum = 0.f;
        for (int e = in_warp; e < V; e += 32) sum = fmaf(os[e], os[e], sum);
        sum = warp_sum(sum);
        if (in_warp == 0) scalars[2] = 1.f / sqrtf(sum / (float)V + eps);
    }
    __syncthreads();
    for (int e = threadIdx.x; e < V; e += blockDim.x)
        mixed[(size_t)r * sizes.inner() + (size_t)h * V + e] =
            from_float<T>(os[e] * scalars[2] * norm_weight[e] * gates[e]);
}

// ------------------------------------------------------------------ finish
// One warp per (token, head): mixed[t, h, :] = o / sqrt(mean(o^2) + eps) * weight * sigmoid(gate).
template <typename T>
__global__ void __launch_bounds__(256)
channel_finish_kernel(const float* __restrict__ o, const T* __restrict__ gate,
                      const float* __restrict__ weight, T* __restrict__ mixed, long long items,
                      int V, float eps) {
    griddep_launch();
    griddep_wait();
    o = settled(o);
    gate = settled(gate);
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= items) return;
    const int lane = threadIdx.x & 31;
    const float* row = o + item * V;
    float sum = 0.f;
    for (int e = lane; e < V; e += 32) sum = fmaf(row[e], row[e], sum);
    sum = warp_sum(sum);
    const float inv = 1.f / sqrtf(sum / (float)V + eps);
    for (int e = lane; e < V; e += 32)
        mixed[item * V + e] =
            from_float<T>(row[e] * inv * weight[e] * sigmoid(to_float<T>(gate[item * V + e])));
}

struct DeltaCall {
    const void* projected;
    int ld;
    const float* conv;
    const float* a_log;
    const float* dt_bias;
    const float* norm_weight;
    float eps, unit_eps;
    float* state;
    const int* slots;
    const int* request_start;
    const int* history;
    void* mixed;
    int tokens, requests;
    DeltaSizes sizes;
    int write;
    cudaStream_t stream;
};

template <typename T>
int launch_step(const DeltaCall& call, const void* decay_up, int decay_at, int decay_rank,
                const void* gate_up, int gate_at, int gate_rank) {
    const int D = call.sizes.key_dim, V = call.sizes.value_dim, H = call.sizes.heads;
    const int per = D <= 16 ? 4 : D <= 32 ? 8 : D <= 64 ? 16 : D <= 128 ? 32 : 64;
    const size_t shared = (size_t)(3 * per * STEP_LANES + (decay_rank + 3) / 4 * 4 +
                                   (gate_rank + 3) / 4 * 4 + 3 * V + 4) * sizeof(float);
    MLXONE_REQUIRE(shared <= 48 * 1024, "channel delta rule: inner rows of %d and %d do not fit",
                   decay_rank, gate_rank);
    const int threads = (STEP_LANES * V + 31) / 32 * 32;
    const auto fits = [](const void* p, int rank) {
        return rank % 4 == 0 && rank <= 128 && (reinterpret_cast<uintptr_t>(p) & 7) == 0;
    };
    const int held = sizeof(T) == 2 && fits(decay_up, decay_rank) && fits(gate_up, gate_rank) &&
                     D + V <= STEP_ROWS * (threads / 32) && per <= 32;
#define STEP(PER)                                                                                   \
    launch_kernel(channel_step_kernel<T, PER>, dim3(H, call.requests), dim3(threads), shared,       \
                  call.stream, true, (const T*)call.projected, (const T*)decay_up, decay_at,        \
                  decay_rank, (const T*)gate_up, gate_at, gate_rank, call.conv, call.a_log,         \
                  call.dt_bias, call.norm_weight, call.eps, call.unit_eps, call.state, call.slots,  \
                  call.history, (T*)call.mixed, call.sizes, call.write, call.ld, held)
    if (per == 4) STEP(4);
    else if (per == 8) STEP(8);
    else if (per == 16) STEP(16);
    else if (per == 32) STEP(32);
    else STEP(64);
#undef STEP
    MLXONE_LAUNCH_CHECK("channel delta rule (single tokens)");
    return 0;
}

template <typename T, int PER, int LANES>
int launch_scan(const DeltaCall& call, const float* kc, const float* qc, const float* ks, const float* v,
                const float* cum, const float* solve, float* o) {
    using Shape = ScanShape<PER, LANES>;
    const dim3 grid(ceil_div_host(call.sizes.value_dim, Shape::COLUMNS), call.sizes.heads + 1,
                    call.requests);
    constexpr size_t shared = (size_t)Shape::TOTAL * sizeof(float);
    if (shared > 48 * 1024)
        cudaFuncSetAttribute(channel_scan_kernel<T, PER, LANES>,
                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
    launch_kernel(channel_scan_kernel<T, PER, LANES>, grid, dim3(SCAN_THREADS), shared, call.stream,
                  true, kc, qc, ks, v, cum, solve, (const T*)call.projected, call.state, call.slots,
                  call.request_start, call.history, o, call.sizes, call.write, call.ld);
    MLXONE_LAUNCH_CHECK("channel delta rule (scan)");
    return 0;
}

template <typename T>
int launch_portions(const DeltaCall& call, const float* steps, const void* gate, float* scratch) {
    const int G = call.sizes.kv_heads, D = call.sizes.key_dim, H = call.sizes.heads,
              V = call.sizes.value_dim;
    // scratch: solve [tokens, H, SOLVE]; kc, qc, ks, cum [tokens, H, D]; v, o [tokens, H, V]
    const size_t wide = (size_t)call.tokens * H * D, values = (size_t)call.tokens * H * V;
    float* solve = scratch;
    float* kc = solve + (size_t)call.tokens * H * SOLVE;
    float* qc = kc + wide;
    float* ks = qc + wide;
    float* cum = ks + wide;
    float* v = cum + wide;
    float* o = v + values;
    const dim3 grid(call.tokens / GROUP + call.requests, G);
    const size_t shared = (size_t)2 * GROUP * D * sizeof(float);
    auto prepare = [&](auto kernel) {
        launch_kernel(kernel, grid, dim3(PREP_THREADS), shared, call.stream, true,
                      (const T*)call.projected, steps, call.conv, call.a_log, call.dt_bias,
                      (const float*)call.state, call.slots, call.request_start, call.history, kc, qc,
                      ks, v, cum, solve, call.sizes, call.requests, call.unit_eps, call.ld);
    };
    if (call.sizes.taps == 4) prepare(channel_prepare_kernel<T, 4>);
    else prepare(channel_prepare_kernel<T, 0>);
    MLXONE_LAUNCH_CHECK("channel delta rule (prepare)");
    const int code = D <= 32 ? launch_scan<T, 4, 8>(call, kc, qc, ks, v, cum, solve, o)
                   : D <= 64 ? launch_scan<T, 4, 16>(call, kc, qc, ks, v, cum, solve, o)
                   : D <= 128 ? launch_scan<T, 4, 32>(call, kc, qc, ks, v, cum, solve, o)
                              : launch_scan<T, 8, 32>(call, kc, qc, ks, v, cum, solve, o);
    if (code) return code;
    const long long items = (long long)call.tokens * H;
    launch_kernel(channel_finish_kernel<T>, dim3(ceil_div_host(items, 8)), dim3(256), 0, call.stream,
                  true, (const float*)o, (const T*)gate, call.norm_weight, (T*)call.mixed, items, V,
                  call.eps);
    MLXONE_LAUNCH_CHECK("channel delta rule (finish)");
    return 0;
}

int check(const DeltaCall& call) {
    const DeltaSizes& sizes = call.sizes;
    MLXONE_REQUIRE(call.tokens > 0 && call.requests > 0 && sizes.heads > 0 && sizes.kv_heads > 0 &&
                       sizes.heads % sizes.kv_heads == 0, "channel delta rule: bad sizes");
    MLXONE_REQUIRE(sizes.key_dim >= 1 && sizes.key_dim <= 256,
                   "channel delta rule: key size %d is not in 1..256", sizes.key_dim);
    MLXONE_REQUIRE(sizes.value_dim >= 1 && sizes.taps >= 1,
                   "channel delta rule: bad value size or taps");
    MLXONE_REQUIRE(call.requests <= 65535 && sizes.heads < 65535,
                   "channel delta rule: too many requests or heads");
    MLXONE_REQUIRE(call.ld >= sizes.channels() + sizes.heads,
                   "channel delta rule: rows %d apart are too short", call.ld);
    return 0;
}

}  // namespace

// The most columns of S that the single-token kernel takes.
MLXONE_API int mlxone_channel_delta_step_columns() { return STEP_MAX_COLUMNS; }

// 32-bit values of scratch that a call with `tokens` tokens needs.
MLXONE_API long long mlxone_channel_delta_scratch(int tokens, int heads, int key_dim, int value_dim) {
    return (long long)tokens * heads * (SOLVE + 4LL * key_dim + 2LL * value_dim);
}

// A step of single tokens (request r brings token r, value_dim up to the limit above).
MLXONE_API int mlxone_channel_delta_step(const void* projected, int ld, const void* decay_up,
                                         int decay_at, int decay_rank, const void* gate_up,
                                         int gate_at, int gate_rank, const float* conv,
                                         const float* a_log, const float* dt_bias,
                                         const float* norm_weight, float eps, float unit_eps,
                                         float* state, const int* slots, const int* history,
                                         void* mixed, int requests, int heads, int kv_heads,
                                         int key_dim, int value_dim, int taps, int write, int dtype,
                                         cudaStream_t stream) {
    if (requests == 0) return 0;
    const DeltaCall call = {projected, ld, conv, a_log, dt_bias, norm_weight, eps, unit_eps, state,
                            slots, nullptr, history, mixed, requests, requests,
                            {heads, kv_heads, key_dim, value_dim, taps}, write, stream};
    if (const int code = check(call)) return code;
    MLXONE_REQUIRE(value_dim <= STEP_MAX_COLUMNS, "channel delta rule: %d columns in one block",
                   value_dim);
    MLXONE_REQUIRE(decay_rank > 0 && gate_rank > 0 && decay_at >= 0 && gate_at >= 0 &&
                       decay_at + decay_rank <= ld && gate_at + gate_rank <= ld,
                   "channel delta rule: inner rows outside the projection");
    return dtype == MLXONE_BF16
        ? launch_step<__nv_bfloat16>(call, decay_up, decay_at, decay_rank, gate_up, gate_at, gate_rank)
        : launch_step<float>(call, decay_up, decay_at, decay_rank, gate_up, gate_at, gate_rank);
}

// A step with portions. steps: float32 [tokens, heads, key_dim], the decay's second product;
// gate: [tokens, heads, value_dim] in the compute type, the gate's.
MLXONE_API int mlxone_channel_delta(const void* projected, int ld, const float* steps,
                                    const void* gate, const float* conv, const float* a_log,
                                    const float* dt_bias, const float* norm_weight, float eps,
                                    float unit_eps, float* state, const int* slots,
                                    const int* request_start, const int* history, float* scratch,
                                    void* mixed, int tokens, int requests, int heads, int kv_heads,
                                    int key_dim, int value_dim, int taps, int write, int dtype,
                                    cudaStream_t stream) {
    if (tokens == 0) return 0;
    const DeltaCall call = {projected, ld, conv, a_log, dt_bias, norm_weight, eps, unit_eps, state,
                            slots, request_start, history, mixed, tokens, requests,
                            {heads, kv_heads, key_dim, value_dim, taps}, write, stream};
    if (const int code = check(call)) return code;
    return dtype == MLXONE_BF16 ? launch_portions<__nv_bfloat16>(call, steps, gate, scratch)
                                : launch_portions<float>(call, steps, gate, scratch);
}
