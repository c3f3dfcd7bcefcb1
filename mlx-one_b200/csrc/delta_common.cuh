// What the delta rule's kernels share: sizes, a slot's layout, the convolution's inputs, copies
// into shared memory.
#pragma once

#include "common.cuh"

namespace {

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

__device__ __forceinline__ void copy_async_4(float* dst, const float* src) {
    const uint32_t to = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(to), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copy_async_16(float* dst, const float* src) {
    const uint32_t to = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to), "l"(src) : "memory");
}
template <int N>
__device__ __forceinline__ void copy_wait_for() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

struct DeltaSizes {
    int heads, kv_heads, key_dim, value_dim, taps;
    __host__ __device__ int qk() const { return kv_heads * key_dim; }
    __host__ __device__ int inner() const { return heads * value_dim; }
    __host__ __device__ int channels() const { return 2 * qk() + inner(); }
    __host__ __device__ long long matrices() const { return (long long)heads * key_dim * value_dim; }
    __host__ __device__ long long state() const {
        return matrices() + (long long)taps * channels();
    }
};

// The input of channel c at `position` - back, for a token at place `index` of its portion:
// a row of this step, the ring, or zero before the request's start.
template <typename T>
__device__ __forceinline__ float conv_input(const T* projected, int ld, const float* ring,
                                            int channels, int taps, int t, int index, int position,
                                            int back, int c) {
    if (index - back >= 0) return to_float<T>(projected[(size_t)(t - back) * ld + c]);
    if (position - back >= 0) return ring[(size_t)((position - back) % taps) * channels + c];
    return 0.f;
}

}  // namespace
