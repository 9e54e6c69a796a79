// What the kernels of layers with a state per request share: elementwise functions, matrices that may still be the
// slices of a split product, and asynchronous copies into shared memory.
#pragma once

#include "common.cuh"

namespace distie {

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return log1pf(expf(-fabsf(z))) + fmaxf(z, 0.f); }
__device__ __forceinline__ float gate_f(int sigmoid, float z) { return sigmoid ? sigmoid_f(z) : silu_f(z); }

// A float32 matrix that may still be the slices of a split product: `splits` matrices `split_stride` floats apart
// whose sum it is (splits == 1: the matrix itself).  Loads add the slices up, in their order.
struct Sliced {
  const float* p;
  int stride;  // of a row
  int splits;
  long long split_stride;
  const float* bias = nullptr;  // per column, added to the sum of the slices (a projection's bias); null: none
  __device__ __forceinline__ float at(size_t row, int col) const {
    const float* q = p + row * stride + col;
    float v = q[0];
    for (int s = 1; s < splits; ++s) v += q[(size_t)s * split_stride];
    return bias ? v + bias[col] : v;
  }
  __device__ __forceinline__ float4 at4(size_t row, int col) const {
    const float* q = p + row * stride + col;
    float4 v = *reinterpret_cast<const float4*>(q);
    for (int s = 1; s < splits; ++s) {
      const float4 w = *reinterpret_cast<const float4*>(q + (size_t)s * split_stride);
      v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
    }
    if (bias) {
      const float4 b = *reinterpret_cast<const float4*>(bias + col);
      v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
    }
    return v;
  }
};

__device__ __forceinline__ void cp_async_f4(float* dst, const float* src, bool live) {
  const int bytes = live ? 16 : 0;  // zero-fills when not live
  asm volatile("cp.async.ca.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_f1(float* dst, const float* src, bool live) {
  const int bytes = live ? 4 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace distie
