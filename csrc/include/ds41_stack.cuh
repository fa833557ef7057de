// Shared device helpers of the layer-stack kernels (stack_ops.cu, latent_attn.cu, mlstm.cu).
#pragma once
#include "ds41_api.h"
#include "ds41_launch.cuh"
#include "ds41_ptx.cuh"

namespace ds41 {

// One element of a projection as its consumer finds it: the sum of the split-K planes, or a bf16 value.
__device__ __forceinline__ float proj_at(const ds41_proj& a, long long row, int col) {
  const long long i = row * a.ld + a.col + col;
  if (a.bf16) return __bfloat162float(static_cast<const __nv_bfloat16*>(a.data)[i]);
  const float* p = static_cast<const float*>(a.data) + i;
  float s = p[0];
#pragma unroll 4
  for (int k = 1; k < a.splits; ++k) s += p[k * a.plane];
  return s;
}

template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
// log(sigmoid(x)) without overflow on either side
__device__ __forceinline__ float log_sigmoid_f32(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

// Sum over the block; every thread gets the result.  `red` holds at least 33 floats and may be reused after the call.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < n_warps ? red[lane] : 0.f;
    t = warp_sum(t);
    if (lane == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}

// First row of a run of rows that belong to one request (rows of one request are adjacent and in order).
__device__ __forceinline__ bool segment_start(const int* row_slot, int r) {
  return row_slot[r] >= 0 && (r == 0 || row_slot[r - 1] != row_slot[r]);
}

}  // namespace ds41
