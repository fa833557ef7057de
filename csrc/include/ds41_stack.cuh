// Shared device helpers of the layer-stack kernels (stack_ops.cu, latent_attn.cu, group_attn.cu, mlstm.cu).
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

// Four neighbouring elements at a column that is a multiple of 4 (rows and planes 16-byte aligned).
__device__ __forceinline__ float4 proj_at4(const ds41_proj& a, long long row, int col) {
  const long long i = row * a.ld + a.col + col;
  if (a.bf16) {
    const uint2 v = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(a.data) + i);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                       __uint_as_float(v.y & 0xffff0000u));
  }
  const float* p = static_cast<const float*>(a.data) + i;
  float4 s = *reinterpret_cast<const float4*>(p);
#pragma unroll 4
  for (int k = 1; k < a.splits; ++k) {
    const float4 t = *reinterpret_cast<const float4*>(p + k * a.plane);
    s.x += t.x;
    s.y += t.y;
    s.z += t.z;
    s.w += t.w;
  }
  return s;
}
// Two neighbouring elements at an even column (even row lengths and planes).
__device__ __forceinline__ float2 proj_at2(const ds41_proj& a, long long row, int col) {
  const long long i = row * a.ld + a.col + col;
  if (a.bf16) {
    const uint32_t v = *reinterpret_cast<const uint32_t*>(static_cast<const __nv_bfloat16*>(a.data) + i);
    return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
  }
  const float* p = static_cast<const float*>(a.data) + i;
  float2 s = *reinterpret_cast<const float2*>(p);
#pragma unroll 4
  for (int k = 1; k < a.splits; ++k) {
    const float2 t = *reinterpret_cast<const float2*>(p + k * a.plane);
    s.x += t.x;
    s.y += t.y;
  }
  return s;
}
__device__ __forceinline__ void store2(float* p, float x, float y) { *reinterpret_cast<float2*>(p) = make_float2(x, y); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float x, float y) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(x, y);
}
inline bool proj_ok(const ds41_proj& p) {
  return p.data != nullptr && p.ld > 0 && p.splits >= 1 && p.col >= 0 && (p.splits == 1 || (p.plane > 0 && !p.bf16));
}
inline bool proj_vec4(const ds41_proj& p) {
  return !(p.ld & 3) && !(p.col & 3) && !(p.plane & 3) && !(reinterpret_cast<uintptr_t>(p.data) & 15);
}

// Four values of a vector of which `valid` exist (the rest read as zero).
__device__ __forceinline__ float4 load4(const float* p, int valid) {
  if (valid >= 4) return *reinterpret_cast<const float4*>(p);
  return make_float4(valid > 0 ? p[0] : 0.f, valid > 1 ? p[1] : 0.f, valid > 2 ? p[2] : 0.f, 0.f);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
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

// Cache row of position `pos` of a request, or null when its page is not leased.
template <typename T>
__device__ __forceinline__ T* cache_row(T* pool, const int* page_table, int max_pages, int page_tokens, int row_len,
                                        int slot, int pos) {
  const int pg = pos / page_tokens;
  if (pg < 0 || pg >= max_pages) return nullptr;
  const int id = page_table[1ll * slot * max_pages + pg];
  if (id < 0) return nullptr;
  return pool + (1ll * id * page_tokens + (pos - pg * page_tokens)) * row_len;
}

// First row of a run of rows that belong to one request (rows of one request are adjacent and in order).
__device__ __forceinline__ bool segment_start(const int* row_slot, int r) {
  return row_slot[r] >= 0 && (r == 0 || row_slot[r - 1] != row_slot[r]);
}

}  // namespace ds41
