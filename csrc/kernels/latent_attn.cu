// Latent attention: every head's keys and values are linear maps of one cached latent row per token, beside one rotated
// key part that all heads share.  A cache row is [latent (kv_pad) | rotated key part (rot_pad)], zero in the padding.
//
//  latent_post   : RMS norm of the query latent; RMS norm of the key/value latent and rotation of the shared key part into
//                  the request's cache pages
//  latent_query  : per-head queries [dim | rotated part] from a projection, the rotated part turned by the row's position
//  latent_gather : one request's cache rows as two contiguous matrices (prompt passes expand keys and values from them)
//  latent_attend : causal attention over the cache with absorbed queries (q W_uk, so that the latent row itself is key and
//                  value), partial results per key split
//  latent_merge  : sums the splits; the softmax denominator also contains exp(sink) per head
#include "ds41_mma.cuh"
#include "ds41_stack.cuh"

namespace ds41 {

__device__ __forceinline__ void rotate_pair(float u, float v, int pos, float freq, float mag, float& ru, float& rv) {
  float s, c;
  sincosf(static_cast<float>(pos) * freq, &s, &c);
  c *= mag;
  s *= mag;
  ru = u * c - v * s;
  rv = v * c + u * s;
}

// RMS norm of `n` columns of a projection row into `out` (columns up to the next multiple of four are written as zeros).
// The row stays in registers while it is short (kHeld pieces per thread).
template <typename T>
__device__ __forceinline__ void norm_row(const ds41_proj& p, int r, int n, const float* w, float eps, T* out, float* red) {
  constexpr int kHeld = 2;
  float4 held[kHeld], wh[kHeld];
  float q = 0.f;
  int c = 0;
  for (int i = 4 * threadIdx.x; i < n; i += 4 * blockDim.x, ++c) {
    float4 v = proj_at4(p, r, i);
    if (i + 1 >= n) v.y = 0.f;
    if (i + 2 >= n) v.z = 0.f;
    if (i + 3 >= n) v.w = 0.f;
#pragma unroll
    for (int k = 0; k < kHeld; ++k)
      if (c == k) {
        held[k] = v;
        wh[k] = load4(w + i, n - i);
      }
    q += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float s = 1.0f / sqrtf(block_sum(q, red) / n + eps);
  c = 0;
  for (int i = 4 * threadIdx.x; i < n; i += 4 * blockDim.x, ++c) {
    float4 v, g;
    if (c < kHeld) {
#pragma unroll
      for (int k = 0; k < kHeld; ++k)
        if (c == k) {
          v = held[k];
          g = wh[k];
        }
    } else {
      v = proj_at4(p, r, i);
      g = load4(w + i, n - i);
    }
    store4(out + i, make_float4(v.x * s * g.x, i + 1 < n ? v.y * s * g.y : 0.f, i + 2 < n ? v.z * s * g.z : 0.f,
                                i + 3 < n ? v.w * s * g.w : 0.f));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_post_kernel(ds41_latent_post_args p) {
  __shared__ float red[33];
  const int r = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  if (blockIdx.y == 0) {
    norm_row(p.dq, r, p.q_rank, p.dq_norm, p.eps, static_cast<T*>(p.cq) + 1ll * r * p.ld_cq, red);
    return;
  }
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  if (slot < 0) return;
  T* row = cache_row(static_cast<T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, p.row_len, slot, pos);
  if (row == nullptr) return;
  for (int i = threadIdx.x; i < p.rot_dim / 2; i += blockDim.x) {
    float a, b;
    rotate_pair(proj_at(p.kr, r, 2 * i), proj_at(p.kr, r, 2 * i + 1), pos, p.freq[i], p.magnitude, a, b);
    row[p.kv_pad + 2 * i] = from_f32<T>(a);
    row[p.kv_pad + 2 * i + 1] = from_f32<T>(b);
  }
  norm_row(p.kv, r, p.kv_rank, p.kv_norm, p.eps, row, red);
}

// Long passes: one warp per row and part, the row in registers (up to 2048 columns).
constexpr int kWarpPieces = 16;
template <typename T>
__device__ __forceinline__ void norm_row_warp(const ds41_proj& p, int r, int n, const float* w, float eps, T* out) {
  const int lane = threadIdx.x & 31;
  float4 v[kWarpPieces];
  float q = 0.f;
#pragma unroll
  for (int k = 0; k < kWarpPieces; ++k) {
    const int i = 4 * (lane + 32 * k);
    v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < n) {
      v[k] = proj_at4(p, r, i);
      if (i + 1 >= n) v[k].y = 0.f;
      if (i + 2 >= n) v[k].z = 0.f;
      if (i + 3 >= n) v[k].w = 0.f;
      q += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    }
  }
  const float s = 1.0f / sqrtf(warp_sum(q) / n + eps);
#pragma unroll
  for (int k = 0; k < kWarpPieces; ++k) {
    const int i = 4 * (lane + 32 * k);
    if (i >= n) break;
    const float4 g = load4(w + i, n - i);
    store4(out + i, make_float4(v[k].x * s * g.x, v[k].y * s * g.y, v[k].z * s * g.z, v[k].w * s * g.w));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_post_warp_kernel(ds41_latent_post_args p) {
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  if (r >= p.rows) return;
  if (blockIdx.y == 0) {
    norm_row_warp(p.dq, r, p.q_rank, p.dq_norm, p.eps, static_cast<T*>(p.cq) + 1ll * r * p.ld_cq);
    return;
  }
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  if (slot < 0) return;
  T* row = cache_row(static_cast<T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, p.row_len, slot, pos);
  if (row == nullptr) return;
  for (int i = lane; i < p.rot_dim / 2; i += 32) {
    float a, b;
    rotate_pair(proj_at(p.kr, r, 2 * i), proj_at(p.kr, r, 2 * i + 1), pos, p.freq[i], p.magnitude, a, b);
    row[p.kv_pad + 2 * i] = from_f32<T>(a);
    row[p.kv_pad + 2 * i + 1] = from_f32<T>(b);
  }
  norm_row_warp(p.kv, r, p.kv_rank, p.kv_norm, p.eps, row);
}

// In place when q is the projection itself (q.data == out): then only the rotated parts change.  A block's heads share the
// sines and cosines of its row.
constexpr int kMaxTurns = 256;         // pairs whose sine and cosine are kept per block
template <typename T>
__global__ void __launch_bounds__(256) latent_query_kernel(ds41_proj q, const int* row_pos, const float* freq,
                                                           float magnitude, int heads, int dim_pad, int rot_pad,
                                                           int rot_dim, T* out, int ld_out, int in_place) {
  __shared__ float2 turn[kMaxTurns];
  const int r = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  const int pos = row_pos[r];
  for (int i = threadIdx.x; i < rot_dim / 2; i += blockDim.x) {
    float s, c;
    sincosf(static_cast<float>(pos) * freq[i], &s, &c);
    turn[i] = make_float2(c * magnitude, s * magnitude);
  }
  __syncthreads();
  const int hs = dim_pad + rot_pad;
  const int half = in_place ? rot_pad / 2 : hs / 2;
  const int first = in_place ? dim_pad : 0;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < heads * half; i += gridDim.x * blockDim.x) {
    const int h = i / half, j = 2 * (i - h * half) + first, c = h * hs + j;
    const float2 ab = proj_at2(q, r, c);
    float a = ab.x, b = ab.y;
    const int t = j - dim_pad;
    if (t >= 0 && t < rot_dim) {
      const float2 cs = turn[t / 2];
      const float u = a, v = b;
      a = u * cs.x - v * cs.y;
      b = v * cs.x + u * cs.y;
    }
    store2(out + 1ll * r * ld_out + c, a, b);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* pool, const int* page_table, int max_pages,
                                                            int page_tokens, int row_len, int kv_pad, int slot_row,
                                                            const int* row_slot, int n_keys, T* lat, T* rot) {
  const int key = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  if (key >= n_keys) return;
  const int slot = row_slot[slot_row];
  const T* src = slot < 0 ? nullptr
                          : cache_row(const_cast<T*>(pool), page_table, max_pages, page_tokens, row_len, slot, key);
  const int rot_pad = row_len - kv_pad;
  // rows are multiples of 16 elements: whole 16-byte pieces
  constexpr int kPer = 16 / sizeof(T);
  for (int i = lane * kPer; i < row_len; i += 32 * kPer) {
    const uint4 v = src != nullptr ? *reinterpret_cast<const uint4*>(src + i) : make_uint4(0, 0, 0, 0);
    T* dst = i < kv_pad ? lat + 1ll * key * kv_pad + i : rot + 1ll * key * rot_pad + (i - kv_pad);
    *reinterpret_cast<uint4*>(dst) = v;
  }
}

// Plain form for every type and size: one block per (row, head, split), a tile of 32 keys at a time.
template <typename T>
__global__ void __launch_bounds__(128) latent_attend_plain_kernel(ds41_latent_attend_args p) {
  extern __shared__ float att_smem[];
  float* qs = att_smem;                  // [kv_pad + rot_pad] query, scaled
  float* os = qs + p.row_len;            // [kv_pad] running output
  float* sc = os + p.kv_pad;             // [32] scores
  const int h = blockIdx.x, split = blockIdx.y, r = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  const int n_keys = slot < 0 ? 0 : pos + 1;
  int per = (n_keys + p.n_splits - 1) / p.n_splits;
  per = (per + 63) / 64 * 64;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  const long long cell = (1ll * r * p.n_splits + split) * p.heads + h;
  if (k0 >= k1) {
    if (tid == 0) {
      p.part_ml[2 * cell] = -INFINITY;
      p.part_ml[2 * cell + 1] = 0.f;
    }
    return;
  }
  const T* qa = static_cast<const T*>(p.q_abs) + r * p.ld_q_abs + 1ll * h * p.kv_pad;
  const T* qr = static_cast<const T*>(p.q_rot) + r * p.ld_q_rot + 1ll * h * p.q_rot_stride;
  for (int i = tid; i < p.row_len; i += 128) qs[i] = to_f32(i < p.kv_pad ? qa[i] : qr[i - p.kv_pad]);
  for (int i = tid; i < p.kv_pad; i += 128) os[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  __syncthreads();
  for (int t0 = k0; t0 < k1; t0 += 32) {
    for (int j = warp; j < 32; j += 4) {
      const int key = t0 + j;
      float s = -INFINITY;
      if (key < k1) {
        const T* kv = cache_row(static_cast<T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, p.row_len, slot, key);
        float a = 0.f;
        if (kv != nullptr)
          for (int i = lane; i < p.row_len; i += 32) a += qs[i] * to_f32(kv[i]);
        a = warp_sum(a);
        if (kv != nullptr) s = a * p.scale;
      }
      if (lane == 0) sc[j] = s;
    }
    __syncthreads();
    const float mine = sc[lane];
    const float m_new = fmaxf(m, warp_max(mine));
    const float e = m_new == -INFINITY ? 0.f : expf(mine - m_new);
    const float keep = m == -INFINITY ? 0.f : expf(m - m_new);
    l = l * keep + warp_sum(e);
    m = m_new;
    __syncthreads();
    if (warp == 0) sc[lane] = e;
    __syncthreads();
    for (int i = tid; i < p.kv_pad; i += 128) {
      float a = os[i] * keep;
      for (int j = 0; j < 32 && t0 + j < k1; ++j) {
        const T* kv = cache_row(static_cast<T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, p.row_len, slot, t0 + j);
        if (kv != nullptr) a += sc[j] * to_f32(kv[i]);
      }
      os[i] = a;
    }
    __syncthreads();
  }
  for (int i = tid; i < p.kv_pad; i += 128) p.part_o[cell * p.kv_pad + i] = os[i];
  if (tid == 0) {
    p.part_ml[2 * cell] = m;
    p.part_ml[2 * cell + 1] = l;
  }
}

// bf16 form on the warp-level tensor cores: one CTA per (row, MT x 16 heads, split) walks its keys 64 at a time through two
// shared-memory buffers; the key tile is the value tile as well.  Four warps per 16 heads: each scores 16 of the 64 keys,
// then accumulates a quarter of the latent columns (NP pairs of 8 columns).
constexpr int kKeyTile = 64;
constexpr int kProbStride = kKeyTile + 8;

template <int MT, int NP>
__global__ void __launch_bounds__(MT * 128) latent_attend_mma_kernel(ds41_latent_attend_args p) {
  extern __shared__ __align__(16) uint8_t la_smem[];
  const int RL = p.row_len, RS = RL + 8;
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(la_smem);              // [MT * 16][RS]
  __nv_bfloat16* sk = sq + MT * 16 * RS;                                      // [2][64][RS]
  __nv_bfloat16* sp = sk + 2 * kKeyTile * RS;                                 // [MT][16][72]
  float* tops = reinterpret_cast<float*>(sp + MT * 16 * kProbStride);         // [MT][4][16] maxima, then sums
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, mt = warp >> 2, w = warp & 3;
  const int g = lane >> 2, q2 = 2 * (lane & 3);
  const int split = blockIdx.x, r = blockIdx.y, h0 = blockIdx.z * MT * 16;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[r];
  const int n_keys = slot < 0 ? 0 : p.row_pos[r] + 1;
  const int per = ((n_keys + kKeyTile - 1) / kKeyTile + p.n_splits - 1) / p.n_splits * kKeyTile;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  const long long cell0 = (1ll * r * p.n_splits + split) * p.heads;
  if (k0 >= k1) {
    for (int h = tid; h < MT * 16; h += MT * 128)
      if (h0 + h < p.heads) {
        p.part_ml[2 * (cell0 + h0 + h)] = -INFINITY;
        p.part_ml[2 * (cell0 + h0 + h) + 1] = 0.f;
      }
    return;
  }
  const uint4 zero = make_uint4(0, 0, 0, 0);
  // lane i knows where the warp's i-th key of a tile lies; looked up one tile ahead of the copies
  constexpr int kMine = kKeyTile / (MT * 4);
  auto locate = [&](int key0) {
    const int key = key0 + warp + (lane % kMine) * MT * 4;
    return key < k1 ? cache_row(static_cast<__nv_bfloat16*>(p.pool), p.page_table, p.max_pages, p.page_tokens, RL, slot, key)
                    : nullptr;
  };
  auto load = [&](__nv_bfloat16* where, int buf) {
    __nv_bfloat16* dst = sk + buf * kKeyTile * RS + warp * RS;
#pragma unroll 4
    for (int i = 0; i < kMine; ++i) {
      const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(
          __shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(where), i));
      for (int d = lane * 8; d < RL; d += 256) {
        if (src != nullptr) cp_async_16(dst + i * MT * 4 * RS + d, src + d);
        else *reinterpret_cast<uint4*>(dst + i * MT * 4 * RS + d) = zero;
      }
    }
    cp_async_commit();
  };
  __nv_bfloat16* where = locate(k0);
  for (int i = warp; i < MT * 16; i += MT * 4) {
    const int h = h0 + i;
    const __nv_bfloat16* qa = static_cast<const __nv_bfloat16*>(p.q_abs) + r * p.ld_q_abs + 1ll * h * p.kv_pad;
    const __nv_bfloat16* qr = static_cast<const __nv_bfloat16*>(p.q_rot) + r * p.ld_q_rot + 1ll * h * p.q_rot_stride;
    for (int d = lane * 8; d < RL; d += 256) {
      if (h < p.heads) cp_async_16(sq + i * RS + d, d < p.kv_pad ? qa + d : qr + (d - p.kv_pad));
      else *reinterpret_cast<uint4*>(sq + i * RS + d) = zero;
    }
  }
  load(where, 0);
  where = locate(k0 + kKeyTile);
  float acc[NP][2][4];
#pragma unroll
  for (int i = 0; i < NP; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float scale2 = p.scale * 1.4426950408889634f;
  const int n_pairs = p.kv_pad / 16;
  int buf = 0;
  for (int t0 = k0; t0 < k1; t0 += kKeyTile, buf ^= 1) {
    if (t0 + kKeyTile < k1) {
      load(where, buf ^ 1);
      where = locate(t0 + 2 * kKeyTile);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* kt = sk + buf * kKeyTile * RS;
    float s[2][4] = {}, s_odd[2][4] = {};       // two chains: consecutive products into one accumulator wait for each other
    {
      const __nv_bfloat16* arow = sq + (mt * 16 + (lane & 15)) * RS + (lane >> 4) * 8;
      const __nv_bfloat16* brow = kt + (w * 16 + (lane & 7) + (lane >> 4) * 8) * RS + ((lane >> 3) & 1) * 8;
      int k = 0;
#pragma unroll 3
      for (; k + 32 <= RL; k += 32) {
        uint32_t a[4], b[4], c[4], d[4];
        ldmatrix_x4(a[0], a[1], a[2], a[3], arow + k);
        ldmatrix_x4(b[0], b[1], b[2], b[3], brow + k);
        ldmatrix_x4(c[0], c[1], c[2], c[3], arow + k + 16);
        ldmatrix_x4(d[0], d[1], d[2], d[3], brow + k + 16);
        mma_bf16_16816(s[0], a, b[0], b[1]);
        mma_bf16_16816(s[1], a, b[2], b[3]);
        mma_bf16_16816(s_odd[0], c, d[0], d[1]);
        mma_bf16_16816(s_odd[1], c, d[2], d[3]);
      }
      if (k < RL) {
        uint32_t a[4], b[4];
        ldmatrix_x4(a[0], a[1], a[2], a[3], arow + k);
        ldmatrix_x4(b[0], b[1], b[2], b[3], brow + k);
        mma_bf16_16816(s[0], a, b[0], b[1]);
        mma_bf16_16816(s[1], a, b[2], b[3]);
      }
    }
    float top[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = t0 + w * 16 + 8 * j + q2 + (e & 1);
        s[j][e] = key < k1 ? (s[j][e] + s_odd[j][e]) * scale2 : -INFINITY;
        top[e >> 1] = fmaxf(top[e >> 1], s[j][e]);
      }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      top[u] = fmaxf(top[u], __shfl_xor_sync(0xffffffffu, top[u], 1));
      top[u] = fmaxf(top[u], __shfl_xor_sync(0xffffffffu, top[u], 2));
      if ((lane & 3) == 0) tops[(mt * 4 + w) * 16 + g + 8 * u] = top[u];
    }
    __syncthreads();
    float keep[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      float x = m[u];
#pragma unroll
      for (int i = 0; i < 4; ++i) x = fmaxf(x, tops[(mt * 4 + i) * 16 + g + 8 * u]);
      keep[u] = m[u] == -INFINITY ? 0.f : ex2_approx(m[u] - x);
      m[u] = x;
      l[u] *= keep[u];
    }
    // the tile holds at least one visible key, so m is finite here
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const float x = ex2_approx(s[j][2 * u] - m[u]), y = ex2_approx(s[j][2 * u + 1] - m[u]);
        l[u] += x + y;
        *reinterpret_cast<uint32_t*>(sp + (mt * 16 + g + 8 * u) * kProbStride + w * 16 + 8 * j + q2) = pack_bf16(x, y);
      }
#pragma unroll
    for (int i = 0; i < NP; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][j][e] *= keep[e >> 1];
    __syncthreads();
    const __nv_bfloat16* prow = sp + (mt * 16 + (lane & 15)) * kProbStride + (lane >> 4) * 8;
#pragma unroll
    for (int k = 0; k < kKeyTile; k += 16) {
      uint32_t a[4];
      ldmatrix_x4(a[0], a[1], a[2], a[3], prow + k);
      const __nv_bfloat16* brow = kt + (k + (lane & 15)) * RS + (lane >> 4) * 8;
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int pair = w + 4 * i;
        if (pair < n_pairs) {
          uint32_t b[4];
          ldmatrix_x4_trans(b[0], b[1], b[2], b[3], brow + 16 * pair);
          mma_bf16_16816(acc[i][0], a, b[0], b[1]);
          mma_bf16_16816(acc[i][1], a, b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    l[u] += __shfl_xor_sync(0xffffffffu, l[u], 1);
    l[u] += __shfl_xor_sync(0xffffffffu, l[u], 2);
    if ((lane & 3) == 0) tops[(mt * 4 + w) * 16 + g + 8 * u] = l[u];
  }
  __syncthreads();
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int h = h0 + mt * 16 + g + 8 * u;
    if (h >= p.heads) continue;
    const long long cell = cell0 + h;
    if (w == 0 && (lane & 3) == 0) {
      float x = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) x += tops[(mt * 4 + i) * 16 + g + 8 * u];
      p.part_ml[2 * cell] = m[u] * 0.6931471805599453f;       // natural-log units, like the plain kernel
      p.part_ml[2 * cell + 1] = x;
    }
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int pair = w + 4 * i;
      if (pair < n_pairs)
#pragma unroll
        for (int j = 0; j < 2; ++j)
          *reinterpret_cast<float2*>(p.part_o + cell * p.kv_pad + 16 * pair + 8 * j + q2) =
              make_float2(acc[i][j][2 * u], acc[i][j][2 * u + 1]);
    }
  }
}

template <int MT, int NP>
static int launch_attend_mma(const ds41_latent_attend_args& a, cudaStream_t st) {
  const int smem = (MT * 16 + 2 * kKeyTile) * (a.row_len + 8) * 2 + MT * 16 * kProbStride * 2 + MT * 64 * 4;
  static int allowed = 47 * 1024;
  if (smem > allowed) {
    const cudaError_t e = cudaFuncSetAttribute(latent_attend_mma_kernel<MT, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    allowed = smem;
  }
  const dim3 grid(a.n_splits, a.rows, (a.heads + MT * 16 - 1) / (MT * 16));
  return launch_pdl(latent_attend_mma_kernel<MT, NP>, grid, dim3(MT * 128), smem, st, a);
}

template <int MT>
static int dispatch_attend_mma(const ds41_latent_attend_args& a, cudaStream_t st) {
  if (a.kv_pad <= 64) return launch_attend_mma<MT, 1>(a, st);
  if (a.kv_pad <= 128) return launch_attend_mma<MT, 2>(a, st);
  if (a.kv_pad <= 256) return launch_attend_mma<MT, 4>(a, st);
  return launch_attend_mma<MT, 8>(a, st);
}

// heads per CTA of the tensor-core form for this row length (0: it does not fit, the plain form runs)
static int attend_mma_heads(const ds41_latent_attend_args& a) {
  if (a.f32 || a.kv_pad > 512 || (a.kv_pad & 15) || (a.row_len & 15) || (a.ld_q_abs & 7) || (a.ld_q_rot & 7) ||
      (a.q_rot_stride & 7) || ((reinterpret_cast<uintptr_t>(a.q_abs) | reinterpret_cast<uintptr_t>(a.q_rot) |
                                reinterpret_cast<uintptr_t>(a.pool)) & 15))
    return 0;
  auto fits = [&](int mt) {
    return (mt * 16 + 2 * kKeyTile) * (a.row_len + 8) * 2 + mt * 16 * kProbStride * 2 + mt * 256 <= 226 * 1024;
  };
  if (a.heads > 16 && fits(2)) return 32;
  return fits(1) ? 16 : 0;
}

// one block per (head, row): the splits' weights first, then every thread sums four columns over the splits
constexpr int kMaxSplits = 256;
template <typename T>
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* part_o, const float* part_ml, const float* sink,
                                                           int n_splits, int heads, int kv_pad, T* out, int ld_out) {
  __shared__ float wt[kMaxSplits];
  __shared__ float red[33];
  const int h = blockIdx.x, r = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  const long long cell0 = 1ll * r * n_splits * heads + h;
  const float sk = sink != nullptr ? sink[h] : -INFINITY;
  float m = sk;
  for (int s = 0; s < n_splits; ++s) m = fmaxf(m, part_ml[2 * (cell0 + 1ll * s * heads)]);
  float den = 0.f;
  for (int s = threadIdx.x; s < n_splits; s += blockDim.x) {
    const float2 ml = *reinterpret_cast<const float2*>(part_ml + 2 * (cell0 + 1ll * s * heads));
    const float e = ml.y > 0.f ? expf(ml.x - m) : 0.f;
    wt[s] = e;
    den += e * ml.y;
  }
  den = block_sum(den, red) + (sink != nullptr ? expf(sk - m) : 0.f);
  const float inv = den > 0.f ? 1.0f / den : 0.f;
  for (int i = 4 * threadIdx.x; i < kv_pad; i += 4 * blockDim.x) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < n_splits; ++s) {
      const float e = wt[s];
      if (e > 0.f) {
        const float4 o = *reinterpret_cast<const float4*>(part_o + (cell0 + 1ll * s * heads) * kv_pad + i);
        a.x += e * o.x;
        a.y += e * o.y;
        a.z += e * o.z;
        a.w += e * o.w;
      }
    }
    store4(out + 1ll * r * ld_out + h * kv_pad + i, make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv));
  }
}

}  // namespace ds41

using namespace ds41;

extern "C" int ds41_latent_post(const ds41_latent_post_args* a, void* stream) {
  if (a == nullptr || a->rows <= 0 || !proj_ok(a->dq) || a->cq == nullptr || a->dq_norm == nullptr || a->q_rank <= 0 ||
      a->ld_cq < a->q_rank)
    return cudaErrorInvalidValue;
  const bool kv = a->pool != nullptr;       // a layer that reads another layer's rows writes none
  if (!proj_vec4(a->dq) || (a->ld_cq & 3) || a->ld_cq < (a->q_rank + 3) / 4 * 4 ||
      (kv && (!proj_vec4(a->kv) || (a->row_len & 3) || a->kv_pad < (a->kv_rank + 3) / 4 * 4)))
    return cudaErrorInvalidValue;
  if (kv && (!proj_ok(a->kv) || !proj_ok(a->kr) || a->kv_norm == nullptr || a->freq == nullptr || a->kv_rank <= 0 ||
             a->kv_pad < a->kv_rank || a->row_len < a->kv_pad + a->rot_dim || (a->rot_dim & 1) || a->page_tokens <= 0 ||
             a->max_pages <= 0 || a->page_table == nullptr || a->row_pos == nullptr || a->row_slot == nullptr))
    return cudaErrorInvalidValue;
  const dim3 grid(a->rows, kv ? 2 : 1);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->rows >= 256 && a->q_rank <= 128 * kWarpPieces && (!kv || a->kv_rank <= 128 * kWarpPieces)) {
    const dim3 warps((a->rows + 7) / 8, kv ? 2 : 1);
    return a->f32 ? launch_pdl(latent_post_warp_kernel<float>, warps, dim3(256), 0, st, *a)
                  : launch_pdl(latent_post_warp_kernel<__nv_bfloat16>, warps, dim3(256), 0, st, *a);
  }
  return a->f32 ? launch_pdl(latent_post_kernel<float>, grid, dim3(256), 0, st, *a)
                : launch_pdl(latent_post_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, *a);
}

extern "C" int ds41_latent_query(const ds41_proj* q, const int* row_pos, const float* freq, float magnitude, int rows,
                                 int heads, int dim_pad, int rot_pad, int rot_dim, void* out, int ld_out, int f32,
                                 void* stream) {
  if (q == nullptr || !proj_ok(*q) || row_pos == nullptr || freq == nullptr || rows <= 0 || rows > 65535 || heads <= 0 ||
      dim_pad < 0 || (dim_pad & 1) || (rot_pad & 1) || (rot_dim & 1) || rot_dim > rot_pad || rot_dim > 2 * kMaxTurns || out == nullptr ||
      ld_out < heads * (dim_pad + rot_pad))
    return cudaErrorInvalidValue;
  if ((q->ld & 1) || (q->col & 1) || (q->plane & 1) || (ld_out & 1)) return cudaErrorInvalidValue;
  const int in_place = q->data == out ? 1 : 0;
  if (in_place && ((f32 != 0) == (q->bf16 != 0) || q->splits != 1 || q->col != 0 || q->ld != ld_out)) return cudaErrorInvalidValue;
  if (in_place && rot_pad == 0) return cudaSuccess;
  const int half = in_place ? rot_pad / 2 : (dim_pad + rot_pad) / 2;
  int across = (heads * half + 255) / 256;
  if (rows > 64 && across > 4) across = 4;          // long passes: fewer blocks per row, each turns more heads
  const dim3 grid(across, rows);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return launch_pdl(latent_query_kernel<float>, grid, dim3(256), 0, st, *q, row_pos, freq, magnitude, heads, dim_pad,
                      rot_pad, rot_dim, static_cast<float*>(out), ld_out, in_place);
  return launch_pdl(latent_query_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, *q, row_pos, freq, magnitude, heads,
                    dim_pad, rot_pad, rot_dim, static_cast<__nv_bfloat16*>(out), ld_out, in_place);
}

extern "C" int ds41_latent_gather(const void* pool, const int* page_table, int max_pages, int page_tokens, int row_len,
                                  int kv_pad, int slot_row, const int* row_slot, int n_keys, void* lat, void* rot,
                                  int f32, void* stream) {
  if (pool == nullptr || page_table == nullptr || lat == nullptr || row_slot == nullptr || slot_row < 0 || n_keys <= 0 ||
      page_tokens <= 0 || max_pages <= 0 || kv_pad <= 0 || (kv_pad & 15) || (row_len & 15) || row_len < kv_pad ||
      (row_len > kv_pad && rot == nullptr))
    return cudaErrorInvalidValue;
  const dim3 grid((n_keys + 7) / 8);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return launch_pdl(latent_gather_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(pool), page_table,
                      max_pages, page_tokens, row_len, kv_pad, slot_row, row_slot, n_keys, static_cast<float*>(lat),
                      static_cast<float*>(rot));
  return launch_pdl(latent_gather_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(pool),
                    page_table, max_pages, page_tokens, row_len, kv_pad, slot_row, row_slot, n_keys,
                    static_cast<__nv_bfloat16*>(lat), static_cast<__nv_bfloat16*>(rot));
}

extern "C" int ds41_latent_attend(const ds41_latent_attend_args* a, void* stream) {
  if (a == nullptr || a->rows <= 0 || a->rows > 65535 || a->heads <= 0 || a->n_splits <= 0 || a->n_splits > 65535 ||
      a->kv_pad <= 0 || a->row_len < a->kv_pad || a->page_tokens <= 0 || a->max_pages <= 0 || a->q_abs == nullptr ||
      (a->row_len > a->kv_pad && a->q_rot == nullptr) || a->pool == nullptr || a->page_table == nullptr ||
      a->row_pos == nullptr || a->row_slot == nullptr || a->part_o == nullptr || a->part_ml == nullptr)
    return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int mma_heads = attend_mma_heads(*a);
  if (mma_heads == 32) return dispatch_attend_mma<2>(*a, st);
  if (mma_heads == 16) return dispatch_attend_mma<1>(*a, st);
  const size_t smem = (1ull * a->row_len + a->kv_pad + 32) * sizeof(float);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const dim3 grid(a->heads, a->n_splits, a->rows);
  return a->f32 ? launch_pdl(latent_attend_plain_kernel<float>, grid, dim3(128), smem, st, *a)
                : launch_pdl(latent_attend_plain_kernel<__nv_bfloat16>, grid, dim3(128), smem, st, *a);
}

extern "C" int ds41_latent_merge(const float* part_o, const float* part_ml, const float* sink, int n_splits, int rows,
                                 int heads, int kv_pad, void* out, int ld_out, int f32, void* stream) {
  if (part_o == nullptr || part_ml == nullptr || n_splits <= 0 || n_splits > kMaxSplits || (kv_pad & 3) || rows <= 0 || rows > 65535 || heads <= 0 ||
      kv_pad <= 0 || out == nullptr || ld_out < heads * kv_pad)
    return cudaErrorInvalidValue;
  const dim3 grid(heads, rows);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return launch_pdl(latent_merge_kernel<float>, grid, dim3(128), 0, st, part_o, part_ml, sink, n_splits, heads, kv_pad,
                      static_cast<float*>(out), ld_out);
  return launch_pdl(latent_merge_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, part_o, part_ml, sink, n_splits, heads,
                    kv_pad, static_cast<__nv_bfloat16*>(out), ld_out);
}
