// Attention of a long prompt pass of one request on tcgen05: adjacent rows against keys that TMA can fetch.
//
// One CTA owns two tiles of 128 query rows that read the same keys and walks the keys 128 at a time; both tiles share every
// key / value tile.
//   warps 0-3, 4-7 : softmax of tile 0 / 1 (one thread per query row), output epilogue
//   warp 8         : TMA producer (Q once, then K and V tiles into stage rings)
//   warp 9         : tcgen05.mma issue: S = Q K^T into TMEM, O += P V with P read from TMEM where it replaces its S
// While one tile's warps work on its softmax the tensor core runs the other tile's products.  The running maximum is only
// raised when it grew by more than 2^8, so the accumulated output is rarely rescaled.
//
// `Form` says what the tiles are and where operands come from:
//   PromptTiles tiles(p, block)                 the CTA's two tiles, the key tiles they see and the first key
//   load_q / load_k / load_v                    TMA loads of one tile of 128 rows in 64-column chunks (kPreChunk bytes each)
//   first_key(pos)                              first position that `pos` sees (kLowerBound: it is not always 0)
//   sink(h)                                     extra logit in the denominator, -inf for none (in units of log2)
//   gate(row, h, c, f)                          factors on 16 output columns
#pragma once
#include <cuda.h>

#include "ds41_stack.cuh"
#include "ds41_tma.h"

namespace ds41 {

constexpr int kPreThreads = 320;
constexpr int kPreTile = 128;                  // query rows per tile, keys per tile
constexpr int kPreChunk = kPreTile * 128;      // bytes of 128 rows x 64 bf16 columns

struct PromptParams {
  int rows, heads, dp, rp, vp, n_keys, pos0;
  int kd, kr, vc;            // 64-column chunks of the unrotated part, the rotated part and the value
  int k_stages, v_stages;
  float scale_log2;          // scale * log2(e)
  __nv_bfloat16* out;
  int ld_out;
  int* status;
};

struct PromptTiles {
  int head[2], row0[2];
  int n[2];                  // key tiles that the rows see (0: no such tile)
  int key0;                  // first key of key tile 0
};

__device__ __forceinline__ void drain_barrier(uint64_t* bar, uint32_t parity) {
  for (int i = 0; i < (1 << 20) && !mbar_test_wait(bar, parity); ++i) {
  }
}

template <typename Form>
__global__ void __launch_bounds__(kPreThreads, 1)
prompt_attend_kernel(const __grid_constant__ Form form, const PromptParams p) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = smem_u32(smem_raw);
  uint8_t* smem = smem_raw + ((1024u - (raw & 1023u)) & 1023u);
  const int qk_chunks = p.kd + p.kr;
  const int q_bytes = qk_chunks * kPreChunk, k_bytes = q_bytes, v_bytes = p.vc * kPreChunk;
  uint8_t* s_q = smem;                                   // two tiles
  uint8_t* s_k = s_q + 2 * q_bytes;
  uint8_t* s_v = s_k + p.k_stages * k_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_v + p.v_stages * v_bytes);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;        // [2]
  uint64_t* k_empty = bars + 3;
  uint64_t* v_full = bars + 5;
  uint64_t* v_empty = bars + 7;
  uint64_t* s_full = bars + 9;        // [2] per tile: S complete (and every earlier MMA of the issuing thread)
  uint64_t* p_full = bars + 11;       // [2] per tile: P written, O rescaled
  uint64_t* o_full = bars + 13;       // [2] per tile
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  const PromptTiles tile = form.tiles(p, blockIdx.x);
  const int n = max(tile.n[0], tile.n[1]);

  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], kPreTile);
      mbar_init(&o_full[i], 1);
    }
    mbar_init_fence();
  }
  if (warp == 9) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  pdl_wait();

  if (warp == 8) {
    if (lane == 0) {
      form.prefetch();
      const int tiles = tile.n[1] > 0 ? 2 : 1;
      mbar_expect_tx(q_full, tiles * q_bytes);
      for (int t = 0; t < tiles; ++t) form.load_q(p, s_q + t * q_bytes, q_full, tile.head[t], tile.row0[t]);
      bool ok = true;
      int j = 0;
      for (; j < n && ok; ++j) {
        const int ks = j % p.k_stages, vs = j % p.v_stages;
        ok = mbar_wait(&k_empty[ks], ((j / p.k_stages) & 1) ^ 1, p.status, 400);
        if (!ok) break;
        mbar_expect_tx(&k_full[ks], k_bytes);
        form.load_k(p, s_k + ks * k_bytes, &k_full[ks], tile.head[0], tile.key0 + j * kPreTile);
        ok = mbar_wait(&v_empty[vs], ((j / p.v_stages) & 1) ^ 1, p.status, 401);
        if (!ok) {
          drain_barrier(&k_full[ks], (j / p.k_stages) & 1);
          break;
        }
        mbar_expect_tx(&v_full[vs], v_bytes);
        form.load_v(p, s_v + vs * v_bytes, &v_full[vs], tile.head[0], tile.key0 + j * kPreTile);
      }
      if (!ok) {
        // something else gave up: let the copies of the last tiles land before the shared memory goes away
        drain_barrier(q_full, 0);
        for (int b = max(0, j - 2); b < j; ++b) {
          drain_barrier(&k_full[b % p.k_stages], (b / p.k_stages) & 1);
          drain_barrier(&v_full[b % p.v_stages], (b / p.v_stages) & 1);
        }
      }
    }
  } else if (warp == 9) {
    const bool leader = elect_one();
    const uint32_t idesc_s = umma_idesc(kPreTile, kPreTile, 1u, 1u);
    const uint32_t idesc_pv = umma_idesc_bmn(kPreTile, p.vp, 1u, 1u);
    const uint64_t q_desc = umma_desc_sw128(smem_u32(s_q)), k_desc = umma_desc_sw128(smem_u32(s_k));
    const uint64_t v_desc = umma_desc_sw128_mn(smem_u32(s_v), kPreChunk, 1024);
    const int kd16 = p.dp / 16, kr16 = p.rp / 16;
    auto wait = [&](uint64_t* bar, uint32_t parity, int where) {
      const bool ok = mbar_wait(bar, parity, p.status, where);
      return __all_sync(0xffffffffu, ok) != 0;
    };
    auto issue_s = [&](int t, int stage) {
      const uint64_t qd = q_desc + static_cast<uint64_t>(t * q_bytes / 16);
      const uint64_t kd = k_desc + static_cast<uint64_t>(stage * k_bytes / 16);
      for (int k = 0; k < kd16; ++k) {
        const uint64_t off = static_cast<uint64_t>((k >> 2) * (kPreChunk / 16) + (k & 3) * 2);
        umma_bf16_if(leader, tmem + t * 128, qd + off, kd + off, idesc_s, k > 0 ? 1u : 0u);
      }
      for (int k = 0; k < kr16; ++k) {
        const uint64_t off = static_cast<uint64_t>((p.kd + (k >> 2)) * (kPreChunk / 16) + (k & 3) * 2);
        umma_bf16_if(leader, tmem + t * 128, qd + off, kd + off, idesc_s, kd16 + k > 0 ? 1u : 0u);
      }
      tc_commit_if(leader, &s_full[t]);
    };
    auto issue_pv = [&](int t, int stage, bool first) {
      const uint64_t vd = v_desc + static_cast<uint64_t>(stage * v_bytes / 16);
#pragma unroll
      for (int k = 0; k < kPreTile / 16; ++k)
        umma_bf16_ts_if(leader, tmem + 256 + t * 128, tmem + t * 128 + 8 * k, vd + 128 * k, idesc_pv, first && k == 0 ? 0u : 1u);
    };
    bool ok = wait(q_full, 0, 410) && wait(&k_full[0], 0, 411);
    if (ok) {
      tc_fence_after();
      issue_s(0, 0);
      if (tile.n[1] > 0) issue_s(1, 0);
      tc_commit_if(leader, &k_empty[0]);
    }
    for (int j = 0; j < n && ok; ++j) {
      const int vs = j % p.v_stages, ks = (j + 1) % p.k_stages;
      ok = wait(&v_full[vs], (j / p.v_stages) & 1, 412);
      if (ok && j + 1 < n) ok = wait(&k_full[ks], ((j + 1) / p.k_stages) & 1, 413);
      if (!ok) break;
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        if (j < tile.n[t]) {
          if (ok) ok = wait(&p_full[t], j & 1, 414 + t);
          if (!ok) break;
          tc_fence_after();
          issue_pv(t, vs, j == 0);
          if (j == tile.n[t] - 1) tc_commit_if(leader, &o_full[t]);
        }
        if (t == 1) tc_commit_if(leader, &v_empty[vs]);
        if (j + 1 < tile.n[t]) issue_s(t, ks);
      }
      if (ok && j + 1 < n) tc_commit_if(leader, &k_empty[ks]);
    }
  } else {
    const int t = warp >> 2, quad = warp & 3;
    const int h = tile.head[t], row = tile.row0[t] + quad * 32 + lane;
    const int pos = p.pos0 + row, warp_pos = p.pos0 + tile.row0[t] + quad * 32;
    const int low = Form::kLowerBound ? form.first_key(pos) : 0;
    const int warp_low = Form::kLowerBound ? form.first_key(warp_pos + 31) : 0;
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t s_t = tmem + lanes + t * 128, o_t = tmem + lanes + 256 + t * 128;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < tile.n[t] && ok; ++j) {
      ok = __all_sync(0xffffffffu, mbar_wait(&s_full[t], j & 1, p.status, 420 + t)) != 0;
      if (!ok) break;
      tc_fence_after();
      const int key0 = tile.key0 + j * kPreTile;
      const bool edge = key0 + kPreTile - 1 > warp_pos || (Form::kLowerBound && key0 < warp_low);
      const int seen = pos - key0;                       // columns [hidden, seen] of this tile are visible
      const int hidden = Form::kLowerBound ? low - key0 : 0;
      float top = -INFINITY;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(s_t + 32 * c, v);
        tmem_wait_ld();
        if (edge) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (32 * c + i <= seen && (!Form::kLowerBound || 32 * c + i >= hidden))
              top = fmaxf(top, __uint_as_float(v[i]) * p.scale_log2);
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) top = fmaxf(top, __uint_as_float(v[i]) * p.scale_log2);
        }
      }
      const bool grow = top > m + 8.f || (m == -INFINITY && top > m);
      if (__any_sync(0xffffffffu, grow)) {
        const float m_new = grow ? top : m;
        const float alpha = m == -INFINITY ? 0.f : ex2_approx(m - m_new);
        l *= alpha;
        m = m_new;
        if (j > 0) {
          const float keep = grow ? alpha : 1.f;
          for (int c = 0; c < p.vp; c += 16) {
            uint32_t o[16];
            tmem_ld_32x16(o_t + c, o);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * keep);
            tmem_st_32x16(o_t + c, o);
          }
        }
      }
      const float neg = m == -INFINITY ? 0.f : -m;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t v[32], w[16];
        tmem_ld_32x32(s_t + 32 * c, v);
        tmem_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float a = ex2_approx(fmaf(__uint_as_float(v[2 * i]), p.scale_log2, neg));
          float b = ex2_approx(fmaf(__uint_as_float(v[2 * i + 1]), p.scale_log2, neg));
          if (edge) {
            const int x = 32 * c + 2 * i;
            a = x <= seen && (!Form::kLowerBound || x >= hidden) ? a : 0.f;
            b = x + 1 <= seen && (!Form::kLowerBound || x + 1 >= hidden) ? b : 0.f;
          }
          l += a + b;
          const __nv_bfloat162 q = __floats2bfloat162_rn(a, b);
          w[i] = *reinterpret_cast<const uint32_t*>(&q);
        }
        tmem_st_32x16(s_t + 16 * c, w);                  // columns whose S this thread has read
      }
      tmem_wait_st();
      tc_fence_before();
      mbar_arrive(&p_full[t]);
    }
    if (ok && tile.n[t] > 0) ok = __all_sync(0xffffffffu, mbar_wait(&o_full[t], 0, p.status, 430 + t)) != 0;
    if (ok && tile.n[t] > 0) {
      tc_fence_after();
      const float sink2 = form.sink(h);
      const float m_fin = fmaxf(m, sink2);
      const float w_o = m == -INFINITY ? 0.f : ex2_approx(m - m_fin);
      const float den = l * w_o + (sink2 == -INFINITY ? 0.f : ex2_approx(sink2 - m_fin));
      const float f = den > 0.f ? w_o / den : 0.f;
      for (int c = 0; c < p.vp; c += 16) {
        uint32_t o[16];
        tmem_ld_32x16(o_t + c, o);
        tmem_wait_ld();
        if (row < p.rows) {
          float g[16];
          form.gate(p, row, h, c, g);
          uint32_t w[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const float a = __uint_as_float(o[2 * i]) * f * g[2 * i], b = __uint_as_float(o[2 * i + 1]) * f * g[2 * i + 1];
            const __nv_bfloat162 q = __floats2bfloat162_rn(a, b);
            w[i] = *reinterpret_cast<const uint32_t*>(&q);
          }
          uint4* dst = reinterpret_cast<uint4*>(p.out + 1ll * row * p.ld_out + h * p.vp + c);
          dst[0] = make_uint4(w[0], w[1], w[2], w[3]);
          dst[1] = make_uint4(w[4], w[5], w[6], w[7]);
        }
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// Stage counts and shared memory of a launch; returns the bytes, 0 when the sizes do not fit.
inline int prompt_smem(PromptParams& p) {
  p.kd = (p.dp + 63) / 64;
  p.kr = (p.rp + 63) / 64;
  p.vc = (p.vp + 63) / 64;
  const int qk = (p.kd + p.kr) * kPreChunk, v = p.vc * kPreChunk;
  constexpr int kLimit = 226 * 1024 - 1024 - 256;
  p.k_stages = p.v_stages = 1;
  if (p.vp > 128 || 2 * qk + qk + v > kLimit) return 0;
  if (2 * qk + 2 * qk + v <= kLimit) p.k_stages = 2;
  if (2 * qk + p.k_stages * qk + 2 * v <= kLimit) p.v_stages = 2;
  return 2 * qk + p.k_stages * qk + p.v_stages * v + 1024 + 256;
}

template <typename Form>
inline cudaError_t launch_prompt_attend(const Form& form, const PromptParams& p, int blocks, int smem, cudaStream_t stream) {
  static bool ready = false;
  if (!ready) {
    const cudaError_t e = cudaFuncSetAttribute(prompt_attend_kernel<Form>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
    if (e != cudaSuccess) return e;
    ready = true;
  }
  return launch_pdl(prompt_attend_kernel<Form>, dim3(blocks), dim3(kPreThreads), smem, stream, form, p);
}

}  // namespace ds41
