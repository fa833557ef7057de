// Grouped-query attention with a paged cache: query head h reads key / value head h / (heads / kv_heads).  A cache row is
// [keys of all key/value heads | values of all key/value heads], every head padded with zeros to a multiple of 16.
//
//  attn_post    : after the projection: causal convolution over time on every channel of q, k and v; RMS norm over all heads
//                 of q and of k at once; rotation of the leading dimensions of a head; q leaves as a matrix, k and v go into
//                 the request's cache pages
//  group_attend : attention of any mix of rows over the cache, each over its own chunk of the sequence (or everything before
//                 it); the head's output is multiplied by the sigmoid of its gate.  bf16 runs on warp-level tensor cores, a
//                 cluster of up to eight CTAs per row and key/value head; 32-bit (and odd sizes) in a plain form
//
// The convolution's last taps - 1 inputs per request live in a ring indexed by position (p % (taps - 1)), so nothing is
// shifted and running a position twice changes nothing.  attn_post reads the ring, the attention kernel that follows writes
// it: rows of one pass never see their successors.
#include <cooperative_groups.h>

#include "ds41_group.cuh"
#include "ds41_mma.cuh"

namespace ds41 {

namespace cg = cooperative_groups;

constexpr int kPostTurns = 512;          // rotated pairs whose sine and cosine are kept per block

// one block per row; the convolved row stays in shared memory between the norm and the rotation
template <typename T>
__global__ void __launch_bounds__(512) attn_post_kernel(ds41_attn_post_args p) {
  extern __shared__ __align__(16) float ap_row[];
  __shared__ float red[2][33];
  __shared__ float2 turn[kPostTurns];
  const int r = blockIdx.x, tid = threadIdx.x;
  const int nq = p.heads * p.dim_pad, nk = p.kv_heads * p.dim_pad, nv = p.kv_heads * p.vdim_pad, C = nq + nk + nv;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  if (slot < 0) return;
  const int half = p.rot_dim / 2, back = p.taps - 1;
  for (int i = tid; i < half; i += blockDim.x) {
    float s, c;
    sincosf(static_cast<float>(pos) * p.freq[i], &s, &c);
    turn[i] = make_float2(c, s);
  }
  // how many of the predecessors are rows of this pass (rows of a request are adjacent and in order)
  int near = 0;
  while (near < back && r - near - 1 >= 0 && p.row_slot[r - near - 1] == slot) ++near;
  const float* ring = p.state + 1ll * slot * back * C;
  float sq = 0.f, sk = 0.f;
  for (int c = 4 * tid; c < C; c += 4 * blockDim.x) {
    float4 a = proj_at4(p.u, r, c);
    if (p.conv != nullptr) {
      const float4 w0 = *reinterpret_cast<const float4*>(p.conv + 1ll * back * C + c);
      a.x *= w0.x;
      a.y *= w0.y;
      a.z *= w0.z;
      a.w *= w0.w;
      for (int d = 1; d <= back && d <= pos; ++d) {
        const float4 u = d <= near ? proj_at4(p.u, r - d, c)
                                   : *reinterpret_cast<const float4*>(ring + 1ll * ((pos - d) % back) * C + c);
        const float4 w = *reinterpret_cast<const float4*>(p.conv + 1ll * (back - d) * C + c);
        a.x += w.x * u.x;
        a.y += w.y * u.y;
        a.z += w.z * u.z;
        a.w += w.w * u.w;
      }
    }
    if (c < nq + nk && p.q_norm != nullptr) {
      const float s = a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
      (c < nq ? sq : sk) += s;
      const float4 w = *reinterpret_cast<const float4*>(c < nq ? p.q_norm + c : p.k_norm + (c - nq));
      a.x *= w.x;
      a.y *= w.y;
      a.z *= w.z;
      a.w *= w.w;
    }
    *reinterpret_cast<float4*>(ap_row + c) = a;
  }
  float fq = 1.f, fk = 1.f;
  if (p.q_norm != nullptr) {
    sq = block_sum(sq, red[0]);
    sk = block_sum(sk, red[1]);
    fq = 1.0f / sqrtf(sq / (p.heads * p.dim) + p.eps);
    fk = 1.0f / sqrtf(sk / (p.kv_heads * p.dim) + p.eps);
  }
  __syncthreads();
  T* q = static_cast<T*>(p.q) + r * p.ld_q;
  T* row = cache_row(static_cast<T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, nk + nv, slot, pos);
  for (int c = 4 * tid; c < C; c += 4 * blockDim.x) {
    const float4 a = *reinterpret_cast<const float4*>(ap_row + c);
    float o[4] = {a.x, a.y, a.z, a.w};
    if (c < nq + nk) {
      const int j0 = c % p.dim_pad;
      if (j0 < p.rot_dim) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = j0 + e;
          if (j < half) o[e] = o[e] * turn[j].x - ap_row[c + e + half] * turn[j].y;
          else if (j < p.rot_dim) o[e] = o[e] * turn[j - half].x + ap_row[c + e - half] * turn[j - half].y;
        }
      }
      const float f = c < nq ? fq : fk;
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] *= f;
    }
    const float4 v = make_float4(o[0], o[1], o[2], o[3]);
    if (c < nq) store4(q + c, v);
    else if (row != nullptr) store4(row + (c - nq), v);
  }
}

// Plain form for every type and size: one block per (head, row), a tile of 32 keys at a time.
template <typename T>
__global__ void __launch_bounds__(128) group_attend_plain_kernel(ds41_group_attend_args p) {
  extern __shared__ __align__(16) float ga_smem[];
  float* qs = ga_smem;                   // [dim_pad]
  float* os = qs + p.dim_pad;            // [vdim_pad] running output
  float* sc = os + p.vdim_pad;           // [32] scores
  const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  T* out = static_cast<T*>(p.out) + 1ll * r * p.ld_out + h * p.vdim_pad;
  if (slot < 0) {
    for (int i = tid; i < p.vdim_pad; i += 128) out[i] = from_f32<T>(0.f);
    return;
  }
  keep_inputs(p, r, slot, pos, h, gridDim.x);
  const int g = h / (p.heads / p.kv_heads), row_len = p.kv_heads * (p.dim_pad + p.vdim_pad);
  const int k_at = g * p.dim_pad, v_at = p.kv_heads * p.dim_pad + g * p.vdim_pad;
  const T* q = static_cast<const T*>(p.q) + r * p.ld_q + h * p.dim_pad;
  for (int i = tid; i < p.dim_pad; i += 128) qs[i] = to_f32(q[i]);
  for (int i = tid; i < p.vdim_pad; i += 128) os[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  __syncthreads();
  auto at = [&](int key) {
    return cache_row(static_cast<const T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, row_len, slot, key);
  };
  for (int t0 = chunk_start(pos, p.chunk); t0 <= pos; t0 += 32) {
    for (int j = warp; j < 32; j += 4) {
      const T* kv = t0 + j <= pos ? at(t0 + j) : nullptr;
      float a = 0.f;
      if (kv != nullptr)
        for (int i = lane; i < p.dim_pad; i += 32) a += qs[i] * to_f32(kv[k_at + i]);
      a = warp_sum(a);
      if (lane == 0) sc[j] = kv != nullptr ? a * p.scale : -INFINITY;
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
    for (int i = tid; i < p.vdim_pad; i += 128) {
      float a = os[i] * keep;
      for (int j = 0; j < 32 && t0 + j <= pos; ++j) {
        const T* kv = at(t0 + j);
        if (kv != nullptr) a += sc[j] * to_f32(kv[v_at + i]);
      }
      os[i] = a;
    }
    __syncthreads();
  }
  const float f = (l > 0.f ? 1.0f / l : 0.f) * (p.gate.data != nullptr ? sigmoid_f32(proj_at(p.gate, r, h)) : 1.f);
  for (int i = tid; i < p.vdim_pad; i += 128) out[i] = from_f32<T>(os[i] * f);
}

// bf16 form: CTA (split, key/value head and 16 of its query heads, row).  Every warp walks its own steps of 16 keys through
// its own ring of shared-memory stages - no block-wide wait until the partial results are merged: over the warps in shared
// memory, over the CTAs of the cluster through distributed shared memory.  NP: 16-column pieces of the value width.
constexpr int kStepKeys = 16;
constexpr int kAttendStages = 3;
constexpr int kAttendWarps = 4;

__host__ __device__ inline int attend_smem(int dp, int vp) {
  return (16 * (dp + 8) + kAttendWarps * kAttendStages * kStepKeys * (dp + vp + 16)) * 2 + kAttendWarps * 32 * 4 + 32 * 4;
}

template <int NP>
__global__ void __launch_bounds__(kAttendWarps * 32) group_attend_mma_kernel(ds41_group_attend_args p) {
  extern __shared__ __align__(16) uint8_t gm_smem[];
  const int dp = p.dim_pad, vp = p.vdim_pad, KS = dp + 8, VS = vp + 8;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, q2 = 2 * (lane & 3);
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(gm_smem);               // [16][KS]
  __nv_bfloat16* stages = sq + 16 * KS;                                        // [warp][stage][16 KS | 16 VS]
  const int stage_len = kStepKeys * (KS + VS);
  __nv_bfloat16* mine = stages + warp * kAttendStages * stage_len;
  float* ml = reinterpret_cast<float*>(stages + kAttendWarps * kAttendStages * stage_len);   // [warp][16]{max, sum}
  float* cml = ml + kAttendWarps * 32;                                         // [16]{max, sum} of the CTA
  const int n = p.heads / p.kv_heads, m_tiles = (n + 15) / 16;
  const int split = blockIdx.x, g = blockIdx.y / m_tiles, h0 = g * n + (blockIdx.y % m_tiles) * 16, r = blockIdx.z;
  const int h_end = (g + 1) * n;                                               // heads [h0, min(h0 + 16, h_end))
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + 1ll * r * p.ld_out;
  if (slot < 0) {                        // the same in every CTA of the cluster
    if (split == 0)
      for (int i = tid; i < 16 * vp; i += blockDim.x)
        if (h0 + i / vp < h_end) out[(h0 + i / vp) * vp + i % vp] = __float2bfloat16_rn(0.f);
    return;
  }
  const int first = chunk_start(pos, p.chunk), steps = (pos - first) / kStepKeys + 1;
  const int per = (steps + p.n_splits - 1) / p.n_splits, s0 = split * per, s1 = min(steps, s0 + per);
  const int row_len = p.kv_heads * (dp + vp), k_at = g * dp, v_at = p.kv_heads * dp + g * vp;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  for (int i = warp; i < 16; i += kAttendWarps) {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q) + r * p.ld_q + (h0 + i) * dp;
    for (int d = lane * 8; d < dp; d += 256) {
      if (h0 + i < h_end) cp_async_16(sq + i * KS + d, q + d);
      else *reinterpret_cast<uint4*>(sq + i * KS + d) = zero;
    }
  }
  cp_async_commit();
  // lane i < 16 knows where key i of a step lies; looked up one step ahead of the copies
  auto locate = [&](int s) -> const __nv_bfloat16* {
    const int key = first + s * kStepKeys + (lane & 15);
    return s < s1 && key <= pos ? cache_row(static_cast<const __nv_bfloat16*>(p.pool), p.page_table, p.max_pages,
                                            p.page_tokens, row_len, slot, key)
                                : nullptr;
  };
  auto load = [&](const __nv_bfloat16* where, int s, int stage) {
    if (s < s1) {
      __nv_bfloat16* k = mine + stage * stage_len;
      __nv_bfloat16* v = k + kStepKeys * KS;
#pragma unroll 4
      for (int i = 0; i < kStepKeys; ++i) {
        const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(
            __shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(where), i));
        for (int d = lane * 8; d < dp + vp; d += 256) {
          __nv_bfloat16* dst = d < dp ? k + i * KS + d : v + i * VS + (d - dp);
          if (src != nullptr) cp_async_16(dst, d < dp ? src + k_at + d : src + v_at + (d - dp));
          else *reinterpret_cast<uint4*>(dst) = zero;
        }
      }
    }
    cp_async_commit();                   // one group per step, empty ones included: the waits count groups
  };
  int s_load = s0 + warp;
  const __nv_bfloat16* where = locate(s_load);
#pragma unroll
  for (int i = 0; i < kAttendStages - 1; ++i) {
    load(where, s_load, i);
    s_load += kAttendWarps;
    where = locate(s_load);
  }
  keep_inputs(p, r, slot, pos, split + p.n_splits * blockIdx.y, p.n_splits * gridDim.y);
  cp_async_wait<kAttendStages - 1>();
  __syncthreads();                       // the queries have landed
  float acc[NP][2][4];
#pragma unroll
  for (int i = 0; i < NP; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float scale2 = p.scale * 1.4426950408889634f;
  const __nv_bfloat16* arow = sq + (lane & 15) * KS + (lane >> 4) * 8;
  int stage = 0, fill = kAttendStages - 1;
  for (int s = s0 + warp; s < s1; s += kAttendWarps) {
    load(where, s_load, fill);
    s_load += kAttendWarps;
    where = locate(s_load);
    fill = fill + 1 == kAttendStages ? 0 : fill + 1;
    cp_async_wait<kAttendStages - 1>();
    __syncwarp();
    const __nv_bfloat16* kt = mine + stage * stage_len;
    const __nv_bfloat16* vt = kt + kStepKeys * KS;
    stage = stage + 1 == kAttendStages ? 0 : stage + 1;
    float sc[2][4] = {};
    const __nv_bfloat16* brow = kt + ((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8;
#pragma unroll 4
    for (int k = 0; k < dp; k += 16) {
      uint32_t a[4], b[4];
      ldmatrix_x4(a[0], a[1], a[2], a[3], arow + k);
      ldmatrix_x4(b[0], b[1], b[2], b[3], brow + k);
      mma_bf16_16816(sc[0], a, b[0], b[1]);
      mma_bf16_16816(sc[1], a, b[2], b[3]);
    }
    const int key0 = first + s * kStepKeys;
    float top[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        sc[j][e] = key0 + 8 * j + q2 + (e & 1) <= pos ? sc[j][e] * scale2 : -INFINITY;
        top[e >> 1] = fmaxf(top[e >> 1], sc[j][e]);
      }
    bool grown = false;
    float keep[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      top[u] = fmaxf(top[u], __shfl_xor_sync(0xffffffffu, top[u], 1));
      top[u] = fmaxf(top[u], __shfl_xor_sync(0xffffffffu, top[u], 2));
      const float x = fmaxf(m[u], top[u]);           // finite: a step holds at least one visible key
      keep[u] = m[u] == -INFINITY ? 0.f : ex2_approx(m[u] - x);
      grown |= x > m[u];
      m[u] = x;
    }
    if (__any_sync(0xffffffffu, grown)) {
#pragma unroll
      for (int u = 0; u < 2; ++u) l[u] *= keep[u];
#pragma unroll
      for (int i = 0; i < NP; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[i][j][e] *= keep[e >> 1];
    }
    float w[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        w[j][e] = ex2_approx(sc[j][e] - m[e >> 1]);
        l[e >> 1] += w[j][e];
      }
    // the accumulator layout of 16 x 16 scores is the operand layout of one 16-key product
    const uint32_t a[4] = {pack_bf16(w[0][0], w[0][1]), pack_bf16(w[0][2], w[0][3]), pack_bf16(w[1][0], w[1][1]),
                           pack_bf16(w[1][2], w[1][3])};
    const __nv_bfloat16* vrow = vt + (lane & 15) * VS + (lane >> 4) * 8;
#pragma unroll
    for (int i = 0; i < NP; ++i)
      if (16 * i < vp) {
        uint32_t b[4];
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], vrow + 16 * i);
        mma_bf16_16816(acc[i][0], a, b[0], b[1]);
        mma_bf16_16816(acc[i][1], a, b[2], b[3]);
      }
    __syncwarp();
  }
  cp_async_wait<0>();
  __syncthreads();                       // the stages become the merge buffers
  float* po = reinterpret_cast<float*>(stages);                    // [warp][16][vp]
  float* co = po + kAttendWarps * 16 * vp;                         // [16][vp] of the CTA
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    l[u] += __shfl_xor_sync(0xffffffffu, l[u], 1);
    l[u] += __shfl_xor_sync(0xffffffffu, l[u], 2);
    const int row = gq + 8 * u;
    if ((lane & 3) == 0) {
      ml[warp * 32 + 2 * row] = m[u];
      ml[warp * 32 + 2 * row + 1] = l[u];
    }
#pragma unroll
    for (int i = 0; i < NP; ++i)
      if (16 * i < vp)
#pragma unroll
        for (int j = 0; j < 2; ++j)
          *reinterpret_cast<float2*>(po + (warp * 16 + row) * vp + 16 * i + 8 * j + q2) =
              make_float2(acc[i][j][2 * u], acc[i][j][2 * u + 1]);
  }
  __syncthreads();
  const bool alone = p.n_splits == 1;
  auto finish = [&](int row, int c, float4 o, float sum) {
    const int h = h0 + row;
    if (h >= h_end) return;
    const float f = (sum > 0.f ? 1.0f / sum : 0.f) * (p.gate.data != nullptr ? sigmoid_f32(proj_at(p.gate, r, h)) : 1.f);
    store4(out + h * vp + c, make_float4(o.x * f, o.y * f, o.z * f, o.w * f));
  };
  // weighted sum of `parts` partial results; where(i) -> {maximum and sum of the row, output piece}
  for (int i = tid; i < 4 * vp; i += blockDim.x) {
    const int row = i / (vp / 4), c = 4 * (i % (vp / 4));
    float top = -INFINITY, sum = 0.f;
#pragma unroll
    for (int k = 0; k < kAttendWarps; ++k) top = fmaxf(top, ml[k * 32 + 2 * row]);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < kAttendWarps; ++k) {
      const float wk = ml[k * 32 + 2 * row] == -INFINITY ? 0.f : ex2_approx(ml[k * 32 + 2 * row] - top);
      const float4 v = *reinterpret_cast<const float4*>(po + (k * 16 + row) * vp + c);
      sum += wk * ml[k * 32 + 2 * row + 1];
      o.x += wk * v.x;
      o.y += wk * v.y;
      o.z += wk * v.z;
      o.w += wk * v.w;
    }
    if (alone) {
      finish(row, c, o, sum);
    } else {
      *reinterpret_cast<float4*>(co + row * vp + c) = o;
      if (c == 0) {
        cml[2 * row] = top;
        cml[2 * row + 1] = sum;
      }
    }
  }
  if (alone) return;
  cg::cluster_group cluster = cg::this_cluster();
  cluster.sync();
  for (int i = split * blockDim.x + tid; i < 4 * vp; i += p.n_splits * blockDim.x) {
    const int row = i / (vp / 4), c = 4 * (i % (vp / 4));
    float top = -INFINITY, sum = 0.f;
    for (int k = 0; k < p.n_splits; ++k) top = fmaxf(top, cluster.map_shared_rank(cml, k)[2 * row]);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < p.n_splits; ++k) {
      const float* km = cluster.map_shared_rank(cml, k);
      const float wk = km[2 * row] == -INFINITY ? 0.f : ex2_approx(km[2 * row] - top);
      const float4 v = *reinterpret_cast<const float4*>(cluster.map_shared_rank(co, k) + row * vp + c);
      sum += wk * km[2 * row + 1];
      o.x += wk * v.x;
      o.y += wk * v.y;
      o.z += wk * v.z;
      o.w += wk * v.w;
    }
    finish(row, c, o, sum);
  }
  cluster.sync();                        // peers may still read this CTA's partial results
}

template <int NP>
static int launch_group_attend(const ds41_group_attend_args& a, cudaStream_t st) {
  const int smem = attend_smem(a.dim_pad, a.vdim_pad);
  static int allowed = 47 * 1024;
  if (smem > allowed) {
    const cudaError_t e = cudaFuncSetAttribute(group_attend_mma_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    allowed = smem;
  }
  const int m_tiles = (a.heads / a.kv_heads + 15) / 16;
  const dim3 grid(a.n_splits, a.kv_heads * m_tiles, a.rows), block(kAttendWarps * 32);
  if (a.n_splits == 1) return launch_pdl(group_attend_mma_kernel<NP>, grid, block, smem, st, a);
  return launch_pdl_cluster(group_attend_mma_kernel<NP>, grid, block, a.n_splits, smem, st, a);
}

}  // namespace ds41

using namespace ds41;

extern "C" int ds41_attn_post(const ds41_attn_post_args* a, void* stream) {
  if (a == nullptr || !proj_ok(a->u) || !proj_vec4(a->u) || a->q == nullptr || a->pool == nullptr || a->page_table == nullptr ||
      a->row_pos == nullptr || a->row_slot == nullptr || a->rows <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->dim <= 0 ||
      a->dim_pad < a->dim || (a->dim_pad & 15) || a->vdim_pad <= 0 || (a->vdim_pad & 15) || a->taps < 1 || a->slots <= 0 ||
      a->max_pages <= 0 || a->page_tokens <= 0 || (a->q_norm != nullptr) != (a->k_norm != nullptr))
    return cudaErrorInvalidValue;
  const int C = (a->heads + a->kv_heads) * a->dim_pad + a->kv_heads * a->vdim_pad;
  if ((a->taps > 1 && (a->conv == nullptr || a->state == nullptr)) || a->u.ld < a->u.col + C ||
      a->ld_q < a->heads * a->dim_pad || (a->ld_q & 3) || (a->rot_dim & 1) || a->rot_dim < 0 || a->rot_dim > a->dim || a->rot_dim > 2 * kPostTurns || (a->rot_dim > 0 && a->freq == nullptr))
    return cudaErrorInvalidValue;
  const int smem = 4 * C;
  if (smem > 220 * 1024) return cudaErrorInvalidValue;
  static int allowed[2] = {40 * 1024, 40 * 1024};
  int& have = allowed[a->f32 ? 1 : 0];
  if (smem > have) {
    const cudaError_t e = a->f32 ? cudaFuncSetAttribute(attn_post_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem)
                                 : cudaFuncSetAttribute(attn_post_kernel<__nv_bfloat16>,
                                                        cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    have = smem;
  }
  const dim3 block(C >= 2048 ? 512 : (C >= 1024 ? 256 : 128));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->f32 ? launch_pdl(attn_post_kernel<float>, dim3(a->rows), block, smem, st, *a)
                : launch_pdl(attn_post_kernel<__nv_bfloat16>, dim3(a->rows), block, smem, st, *a);
}

extern "C" int ds41_group_attend(const ds41_group_attend_args* a, void* stream) {
  if (!group_attend_ok(a) || a->n_splits < 1 || a->n_splits > 8 || a->rows > 65535) return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int m_tiles = (a->heads / a->kv_heads + 15) / 16;
  const bool aligned = !((reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->pool)) & 15) && !(a->ld_q & 7) &&
                       !(a->ld_out & 3) && !(reinterpret_cast<uintptr_t>(a->out) & 7);
  if (!a->f32 && aligned && a->vdim_pad <= 256 && attend_smem(a->dim_pad, a->vdim_pad) <= 226 * 1024 &&
      a->kv_heads * m_tiles <= 65535) {
    if (a->vdim_pad <= 64) return launch_group_attend<4>(*a, st);
    if (a->vdim_pad <= 128) return launch_group_attend<8>(*a, st);
    return launch_group_attend<16>(*a, st);
  }
  const size_t smem = (1ull * a->dim_pad + a->vdim_pad + 32) * sizeof(float);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const dim3 grid(a->heads, a->rows);
  return a->f32 ? launch_pdl(group_attend_plain_kernel<float>, grid, dim3(128), smem, st, *a)
                : launch_pdl(group_attend_plain_kernel<__nv_bfloat16>, grid, dim3(128), smem, st, *a);
}
