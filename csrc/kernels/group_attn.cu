// Grouped-query attention with a paged cache: query head h reads key / value head h / (heads / kv_heads).  A cache row is
// [keys of all key/value heads | values of all key/value heads], every head padded with zeros to a multiple of 16.
//
//  attn_post    : after the projection: causal convolution over time on every channel of q, k and v; RMS norm over all heads
//                 of q and of k at once; rotation of the leading dimensions of a head; q leaves as a matrix, k and v go into
//                 the request's cache pages
//  group_attend : attention of any mix of rows over the cache, each over its own chunk of the sequence (or everything before
//                 it); the head's output is multiplied by the sigmoid of its gate.  bf16 runs on warp-level tensor cores, a
//                 cluster of up to sixteen CTAs per row and key/value head; 32-bit (and odd sizes) in a plain form
//
// The convolution's last taps - 1 inputs per request live in a ring indexed by position (p % (taps - 1)), so nothing is
// shifted and running a position twice changes nothing.  attn_post reads the ring, the attention kernel that follows writes
// it: rows of one pass never see their successors.
#include <cooperative_groups.h>
#include <cuda.h>

#include "ds41_group.cuh"
#include "ds41_mma.cuh"
#include "ds41_tma.h"

namespace ds41 {

namespace cg = cooperative_groups;

constexpr int kAttendSplits = 16;         // CTAs that share a row's keys
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

// bf16 forms for up to four taps and rotations of a multiple of eight values.  A thread owns units of eight channels: in the
// rotated part of a head four channels and the four that they turn with, else eight neighbours.
//  rows of a long pass : one block per kPostRows rows and section (queries | keys and values), RB rows at a time between two
//                        block-wide sums; the taps stay in registers, every input is read once per RB rows
//  few rows            : a cluster of eight CTAs per row, sums merged through distributed shared memory
constexpr int kPostRows = 8;
constexpr int kPostTaps = 4;

struct PostUnit {
  int a, b;             // first channel of both groups of four (columns of u)
  int turn;             // first pair of the rotation, -1: not turned
  int part;             // 0 query, 1 key, 2 value
};
__device__ __forceinline__ PostUnit post_unit(const ds41_attn_post_args& p, int u) {
  const int per = p.dim_pad / 8, rotated = p.rot_dim / 8, qk = (p.heads + p.kv_heads) * per;
  PostUnit t;
  t.turn = -1;
  t.part = u < p.heads * per ? 0 : (u < qk ? 1 : 2);
  t.a = 8 * u;
  t.b = t.a + 4;
  if (t.part < 2) {
    const int k = u % per, h0 = (u - k) * 8;
    if (k < rotated) {
      t.a = h0 + 4 * k;
      t.b = t.a + p.rot_dim / 2;
      t.turn = 4 * k;
    }
  }
  return t;
}
struct Eight {
  float v[8];
};
__device__ __forceinline__ Eight eight(float4 a, float4 b) { return {{a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w}}; }
__device__ __forceinline__ Eight proj_unit(const ds41_proj& u, long long r, const PostUnit& t) {
  return eight(proj_at4(u, r, t.a), proj_at4(u, r, t.b));
}
__device__ __forceinline__ Eight row_unit(const float* row, const PostUnit& t) {
  return eight(*reinterpret_cast<const float4*>(row + t.a), *reinterpret_cast<const float4*>(row + t.b));
}

// Normed, turned and stored: `x` is the convolved unit times the norm's weight, f the norm's factor.
__device__ __forceinline__ void post_store(const ds41_attn_post_args& p, const PostUnit& t, const Eight& x, float f,
                                           const float2* turns, __nv_bfloat16* q, __nv_bfloat16* row) {
  float o[8];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 cs = t.turn >= 0 ? turns[t.turn + e] : make_float2(1.f, 0.f);
    o[e] = (x.v[e] * cs.x - x.v[4 + e] * cs.y) * f;
    o[4 + e] = (x.v[4 + e] * cs.x + x.v[e] * cs.y) * f;
  }
  const int nq = p.heads * p.dim_pad;
  __nv_bfloat16* dst = t.part == 0 ? q : row;
  if (dst == nullptr) return;
  const int off = t.part == 0 ? 0 : nq;
  store4(dst + (t.a - off), make_float4(o[0], o[1], o[2], o[3]));
  store4(dst + (t.b - off), make_float4(o[4], o[5], o[6], o[7]));
}

// A unit of a projection row as it was loaded: bf16 pairs, or eight floats.
template <bool PACKED>
struct RawUnit {
  uint2 a, b;
  __device__ __forceinline__ void load(const ds41_proj& u, long long r, const PostUnit& t) {
    const __nv_bfloat16* row = static_cast<const __nv_bfloat16*>(u.data) + r * u.ld + u.col;
    a = *reinterpret_cast<const uint2*>(row + t.a);
    b = *reinterpret_cast<const uint2*>(row + t.b);
  }
  __device__ __forceinline__ Eight get() const {
    const uint32_t q[4] = {a.x, a.y, b.x, b.y};
    Eight x;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      x.v[2 * i] = __uint_as_float(q[i] << 16);
      x.v[2 * i + 1] = __uint_as_float(q[i] & 0xffff0000u);
    }
    return x;
  }
};
template <>
struct RawUnit<false> {
  Eight x;
  __device__ __forceinline__ void load(const ds41_proj& u, long long r, const PostUnit& t) { x = proj_unit(u, r, t); }
  __device__ __forceinline__ Eight get() const { return x; }
};

template <int RB, int THREADS, bool PACKED>
__global__ void __launch_bounds__(THREADS) attn_post_rows_kernel(ds41_attn_post_args p) {
  extern __shared__ float2 pr_turns[];             // [kPostRows][rot_dim / 2]
  __shared__ float red[2][THREADS / 32][RB];       // sums of squares per row of a batch
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
  const int nk = p.kv_heads * p.dim_pad, nv = p.kv_heads * p.vdim_pad, C = p.heads * p.dim_pad + nk + nv;
  const int q_units = p.heads * p.dim_pad / 8, units = C / 8, half = p.rot_dim / 2, back = p.taps - 1;
  const int r0 = blockIdx.x * kPostRows, r1 = min(p.rows, r0 + kPostRows);
  const int u = blockIdx.y == 0 ? tid : q_units + tid;
  const bool live = u < (blockIdx.y == 0 ? q_units : units);
  const PostUnit t = post_unit(p, live ? u : 0);
  pdl_launch_dependents();
  Eight w[kPostTaps];                              // tap d reaches d positions back
#pragma unroll
  for (int d = 0; d < kPostTaps; ++d)
    if (live && p.conv != nullptr && d <= back) w[d] = row_unit(p.conv + 1ll * (back - d) * C, t);
    else
#pragma unroll
      for (int e = 0; e < 8; ++e) w[d].v[e] = d == 0 ? 1.f : 0.f;
  pdl_wait();
  for (int i = tid; i < (r1 - r0) * half; i += blockDim.x) {
    float s, c;
    sincosf(static_cast<float>(p.row_pos[r0 + i / half]) * p.freq[i % half], &s, &c);
    pr_turns[i] = make_float2(c, s);
  }
  int parity = 0;
  for (int rb = r0; rb < r1; rb += RB, parity ^= 1) {
    constexpr int kOld = kPostTaps - 1;              // rows before the batch that it reaches
    int own[kOld + RB], pos[RB];                   // slots of rows rb - kOld ..., -1 beyond the pass
#pragma unroll
    for (int i = 0; i < kOld + RB; ++i) {
      const int r = rb + i - kOld;
      own[i] = r >= 0 && r < r1 && i >= kOld - back ? p.row_slot[r] : -1;
    }
#pragma unroll
    for (int j = 0; j < RB; ++j) pos[j] = rb + j < r1 ? p.row_pos[rb + j] : 0;
    RawUnit<PACKED> raw[kOld + RB];
#pragma unroll
    for (int i = 0; i < kOld + RB; ++i)
      if (live && own[i] >= 0) raw[i].load(p.u, rb + i - kOld, t);
    Eight acc[RB];
#pragma unroll
    for (int j = 0; j < RB; ++j)
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[j].v[e] = 0.f;
    if (live) {
#pragma unroll
      for (int i = 0; i < kOld + RB; ++i) {
        if (own[i] < 0) continue;
        const Eight x = raw[i].get();
#pragma unroll
        for (int j = 0; j < RB; ++j) {
          const int d = j + kOld - i;              // positions back from row j, if both belong to one request
          if (d >= 0 && d < kPostTaps && own[kOld + j] == own[i])
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[j].v[e] += w[d >= 0 && d < kPostTaps ? d : 0].v[e] * x.v[e];
        }
      }
      // what earlier passes left, for the first rows of a request's portion
#pragma unroll
      for (int j = 0; j < RB; ++j)
#pragma unroll
        for (int d = 1; d < kPostTaps; ++d) {
          const int slot = own[kOld + j];
          if (slot < 0 || d > back || d > pos[j] || own[kOld + j - d] == slot) continue;
          const Eight x = row_unit(p.state + (1ll * slot * back + (pos[j] - d) % back) * C, t);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[j].v[e] += w[d].v[e] * x.v[e];
        }
    }
    if (p.q_norm != nullptr) {
      const bool normed = live && t.part < 2;
#pragma unroll
      for (int j = 0; j < RB; ++j) {
        float q = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) q += acc[j].v[e] * acc[j].v[e];
        q = warp_sum(normed ? q : 0.f);            // values stand in the keys' section but not in their norm
        if (lane == 0) red[parity][warp][j] = q;
      }
      if (normed) {
        const Eight g = blockIdx.y == 0 ? row_unit(p.q_norm, t) : row_unit(p.k_norm - p.heads * p.dim_pad, t);
#pragma unroll
        for (int j = 0; j < RB; ++j)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[j].v[e] *= g.v[e];
      }
    }
    __syncthreads();                               // sums, and the sines of the first batch
#pragma unroll
    for (int j = 0; j < RB; ++j) {
      const int slot = own[kOld + j];
      if (slot < 0) continue;
      float f = 1.f;
      if (p.q_norm != nullptr) {                   // every lane takes part: a warp may hold keys and values
        const float q = warp_sum(lane < n_warps ? red[parity][lane][j] : 0.f);
        if (t.part < 2) f = 1.0f / sqrtf(q / ((blockIdx.y == 0 ? p.heads : p.kv_heads) * p.dim) + p.eps);
      }
      if (!live) continue;
      __nv_bfloat16* row = blockIdx.y == 0 ? nullptr
                                           : cache_row(static_cast<__nv_bfloat16*>(p.pool), p.page_table, p.max_pages,
                                                       p.page_tokens, nk + nv, slot, pos[j]);
      post_store(p, t, acc[j], f, pr_turns + (rb - r0 + j) * half, static_cast<__nv_bfloat16*>(p.q) + (rb + j) * p.ld_q, row);
    }
  }
}

template <int THREADS>
__global__ void __launch_bounds__(THREADS) attn_post_few_kernel(ds41_attn_post_args p) {
  __shared__ float2 turns[kPostTurns];
  __shared__ float red[THREADS / 32][2];
  __shared__ float sums[2];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
  const int nk = p.kv_heads * p.dim_pad, nv = p.kv_heads * p.vdim_pad, C = p.heads * p.dim_pad + nk + nv;
  const int units = C / 8, half = p.rot_dim / 2, back = p.taps - 1;
  const int r = blockIdx.x / 8, part = blockIdx.x % 8, per = (units + 7) / 8;
  const int u = part * per + tid;
  const bool live = tid < per && u < units;
  const PostUnit t = post_unit(p, live ? u : 0);
  pdl_launch_dependents();
  Eight w[kPostTaps], g;
#pragma unroll
  for (int d = 0; d < kPostTaps; ++d)
    if (live && p.conv != nullptr && d <= back) w[d] = row_unit(p.conv + 1ll * (back - d) * C, t);
    else
#pragma unroll
      for (int e = 0; e < 8; ++e) w[d].v[e] = d == 0 ? 1.f : 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) g.v[e] = 1.f;
  if (live && t.part < 2 && p.q_norm != nullptr)
    g = t.part == 0 ? row_unit(p.q_norm, t) : row_unit(p.k_norm - p.heads * p.dim_pad, t);
  pdl_wait();
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  if (slot < 0) return;                            // the same in every CTA of the cluster
  Eight x[kPostTaps];
#pragma unroll
  for (int d = 0; d < kPostTaps; ++d) {
#pragma unroll
    for (int e = 0; e < 8; ++e) x[d].v[e] = 0.f;
    if (!live || d > back || d > pos) continue;
    if (d == 0 || (r - d >= 0 && p.row_slot[r - d] == slot)) x[d] = proj_unit(p.u, r - d, t);
    else x[d] = row_unit(p.state + (1ll * slot * back + (pos - d) % back) * C, t);
  }
  for (int i = tid; i < half; i += blockDim.x) {
    float s, c;
    sincosf(static_cast<float>(pos) * p.freq[i], &s, &c);
    turns[i] = make_float2(c, s);
  }
  float f = 1.f, q = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    float a = 0.f;
#pragma unroll
    for (int d = 0; d < kPostTaps; ++d) a += w[d].v[e] * x[d].v[e];
    q += a * a;
    x[0].v[e] = a * g.v[e];
  }
  if (p.q_norm != nullptr) {
    const float sq = warp_sum(live && t.part == 0 ? q : 0.f), sk = warp_sum(live && t.part == 1 ? q : 0.f);
    if (lane == 0) {
      red[warp][0] = sq;
      red[warp][1] = sk;
    }
    __syncthreads();
    if (tid < 2) {
      float s = 0.f;
      for (int i = 0; i < n_warps; ++i) s += red[i][tid];
      sums[tid] = s;
    }
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    const float* far = cluster.map_shared_rank(sums, lane & 7);
    const float a = warp_sum(lane < 8 ? far[0] : 0.f), b = warp_sum(lane < 8 ? far[1] : 0.f);
    if (t.part == 0) f = 1.0f / sqrtf(a / (p.heads * p.dim) + p.eps);
    if (t.part == 1) f = 1.0f / sqrtf(b / (p.kv_heads * p.dim) + p.eps);
    if (live) {
      __nv_bfloat16* row = t.part == 0 ? nullptr
                                       : cache_row(static_cast<__nv_bfloat16*>(p.pool), p.page_table, p.max_pages,
                                                   p.page_tokens, nk + nv, slot, pos);
      post_store(p, t, x[0], f, turns, static_cast<__nv_bfloat16*>(p.q) + r * p.ld_q, row);
    }
    cluster.sync();                                // peers may still read this CTA's sums
    return;
  }
  __syncthreads();
  if (live) {
    __nv_bfloat16* row = t.part == 0 ? nullptr
                                     : cache_row(static_cast<__nv_bfloat16*>(p.pool), p.page_table, p.max_pages, p.page_tokens,
                                                 nk + nv, slot, pos);
    post_store(p, t, x[0], f, turns, static_cast<__nv_bfloat16*>(p.q) + r * p.ld_q, row);
  }
}

// The form of this launch that the sizes allow: 0 the general one.
static int launch_post_fast(const ds41_attn_post_args& a, cudaStream_t st, bool& done) {
  const int q_units = a.heads * a.dim_pad / 8, units = q_units + a.kv_heads * (a.dim_pad + a.vdim_pad) / 8;
  done = !a.f32 && a.taps <= kPostTaps && !(a.rot_dim & 7) && !(a.ld_q & 3);
  if (!done) return cudaSuccess;
  if (a.rows <= 32) {
    const int threads = ((units + 7) / 8 + 31) / 32 * 32;
    if (threads <= 128) return launch_pdl_cluster(attn_post_few_kernel<128>, dim3(8 * a.rows), dim3(threads), 8, 0, st, a);
    if (threads <= 512) return launch_pdl_cluster(attn_post_few_kernel<512>, dim3(8 * a.rows), dim3(threads), 8, 0, st, a);
  }
  const int most = q_units > units - q_units ? q_units : units - q_units, threads = (most + 31) / 32 * 32;
  const dim3 grid((a.rows + kPostRows - 1) / kPostRows, 2);
  const int smem = kPostRows * (a.rot_dim / 2) * static_cast<int>(sizeof(float2));
  if (threads <= 1024 && smem <= 40 * 1024) {
    if (threads > 512)
      return a.u.bf16 ? launch_pdl(attn_post_rows_kernel<2, 1024, true>, grid, dim3(threads), smem, st, a)
                      : launch_pdl(attn_post_rows_kernel<2, 1024, false>, grid, dim3(threads), smem, st, a);
    if (threads > 256 || !a.u.bf16)
      return a.u.bf16 ? launch_pdl(attn_post_rows_kernel<4, 512, true>, grid, dim3(threads), smem, st, a)
                      : launch_pdl(attn_post_rows_kernel<2, 512, false>, grid, dim3(threads), smem, st, a);
    return launch_pdl(attn_post_rows_kernel<4, 256, true>, grid, dim3(threads), smem, st, a);
  }
  done = false;
  return cudaSuccess;
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
  keep_inputs(p, r, slot, pos, h, gridDim.x, tid, 128);
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

// bf16 form: CTA (split, key/value head and 16 of its query heads, row).  A producer warp brings tiles of 16 NW keys and values
// page by page with TMA (128-byte swizzle) through a ring of stages; each of NW warps scores 16 of the keys and
// accumulates their values with a softmax state of its own - no block-wide wait until the partial results are merged: over
// the warps in shared memory, over the CTAs of the cluster through distributed shared memory.
// KD: 16-column pieces of the key width, NP: of the value width.  A warp's walk is a chain of latencies, so a CTA has eight
// of them; four, and two CTAs share an SM, where there are more CTAs than SMs (or the value width takes the registers).
constexpr int kMaxStages = 4;

struct AttendPlan {
  int warps, kc, vc, stages, box;                     // 64-column chunks, ring length, rows per TMA box
};

inline int attend_smem(const AttendPlan& t, int dp) {
  return 1024 + t.stages * (t.kc + t.vc) * t.warps * 16 * 128 + 16 * (dp + 8) * 2 + (t.warps + 1) * 32 * 4 + 16 * kMaxStages;
}

// Tiles and pages of this launch; false: the plain form has to run.
inline bool plan_attend(const ds41_group_attend_args& a, AttendPlan& t) {
  if (a.f32 || a.vdim_pad > 256 || a.dim_pad > 256 || a.n_pages <= 0 || (a.ld_q & 7) || (a.ld_out & 3) ||
      ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.pool)) & 15) || (reinterpret_cast<uintptr_t>(a.out) & 7))
    return false;
  t.kc = (a.dim_pad + 63) / 64;
  t.vc = (a.vdim_pad + 63) / 64;
  const int m_tiles = (a.heads / a.kv_heads + 15) / 16;
  const bool many = 1ll * a.n_splits * a.kv_heads * m_tiles * a.rows > sm_count();
  for (t.warps = a.vdim_pad <= 128 && !many ? 8 : 4; t.warps >= 4; t.warps -= 4) {
    const int keys = 16 * t.warps;
    t.box = a.page_tokens % keys == 0 ? keys : a.page_tokens;
    if (t.box < 8 || keys % t.box != 0) continue;
    // the partial results of the warps and of the CTA take the place of the stages
    const int merge = (t.warps + 1) * 16 * a.vdim_pad * 4, stage = (t.kc + t.vc) * keys * 128;
    for (int room : {many ? 112 : 226, 226})
      for (t.stages = kMaxStages; t.stages >= 2; --t.stages)
        if (attend_smem(t, a.dim_pad) <= room * 1024 && t.stages * stage >= merge) return true;
  }
  return false;
}

template <int NW, int KD, int NP>
__global__ void __launch_bounds__(32 * (NW + 1))
group_attend_mma_kernel(const __grid_constant__ CUtensorMap pool, const ds41_group_attend_args p, const AttendPlan plan) {
  constexpr int kTileKeys = 16 * NW, kTileChunk = kTileKeys * 128;      // bytes of a tile's rows x 64 bf16 columns
  extern __shared__ uint8_t gm_raw[];
  uint8_t* stages = gm_raw + ((1024u - (smem_u32(gm_raw) & 1023u)) & 1023u);
  const int dp = p.dim_pad, vp = p.vdim_pad, KS = dp + 8, stage_bytes = (plan.kc + plan.vc) * kTileChunk;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, q2 = 2 * (lane & 3);
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(stages + plan.stages * stage_bytes);   // [16][KS]
  float* ml = reinterpret_cast<float*>(sq + 16 * KS);                                         // [warp][16]{max, sum}
  float* cml = ml + NW * 32;                                                        // [16]{max, sum} of the CTA
  uint64_t* full = reinterpret_cast<uint64_t*>(cml + 32);                                     // [stages]
  uint64_t* empty = full + kMaxStages;
  const int n = p.heads / p.kv_heads, m_tiles = (n + 15) / 16;
  const int split = blockIdx.x, g = blockIdx.y / m_tiles, h0 = g * n + (blockIdx.y % m_tiles) * 16, r = blockIdx.z;
  const int h_end = (g + 1) * n;                                               // heads [h0, min(h0 + 16, h_end))
  if (tid == 0) {
    for (int i = 0; i < plan.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], NW);
    }
    mbar_init_fence();
    tma_prefetch_desc(&pool);
  }
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
  const int first = chunk_start(pos, p.chunk), base = first - first % plan.box;
  const int tiles = (pos - base) / kTileKeys + 1, per = (tiles + p.n_splits - 1) / p.n_splits;
  const int t0 = min(tiles, split * per), t1 = min(tiles, t0 + per);
  if (warp < NW) {
    for (int i = warp; i < 16; i += NW) {
      const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q) + r * p.ld_q + (h0 + i) * dp;
      for (int d = lane * 8; d < dp; d += 256)
        *reinterpret_cast<uint4*>(sq + i * KS + d) =
            h0 + i < h_end ? *reinterpret_cast<const uint4*>(q + d) : make_uint4(0, 0, 0, 0);
    }
  }
  __syncthreads();
  float acc[NP][2][4];
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  if (warp == NW) {
    // ---- producer: lane i holds the pool row of box i of the walk (32 boxes at a time)
    const int boxes = kTileKeys / plan.box;
    const int* table = p.page_table + 1ll * slot * p.max_pages;
    int row = 0;
    bool ok = true;
    int t = t0, u = 0;
    for (; t < t1 && ok; ++t) {
      const int stage = (t - t0) % plan.stages;
      for (int i = 0; i < boxes && ok; ++i, ++u) {
        if ((u & 31) == 0) {
          const int key = base + t * kTileKeys + (i + lane) * plan.box, pg = key / p.page_tokens;
          const int id = key <= pos && pg < p.max_pages ? table[pg] : -1;
          row = id >= 0 ? id * p.page_tokens + (key - pg * p.page_tokens) : p.n_pages * p.page_tokens;
        }
        if (i == 0) {
          ok = __all_sync(0xffffffffu, mbar_wait(&empty[stage], (((t - t0) / plan.stages) & 1) ^ 1, p.status, 440)) != 0;
          if (!ok) break;
          if (lane == 0) mbar_expect_tx(&full[stage], stage_bytes);
        }
        const int at = __shfl_sync(0xffffffffu, row, u & 31);
        if (lane == 0) {
          uint8_t* dst = stages + stage * stage_bytes + i * plan.box * 128;
          for (int c = 0; c < plan.kc; ++c) tma_load_3d(dst + c * kTileChunk, &pool, &full[stage], g * dp + 64 * c, at, 0);
          for (int c = 0; c < plan.vc; ++c)
            tma_load_3d(dst + (plan.kc + c) * kTileChunk, &pool, &full[stage], p.kv_heads * dp + g * vp + 64 * c, at, 0);
        }
      }
    }
    if (!ok) {                           // something gave up: let the copies in flight land before the memory changes hands
      for (int b = max(t0, t - 1 - plan.stages); b < t - 1; ++b)
        for (int i = 0; i < (1 << 20) && !mbar_test_wait(&full[(b - t0) % plan.stages], ((b - t0) / plan.stages) & 1); ++i) {
        }
    }
    keep_inputs(p, r, slot, pos, split + p.n_splits * blockIdx.y, p.n_splits * gridDim.y, lane, 32);
  } else {
#pragma unroll
    for (int i = 0; i < NP; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
    const float scale2 = p.scale * 1.4426950408889634f;
    const __nv_bfloat16* arow = sq + (lane & 15) * KS + (lane >> 4) * 8;
    constexpr bool kHeld = KD <= 8;      // the query fragments stay in registers
    uint32_t qf[kHeld ? KD : 1][4];
    if (kHeld)
#pragma unroll
      for (int k = 0; k < KD; ++k)
        if (16 * k < dp) ldmatrix_x4(qf[k][0], qf[k][1], qf[k][2], qf[k][3], arow + 16 * k);
    // this lane's rows of the warp's 16 keys: as operand of the scores, as operand of the values
    const int krow = 16 * warp + (lane & 7) + (lane >> 4) * 8, kpiece = (lane >> 3) & 1;
    const int vrow = 16 * warp + (lane & 15), vpiece = lane >> 4;
    auto swizzled = [](const uint8_t* tile, int row, int piece) {      // 16-byte piece of a row, chunks of 8 pieces
      return tile + (piece >> 3) * kTileChunk + row * 128 + (((piece & 7) ^ (row & 7)) << 4);
    };
    bool ok = true;
    for (int t = t0; t < t1; ++t) {
      const int stage = (t - t0) % plan.stages;
      ok = __all_sync(0xffffffffu, mbar_wait(&full[stage], ((t - t0) / plan.stages) & 1, p.status, 441)) != 0;
      if (!ok) break;
      const uint8_t* kt = stages + stage * stage_bytes;
      const uint8_t* vt = kt + plan.kc * kTileChunk;
      const int key0 = base + t * kTileKeys + 16 * warp;
      if (key0 <= pos && key0 + 15 >= first) {       // the warp's keys hold at least one visible one
        float sc[2][2][4] = {};                      // even and odd pieces: two chains of dependent products
#pragma unroll
        for (int k0 = 0; k0 < KD; k0 += 4) {
          uint32_t b[4][4], a[4][4];
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (16 * (k0 + k) < dp) {
              ldmatrix_x4(b[k][0], b[k][1], b[k][2], b[k][3], swizzled(kt, krow, 2 * (k0 + k) + kpiece));
              if (!kHeld) ldmatrix_x4(a[k][0], a[k][1], a[k][2], a[k][3], arow + 16 * (k0 + k));
            }
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (16 * (k0 + k) < dp) {
              mma_bf16_16816(sc[k & 1][0], kHeld ? qf[kHeld ? k0 + k : 0] : a[k], b[k][0], b[k][1]);
              mma_bf16_16816(sc[k & 1][1], kHeld ? qf[kHeld ? k0 + k : 0] : a[k], b[k][2], b[k][3]);
            }
        }
        float top[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int key = key0 + 8 * j + q2 + (e & 1);
            sc[0][j][e] = key <= pos && key >= first ? (sc[0][j][e] + sc[1][j][e]) * scale2 : -INFINITY;
            top[e >> 1] = fmaxf(top[e >> 1], sc[0][j][e]);
          }
        bool grown = false;
        float keep[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          top[u] = fmaxf(top[u], __shfl_xor_sync(0xffffffffu, top[u], 1));
          top[u] = fmaxf(top[u], __shfl_xor_sync(0xffffffffu, top[u], 2));
          const float x = fmaxf(m[u], top[u]);       // finite
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
            w[j][e] = ex2_approx(sc[0][j][e] - m[e >> 1]);
            l[e >> 1] += w[j][e];
          }
        // the accumulator layout of 16 x 16 scores is the operand layout of one 16-key product
        const uint32_t wa[4] = {pack_bf16(w[0][0], w[0][1]), pack_bf16(w[0][2], w[0][3]), pack_bf16(w[1][0], w[1][1]),
                                pack_bf16(w[1][2], w[1][3])};
#pragma unroll
        for (int i0 = 0; i0 < NP; i0 += 4) {
          uint32_t b[4][4];
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (16 * (i0 + i) < vp)
              ldmatrix_x4_trans(b[i][0], b[i][1], b[i][2], b[i][3], swizzled(vt, vrow, 2 * (i0 + i) + vpiece));
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (16 * (i0 + i) < vp) {
              mma_bf16_16816(acc[i0 + i][0], wa, b[i][0], b[i][1]);
              mma_bf16_16816(acc[i0 + i][1], wa, b[i][2], b[i][3]);
            }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty[stage]);
    }
  }
  __syncthreads();                       // the stages become the merge buffers
  float* po = reinterpret_cast<float*>(stages);                    // [warp][16][vp]
  float* co = po + NW * 16 * vp;                         // [16][vp] of the CTA
  if (warp < NW) {
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
  }
  __syncthreads();
  const bool alone = p.n_splits == 1;
  auto finish = [&](int row, int c, float4 o, float sum) {
    const int h = h0 + row;
    if (h >= h_end) return;
    const float f = (sum > 0.f ? 1.0f / sum : 0.f) * (p.gate.data != nullptr ? sigmoid_f32(proj_at(p.gate, r, h)) : 1.f);
    store4(out + h * vp + c, make_float4(o.x * f, o.y * f, o.z * f, o.w * f));
  };
  const int rows = min(16, h_end - h0);
  for (int i = tid; i < rows * vp / 4; i += blockDim.x) {
    const int row = i / (vp / 4), c = 4 * (i % (vp / 4));
    float top = -INFINITY, sum = 0.f;
#pragma unroll
    for (int k = 0; k < NW; ++k) top = fmaxf(top, ml[k * 32 + 2 * row]);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < NW; ++k) {
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
  for (int i = split * blockDim.x + tid; i < rows * vp / 4; i += p.n_splits * blockDim.x) {
    const int row = i / (vp / 4), c = 4 * (i % (vp / 4));
    float top = -INFINITY, sum = 0.f;
    for (int k = 0; k < p.n_splits; ++k) top = fmaxf(top, cluster.map_shared_rank(cml, k)[2 * row]);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
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

template <int NW, int KD, int NP>
static int launch_group_attend(const ds41_group_attend_args& a, const AttendPlan& plan, cudaStream_t st) {
  const int smem = attend_smem(plan, a.dim_pad), row_len = a.kv_heads * (a.dim_pad + a.vdim_pad);
  static bool ready = false;
  cudaError_t e;
  if (!ready) {
    e = cudaFuncSetAttribute(group_attend_mma_kernel<NW, KD, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
    if (e != cudaSuccess) return e;
    e = cudaFuncSetAttribute(group_attend_mma_kernel<NW, KD, NP>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    if (e != cudaSuccess) return e;
    ready = true;
  }
  CUtensorMap pool;
  e = make_tensor_map_3d(&pool, a.pool, TmaDtype::kBF16, row_len, 1ull * a.n_pages * a.page_tokens, 1, 2ull * row_len, 0, 64,
                         plan.box, true);
  if (e != cudaSuccess) return e;
  const int m_tiles = (a.heads / a.kv_heads + 15) / 16;
  const dim3 grid(a.n_splits, a.kv_heads * m_tiles, a.rows), block(32 * (NW + 1));
  if (a.n_splits == 1) return launch_pdl(group_attend_mma_kernel<NW, KD, NP>, grid, block, smem, st, pool, a, plan);
  return launch_pdl_cluster(group_attend_mma_kernel<NW, KD, NP>, grid, block, a.n_splits, smem, st, pool, a, plan);
}

static int dispatch_group_attend(const ds41_group_attend_args& a, const AttendPlan& plan, cudaStream_t st) {
  if (plan.warps == 8) {
    if (a.dim_pad > 128) return launch_group_attend<8, 16, 8>(a, plan, st);
    if (a.dim_pad > 64)
      return a.vdim_pad <= 64 ? launch_group_attend<8, 8, 4>(a, plan, st) : launch_group_attend<8, 8, 8>(a, plan, st);
    return a.vdim_pad <= 64 ? launch_group_attend<8, 4, 4>(a, plan, st) : launch_group_attend<8, 4, 8>(a, plan, st);
  }
  if (a.dim_pad > 128) return launch_group_attend<4, 16, 16>(a, plan, st);
  if (a.vdim_pad > 128) return launch_group_attend<4, 8, 16>(a, plan, st);
  if (a.dim_pad > 64) return launch_group_attend<4, 8, 8>(a, plan, st);
  return a.vdim_pad <= 64 ? launch_group_attend<4, 4, 4>(a, plan, st) : launch_group_attend<4, 4, 8>(a, plan, st);
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
      a->ld_q < a->heads * a->dim_pad || (a->ld_q & 3) || (a->rot_dim & 1) || a->rot_dim < 0 ||
      a->rot_dim > a->dim || a->rot_dim > 2 * kPostTurns || (a->rot_dim > 0 && a->freq == nullptr))
    return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  bool done = false;
  const int e = launch_post_fast(*a, st, done);
  if (done) return e;
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
  return a->f32 ? launch_pdl(attn_post_kernel<float>, dim3(a->rows), block, smem, st, *a)
                : launch_pdl(attn_post_kernel<__nv_bfloat16>, dim3(a->rows), block, smem, st, *a);
}

extern "C" int ds41_group_attend(const ds41_group_attend_args* a, void* stream) {
  if (!group_attend_ok(a) || a->n_splits < 1 || a->n_splits > kAttendSplits || a->rows > 65535) return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  AttendPlan plan;
  if (plan_attend(*a, plan) && a->kv_heads * ((a->heads / a->kv_heads + 15) / 16) <= 65535)
    return dispatch_group_attend(*a, plan, st);
  const size_t smem = (1ull * a->dim_pad + a->vdim_pad + 32) * sizeof(float);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const dim3 grid(a->heads, a->rows);
  return a->f32 ? launch_pdl(group_attend_plain_kernel<float>, grid, dim3(128), smem, st, *a)
                : launch_pdl(group_attend_plain_kernel<__nv_bfloat16>, grid, dim3(128), smem, st, *a);
}
