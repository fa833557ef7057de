// Matrix-memory recurrence (mLSTM of xLSTM) with a running maximum.
//
// Per head the state is a dim x vdim matrix S, a vector n and a scalar m, all fp32, one set per request slot:
//   m' = max(f + m, i);  S' = exp(f + m - m') S + exp(i - m') k v^T;  n' the same with k alone
//   o  = S'^T q / (max(|n' . q|, exp(-m')) + den_eps)
// A block owns 32 value columns of one head.  Every column block carries its own copy of n and m, so blocks never wait for
// one another.  A request's state starts at zero where its rows start at position 0.
//
//  mlstm_step : one block walks the adjacent rows of a request token by token (decode rows, 32-bit passes)
//  mlstm_chunk: one request's rows, 64 at a time, on the tensor cores.  With F the running sum of f inside a chunk and m0
//               the maximum before it, m_t = F_t + max(m0, max_{s<=t}(i_s - F_s)) is the same maximum the walk would find, and
//                 S'^T q_t = exp(F_t + m0 - m_t) S^T q_t + sum_{s<=t} exp(F_t - F_s + i_s - m_t) (k_s . q_t) v_s
//               fp32 factors of a product (state, decayed scores, decayed values) enter as bf16 high and low parts.
#include "ds41_mma.cuh"
#include "ds41_stack.cuh"

namespace ds41 {

constexpr int kStateCols = 32;

struct GateValues {
  float i, f;
};
__device__ __forceinline__ GateValues mlstm_gates(const ds41_mlstm_args& p, int r, int h) {
  const float gi = proj_at(p.gate_i, r, h) + p.bias_i[h], gf = proj_at(p.gate_f, r, h) + p.bias_f[h];
  return {p.gate_cap * tanhf(gi / p.gate_cap), log_sigmoid_f32(p.gate_cap * tanhf(gf / p.gate_cap))};
}

__global__ void __launch_bounds__(256) mlstm_step_kernel(ds41_mlstm_args p) {
  extern __shared__ float ms_smem[];
  const int D = p.dim_pad;
  float* S = ms_smem;                       // [D][32]
  float* n = S + D * kStateCols;            // [D]
  float* qs = n + D;
  float* ks = qs + D;
  float* vs = ks + D;                       // [32]
  float* part = vs + kStateCols;            // [8][32]
  __shared__ float red[33];
  __shared__ float gates[2];
  const int vb = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_launch_dependents();
  pdl_wait();
  int r = blockIdx.z;
  if (!segment_start(p.row_slot, r)) return;
  const int slot = p.row_slot[r];
  if (slot >= p.slots) return;
  const int nb = gridDim.x, col = vb * kStateCols + lane;
  const bool live = col < p.vdim_pad;
  const bool fresh = p.row_pos[r] == 0;
  const long long head = 1ll * slot * p.heads + h;
  float* gS = p.state_s + head * D * p.vdim_pad;
  float* gn = p.state_n + (head * nb + vb) * D;
  float* gm = p.state_m + head * nb + vb;
#pragma unroll 4
  for (int d = warp; d < D; d += 8) S[d * kStateCols + lane] = fresh || !live ? 0.f : gS[1ll * d * p.vdim_pad + col];
  for (int d = tid; d < D; d += 256) n[d] = fresh ? 0.f : gn[d];
  float m = fresh ? 0.f : *gm;
  for (; r < p.rows && p.row_slot[r] == slot; ++r) {
    __syncthreads();
    for (int d = tid; d < D; d += 256) {
      qs[d] = proj_at(p.q, r, h * D + d) * p.q_scale;
      ks[d] = proj_at(p.k, r, h * D + d);
    }
    if (tid < kStateCols) vs[tid] = live ? proj_at(p.v, r, h * p.vdim_pad + col) : 0.f;
    if (tid == 32) {
      const GateValues g = mlstm_gates(p, r, h);
      gates[0] = g.i;
      gates[1] = g.f;
    }
    __syncthreads();
    const float m_new = fmaxf(gates[1] + m, gates[0]);
    const float keep = expf(gates[1] + m - m_new), add = expf(gates[0] - m_new);
    m = m_new;
    float nq = 0.f;
    for (int d = tid; d < D; d += 256) {
      const float t = keep * n[d] + add * ks[d];
      n[d] = t;
      nq += t * qs[d];
    }
    const float v = vs[lane] * add;
    float o = 0.f;
#pragma unroll 4
    for (int d = warp; d < D; d += 8) {
      const float s = keep * S[d * kStateCols + lane] + ks[d] * v;
      S[d * kStateCols + lane] = s;
      o += s * qs[d];
    }
    part[warp * kStateCols + lane] = o;
    nq = block_sum(nq, red);                // also orders `part`
    if (warp == 0 && live) {
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) t += part[w * kStateCols + lane];
      p.out[1ll * r * p.ld_out + h * p.vdim_pad + col] = t / (fmaxf(fabsf(nq), expf(-m)) + p.den_eps);
    }
  }
  __syncthreads();
  if (live)
#pragma unroll 4
    for (int d = warp; d < D; d += 8) gS[1ll * d * p.vdim_pad + col] = S[d * kStateCols + lane];
  for (int d = tid; d < D; d += 256) gn[d] = n[d];
  if (tid == 0) *gm = m;
}

constexpr int kChunk = 64;
constexpr int kPStride = kChunk + 8;          // bf16 per row of the decayed scores
constexpr int kVStride = kStateCols + 8;      // bf16 per row of a value tile
constexpr int kRedStride = kStateCols + 1;

template <int NTD>
struct ChunkSmem {
  static constexpr int D = NTD * 32;
  static constexpr int kStride = D + 8;                            // bf16 per row of a q / k tile
  static constexpr int kTile = kChunk * kStride * 2;               // bytes
  static constexpr int kStage = 2 * kTile + kChunk * kVStride * 2;
  static constexpr int kFixed = 2 * kChunk * kPStride * 2 + 2 * kChunk * kVStride * 2 + 4 * kChunk * kRedStride * 4 +
                                D * 4 + 7 * kChunk * 4 + 64;
  static constexpr int kStages = 2 * kStage + kFixed <= 226 * 1024 ? 2 : 1;
  static constexpr int kBytes = kStages * kStage + kFixed;
};

// 256 threads.  In the products over the value columns warp w owns columns 16 (w & 1) .. +16 and the (w >> 1)-th quarter of
// the key dimension, whose slice of the transposed state it keeps in registers; in Q K^T it owns 16 rows x 32 keys.
template <int NTD>
__global__ void __launch_bounds__(256) mlstm_chunk_kernel(ds41_mlstm_args p) {
  using Sm = ChunkSmem<NTD>;
  constexpr int D = Sm::D, DQ = D / 4;
  extern __shared__ __align__(16) uint8_t mc_smem[];
  uint8_t* fixed = mc_smem + Sm::kStages * Sm::kStage;
  __nv_bfloat16* p_hi = reinterpret_cast<__nv_bfloat16*>(fixed);
  __nv_bfloat16* p_lo = p_hi + kChunk * kPStride;
  __nv_bfloat16* w_hi = p_lo + kChunk * kPStride;
  __nv_bfloat16* w_lo = w_hi + kChunk * kVStride;
  float* red = reinterpret_cast<float*>(w_lo + kChunk * kVStride);     // [4][64][33]
  float* nv = red + 4 * kChunk * kRedStride;                           // [D]
  float* g_e = nv + D;                 // F_t - m_t
  float* g_a = g_e + kChunk;           // i_s - F_s
  float* g_m = g_a + kChunk;           // m_t
  float* g_w = g_m + kChunk;           // weight of key s in the state after the chunk
  float* nq = g_w + kChunk;            // n . q_t before the chunk
  float* rs = nq + kChunk;             // [2][64] sums of the decayed scores
  float* carry = rs + 2 * kChunk;      // factor on the state, new m
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int vb = blockIdx.x, h = blockIdx.y;
  const int nt = warp & 1, dq = warp >> 1, g = lane >> 2, q2 = 2 * (lane & 3);
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[0];
  if (slot < 0 || slot >= p.slots) return;
  const bool fresh = p.row_pos[0] == 0;
  const int nb = gridDim.x, col0 = vb * kStateCols;
  const long long head = 1ll * slot * p.heads + h;
  float* gS = p.state_s + head * p.dim_pad * p.vdim_pad;
  float* gn = p.state_n + (head * nb + vb) * p.dim_pad;
  float* gm = p.state_m + head * nb + vb;

  // transposed state: tile j holds columns d = dq DQ + 8 j + q2 + {0, 1} of rows nt 16 + g and + 8
  float st[NTD][4];
#pragma unroll
  for (int j = 0; j < NTD; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = dq * DQ + 8 * j + q2 + (e & 1), c = col0 + nt * 16 + g + (e >> 1) * 8;
      st[j][e] = !fresh && d < p.dim_pad && c < p.vdim_pad ? gS[1ll * d * p.vdim_pad + c] : 0.f;
    }
  for (int d = tid; d < D; d += 256) nv[d] = !fresh && d < p.dim_pad ? gn[d] : 0.f;
  float m0 = fresh ? 0.f : *gm;

  const __nv_bfloat16* gq = static_cast<const __nv_bfloat16*>(p.q.data) + p.q.col + h * p.dim_pad;
  const __nv_bfloat16* gk = static_cast<const __nv_bfloat16*>(p.k.data) + p.k.col + h * p.dim_pad;
  const __nv_bfloat16* gv = static_cast<const __nv_bfloat16*>(p.v.data) + p.v.col + h * p.vdim_pad + col0;
  const int n_chunks = (p.rows + kChunk - 1) / kChunk;
  auto load = [&](int c, int stage) {
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(mc_smem + stage * Sm::kStage);
    __nv_bfloat16* sk = sq + kChunk * Sm::kStride;
    __nv_bfloat16* sv = sk + kChunk * Sm::kStride;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    for (int i = tid; i < kChunk * (D / 8); i += 256) {
      const int t = i / (D / 8), d = (i - t * (D / 8)) * 8, r = c * kChunk + t;
      if (r < p.rows && d < p.dim_pad) {
        cp_async_16(sq + t * Sm::kStride + d, gq + 1ll * r * p.q.ld + d);
        cp_async_16(sk + t * Sm::kStride + d, gk + 1ll * r * p.k.ld + d);
      } else {
        *reinterpret_cast<uint4*>(sq + t * Sm::kStride + d) = zero;
        *reinterpret_cast<uint4*>(sk + t * Sm::kStride + d) = zero;
      }
    }
    {
      const int t = tid >> 2, d = (tid & 3) * 8, r = c * kChunk + t;
      if (r < p.rows && col0 + d < p.vdim_pad) cp_async_16(sv + t * kVStride + d, gv + 1ll * r * p.v.ld + d);
      else *reinterpret_cast<uint4*>(sv + t * kVStride + d) = zero;
    }
    cp_async_commit();
  };
  // raw gates of the next chunk travel in registers of warp 0 (rows 2 lane and 2 lane + 1)
  float raw_i[2], raw_f[2];
  auto load_gates = [&](int c) {
    if (warp == 0)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int r = c * kChunk + 2 * lane + u;
        raw_i[u] = r < p.rows ? proj_at(p.gate_i, r, h) + p.bias_i[h] : 0.f;
        raw_f[u] = r < p.rows ? proj_at(p.gate_f, r, h) + p.bias_f[h] : 0.f;
      }
  };
  load(0, 0);
  load_gates(0);
  for (int c = 0; c < n_chunks; ++c) {
    const int stage = Sm::kStages == 2 ? (c & 1) : 0;
    if (Sm::kStages == 2 && c + 1 < n_chunks) {
      load(c + 1, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    const __nv_bfloat16* sq = reinterpret_cast<const __nv_bfloat16*>(mc_smem + stage * Sm::kStage);
    const __nv_bfloat16* sk = sq + kChunk * Sm::kStride;
    const __nv_bfloat16* sv = sk + kChunk * Sm::kStride;
    if (warp == 0) {
      float gi[2], gf[2];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const bool live = c * kChunk + 2 * lane + u < p.rows;
        gi[u] = live ? p.gate_cap * tanhf(raw_i[u] / p.gate_cap) : -INFINITY;
        gf[u] = live ? log_sigmoid_f32(p.gate_cap * tanhf(raw_f[u] / p.gate_cap)) : 0.f;
      }
      float F1 = gf[0] + gf[1];                       // running sum up to row 2 lane + 1
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, F1, o);
        if (lane >= o) F1 += x;
      }
      float F0 = __shfl_up_sync(0xffffffffu, F1, 1);
      F0 = (lane == 0 ? 0.f : F0) + gf[0];
      const float a0 = gi[0] - F0, a1 = gi[1] - F1;
      float top1 = fmaxf(a0, a1);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, top1, o);
        if (lane >= o) top1 = fmaxf(top1, x);
      }
      float top0 = __shfl_up_sync(0xffffffffu, top1, 1);
      top0 = fmaxf(lane == 0 ? m0 : fmaxf(top0, m0), a0);
      top1 = fmaxf(top1, m0);
      const float F_end = __shfl_sync(0xffffffffu, F1, 31), top_end = __shfl_sync(0xffffffffu, top1, 31);
      g_e[2 * lane] = -top0;                          // F_t - m_t
      g_e[2 * lane + 1] = -top1;
      g_a[2 * lane] = a0;
      g_a[2 * lane + 1] = a1;
      g_m[2 * lane] = F0 + top0;
      g_m[2 * lane + 1] = F1 + top1;
      g_w[2 * lane] = expf(a0 - top_end);
      g_w[2 * lane + 1] = expf(a1 - top_end);
      if (lane == 0) {
        carry[0] = expf(m0 - top_end);
        carry[1] = F_end + top_end;
      }
      if (c + 1 < n_chunks) load_gates(c + 1);
    }
    __syncthreads();

    // ---- decayed scores: 16 rows x 32 keys per warp
    {
      const int tm = warp >> 1, sh = warp & 1;
      float acc[4][4] = {};
      if (sh * 32 <= tm * 16 + 15) {
        const __nv_bfloat16* arow = sq + (tm * 16 + (lane & 15)) * Sm::kStride + (lane >> 4) * 8;
        const __nv_bfloat16* brow = sk + (sh * 32 + (lane & 7) + (lane >> 4) * 8) * Sm::kStride + ((lane >> 3) & 1) * 8;
#pragma unroll 4
        for (int k = 0; k < D; k += 16) {
          uint32_t a[4], b[8];
          ldmatrix_x4(a[0], a[1], a[2], a[3], arow + k);
          ldmatrix_x4(b[0], b[1], b[2], b[3], brow + k);
          ldmatrix_x4(b[4], b[5], b[6], b[7], brow + 16 * Sm::kStride + k);
#pragma unroll
          for (int j = 0; j < 4; ++j) mma_bf16_16816(acc[j], a, b[2 * j], b[2 * j + 1]);
        }
      }
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int t = tm * 16 + g + 8 * u;
        const float e = g_e[t];
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int s = sh * 32 + 8 * j + q2;
          const float x = s <= t ? acc[j][2 * u] * p.q_scale * expf(e + g_a[s]) : 0.f;
          const float y = s + 1 <= t ? acc[j][2 * u + 1] * p.q_scale * expf(e + g_a[s + 1]) : 0.f;
          sum += x + y;
          const uint32_t hi = pack_bf16(x, y);
          *reinterpret_cast<uint32_t*>(p_hi + t * kPStride + s) = hi;
          *reinterpret_cast<uint32_t*>(p_lo + t * kPStride + s) = pack_bf16_rest(x, y, hi);
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if ((lane & 3) == 0) rs[sh * kChunk + t] = sum;
      }
    }
    // ---- decayed values, n . q
    {
      const int s = tid >> 2, d = (tid & 3) * 8;
      const float w = g_w[s];
#pragma unroll
      for (int i = 0; i < 8; i += 2) {
        const float x = __bfloat162float(sv[s * kVStride + d + i]) * w, y = __bfloat162float(sv[s * kVStride + d + i + 1]) * w;
        const uint32_t hi = pack_bf16(x, y);
        *reinterpret_cast<uint32_t*>(w_hi + s * kVStride + d + i) = hi;
        *reinterpret_cast<uint32_t*>(w_lo + s * kVStride + d + i) = pack_bf16_rest(x, y, hi);
      }
#pragma unroll 2
      for (int t = warp * 8; t < warp * 8 + 8; ++t) {
        float x = 0.f;
        for (int i = 2 * lane; i < D; i += 64) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sq + t * Sm::kStride + i));
          x += nv[i] * f.x + nv[i + 1] * f.y;
        }
        x = warp_sum(x);
        if (lane == 0) nq[t] = x * p.q_scale;
      }
    }
    __syncthreads();

    // ---- output, transposed: 16 value columns x 64 rows per warp, this warp's quarter of d and of the keys
    {
      float o[8][4] = {};
      const __nv_bfloat16* brow = sq + ((lane & 7) + (lane >> 4) * 8) * Sm::kStride + dq * DQ + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int k = 0; k < NTD / 2; ++k) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = st[2 * k + (e >> 1)][2 * (e & 1)], y = st[2 * k + (e >> 1)][2 * (e & 1) + 1];
          hi[e] = pack_bf16(x, y);
          lo[e] = pack_bf16_rest(x, y, hi[e]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t b[4];
          ldmatrix_x4(b[0], b[1], b[2], b[3], brow + 16 * j * Sm::kStride + 16 * k);
          mma_bf16_16816(o[2 * j], hi, b[0], b[1]);
          mma_bf16_16816(o[2 * j + 1], hi, b[2], b[3]);
          mma_bf16_16816(o[2 * j], lo, b[0], b[1]);
          mma_bf16_16816(o[2 * j + 1], lo, b[2], b[3]);
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int t = 8 * j + q2;
        const float x = p.q_scale * expf(g_e[t] + m0), y = p.q_scale * expf(g_e[t + 1] + m0);
        o[j][0] *= x;
        o[j][1] *= y;
        o[j][2] *= x;
        o[j][3] *= y;
      }
      uint32_t a[4];
      ldmatrix_x4_trans(a[0], a[1], a[2], a[3],
                        sv + (dq * 16 + (lane & 7) + (lane >> 4) * 8) * kVStride + nt * 16 + ((lane >> 3) & 1) * 8);
      const int prow = ((lane & 7) + (lane >> 4) * 8) * kPStride + dq * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        uint32_t b[4];
        ldmatrix_x4(b[0], b[1], b[2], b[3], p_hi + prow + 16 * j * kPStride);
        mma_bf16_16816(o[2 * j], a, b[0], b[1]);
        mma_bf16_16816(o[2 * j + 1], a, b[2], b[3]);
        ldmatrix_x4(b[0], b[1], b[2], b[3], p_lo + prow + 16 * j * kPStride);
        mma_bf16_16816(o[2 * j], a, b[0], b[1]);
        mma_bf16_16816(o[2 * j + 1], a, b[2], b[3]);
      }
      float* dst = red + dq * kChunk * kRedStride + nt * 16 + g;
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) dst[(8 * j + q2 + (e & 1)) * kRedStride + (e >> 1) * 8] = o[j][e];
    }
    // ---- state after the chunk
    {
      const float keep = carry[0];
#pragma unroll
      for (int j = 0; j < NTD; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[j][e] *= keep;
      const int arow = ((lane & 7) + (lane >> 4) * 8) * kVStride + nt * 16 + ((lane >> 3) & 1) * 8;
      const __nv_bfloat16* brow = sk + (lane & 15) * Sm::kStride + dq * DQ + (lane >> 4) * 8;
#pragma unroll
      for (int k = 0; k < kChunk; k += 16) {
        uint32_t hi[4], lo[4];
        ldmatrix_x4_trans(hi[0], hi[1], hi[2], hi[3], w_hi + arow + k * kVStride);
        ldmatrix_x4_trans(lo[0], lo[1], lo[2], lo[3], w_lo + arow + k * kVStride);
#pragma unroll
        for (int j = 0; j < NTD / 2; ++j) {
          uint32_t b[4];
          ldmatrix_x4_trans(b[0], b[1], b[2], b[3], brow + k * Sm::kStride + 16 * j);
          mma_bf16_16816(st[2 * j], hi, b[0], b[1]);
          mma_bf16_16816(st[2 * j + 1], hi, b[2], b[3]);
          mma_bf16_16816(st[2 * j], lo, b[0], b[1]);
          mma_bf16_16816(st[2 * j + 1], lo, b[2], b[3]);
        }
      }
      for (int d = 2 * tid; d < D; d += 512) {
        float x = nv[d] * keep, y = nv[d + 1] * keep;
#pragma unroll 8
        for (int s = 0; s < kChunk; ++s) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sk + s * Sm::kStride + d));
          x += g_w[s] * f.x;
          y += g_w[s] * f.y;
        }
        nv[d] = x;
        nv[d + 1] = y;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = warp * 8 + i, r = c * kChunk + t;
      if (r < p.rows && col0 + lane < p.vdim_pad) {
        float x = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) x += red[(w * kChunk + t) * kRedStride + lane];
        const float dot = expf(g_e[t] + m0) * nq[t] + rs[t] + rs[kChunk + t];
        p.out[1ll * r * p.ld_out + h * p.vdim_pad + col0 + lane] = x / (fmaxf(fabsf(dot), expf(-g_m[t])) + p.den_eps);
      }
    }
    m0 = carry[1];
    __syncthreads();
    if (Sm::kStages == 1 && c + 1 < n_chunks) load(c + 1, 0);
  }
#pragma unroll
  for (int j = 0; j < NTD; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = dq * DQ + 8 * j + q2 + (e & 1), cc = col0 + nt * 16 + g + (e >> 1) * 8;
      if (d < p.dim_pad && cc < p.vdim_pad) gS[1ll * d * p.vdim_pad + cc] = st[j][e];
    }
  for (int d = tid; d < p.dim_pad; d += 256) gn[d] = nv[d];
  if (tid == 0) *gm = m0;
}

template <int NTD>
static int launch_chunk(const ds41_mlstm_args& a, cudaStream_t st) {
  static bool ready = false;
  if (!ready) {
    const cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_kernel<NTD>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               ChunkSmem<NTD>::kBytes);
    if (e != cudaSuccess) return e;
    ready = true;
  }
  const dim3 grid((a.vdim_pad + kStateCols - 1) / kStateCols, a.heads);
  return launch_pdl(mlstm_chunk_kernel<NTD>, grid, dim3(256), ChunkSmem<NTD>::kBytes, st, a);
}

}  // namespace ds41

using namespace ds41;

static bool proj_ok(const ds41_proj& p) {
  return p.data != nullptr && p.ld > 0 && p.splits >= 1 && p.col >= 0 && (p.splits == 1 || (p.plane > 0 && !p.bf16));
}

static bool mlstm_args_ok(const ds41_mlstm_args* a) {
  return a != nullptr && a->rows > 0 && a->rows <= 65535 && a->heads > 0 && a->heads <= 65535 && a->dim_pad > 0 &&
         a->vdim_pad > 0 && a->slots > 0 && a->gate_cap > 0.f && proj_ok(a->q) && proj_ok(a->k) && proj_ok(a->v) &&
         proj_ok(a->gate_i) && proj_ok(a->gate_f) && a->bias_i != nullptr && a->bias_f != nullptr &&
         a->row_pos != nullptr && a->row_slot != nullptr && a->state_s != nullptr && a->state_n != nullptr &&
         a->state_m != nullptr && a->out != nullptr && a->ld_out >= a->heads * a->vdim_pad;
}

extern "C" int ds41_mlstm_step(const ds41_mlstm_args* a, void* stream) {
  if (!mlstm_args_ok(a)) return cudaErrorInvalidValue;
  const size_t smem = (1ull * a->dim_pad * (kStateCols + 3) + kStateCols * 9) * sizeof(float);
  static size_t allowed = 48 * 1024 - 512;
  if (smem > allowed) {
    if (smem > 226 * 1024) return cudaErrorInvalidValue;
    const cudaError_t e = cudaFuncSetAttribute(mlstm_step_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem));
    if (e != cudaSuccess) return e;
    allowed = smem;
  }
  const dim3 grid((a->vdim_pad + kStateCols - 1) / kStateCols, a->heads, a->rows);
  return launch_pdl(mlstm_step_kernel, grid, dim3(256), smem, static_cast<cudaStream_t>(stream), *a);
}

extern "C" int ds41_mlstm_chunk(const ds41_mlstm_args* a, void* stream) {
  if (!mlstm_args_ok(a)) return cudaErrorInvalidValue;
  for (const ds41_proj* x : {&a->q, &a->k, &a->v})
    if (!x->bf16 || (x->ld & 7) || (x->col & 7) || (reinterpret_cast<uintptr_t>(x->data) & 15)) return cudaErrorInvalidValue;
  if ((a->dim_pad & 15) || (a->vdim_pad & 15)) return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->dim_pad <= 64) return launch_chunk<2>(*a, st);
  if (a->dim_pad <= 128) return launch_chunk<4>(*a, st);
  if (a->dim_pad <= 192) return launch_chunk<6>(*a, st);
  if (a->dim_pad <= 256) return launch_chunk<8>(*a, st);
  if (a->dim_pad <= 384) return launch_chunk<12>(*a, st);
  if (a->dim_pad <= 512) return launch_chunk<16>(*a, st);
  return cudaErrorInvalidValue;
}
