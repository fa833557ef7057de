// Matrix-memory recurrence (mLSTM of xLSTM) with a running maximum.
//
// Per head the state is a dim x vdim matrix S, a vector n and a scalar m, all fp32, one set per request slot:
//   m' = max(f + m, i);  S' = exp(f + m - m') S + exp(i - m') k v^T;  n' the same with k alone
//   o  = S'^T q / (max(|n' . q|, exp(-m')) + den_eps)
// A block owns 32 value columns of one head.  Every column block carries its own copy of n and m, so blocks never wait for
// one another.  A request's state starts at zero where its rows start at position 0.
//
//  mlstm_step : one block walks the adjacent rows of a request token by token (decode rows, 32-bit passes), the state in
//               registers, or in shared memory where it is too large for them
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

// The same walk with the state in registers: thread (warp, lane) holds rows d = 32 i + 4 warp + lane / 8 and the four columns
// 4 (lane % 8), i < NR.
template <int NR>
__global__ void __launch_bounds__(256) mlstm_walk_kernel(ds41_mlstm_args p) {
  constexpr int D = NR * 32;
  __shared__ float qs[D], ks[D];
  __shared__ float n[D];
  __shared__ __align__(16) float part[8][kStateCols];
  __shared__ __align__(16) float vs[kStateCols];
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
  const int nb = gridDim.x, col0 = vb * kStateCols, c4 = col0 + 4 * (lane & 7), d0 = 4 * warp + (lane >> 3);
  const bool live = c4 < p.vdim_pad;                 // vdim_pad is a multiple of 4
  const bool fresh = p.row_pos[r] == 0;
  const long long head = 1ll * slot * p.heads + h;
  float* gS = p.state_s + head * p.dim_pad * p.vdim_pad + c4;
  float* gn = p.state_n + (head * nb + vb) * p.dim_pad;
  float* gm = p.state_m + head * nb + vb;
  float4 st[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = 32 * i + d0;
    st[i] = !fresh && live && d < p.dim_pad ? *reinterpret_cast<const float4*>(gS + 1ll * d * p.vdim_pad)
                                            : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int d = tid; d < D; d += 256) n[d] = !fresh && d < p.dim_pad ? gn[d] : 0.f;
  float m = fresh ? 0.f : *gm;
  for (; r < p.rows && p.row_slot[r] == slot; ++r) {
    __syncthreads();
    for (int d = tid; d < D; d += 256) {
      const bool in = d < p.dim_pad;
      qs[d] = in ? proj_at(p.q, r, h * p.dim_pad + d) * p.q_scale : 0.f;
      ks[d] = in ? proj_at(p.k, r, h * p.dim_pad + d) : 0.f;
    }
    if (tid < kStateCols) vs[tid] = col0 + tid < p.vdim_pad ? proj_at(p.v, r, h * p.vdim_pad + col0 + tid) : 0.f;
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
    float4 v = *reinterpret_cast<const float4*>(vs + 4 * (lane & 7));
    v.x *= add;
    v.y *= add;
    v.z *= add;
    v.w *= add;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const float k = ks[32 * i + d0], q = qs[32 * i + d0];
      st[i].x = keep * st[i].x + k * v.x;
      st[i].y = keep * st[i].y + k * v.y;
      st[i].z = keep * st[i].z + k * v.z;
      st[i].w = keep * st[i].w + k * v.w;
      o.x += st[i].x * q;
      o.y += st[i].y * q;
      o.z += st[i].z * q;
      o.w += st[i].w * q;
    }
#pragma unroll
    for (int x = 8; x <= 16; x <<= 1) {
      o.x += __shfl_xor_sync(0xffffffffu, o.x, x);
      o.y += __shfl_xor_sync(0xffffffffu, o.y, x);
      o.z += __shfl_xor_sync(0xffffffffu, o.z, x);
      o.w += __shfl_xor_sync(0xffffffffu, o.w, x);
    }
    if (lane < 8) *reinterpret_cast<float4*>(&part[warp][4 * lane]) = o;
    nq = block_sum(nq, red);                // also orders `part`
    if (warp == 0 && col0 + lane < p.vdim_pad) {
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) t += part[w][lane];
      p.out[1ll * r * p.ld_out + h * p.vdim_pad + col0 + lane] = t / (fmaxf(fabsf(nq), expf(-m)) + p.den_eps);
    }
  }
  if (live)
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = 32 * i + d0;
      if (d < p.dim_pad) *reinterpret_cast<float4*>(gS + 1ll * d * p.vdim_pad) = st[i];
    }
  for (int d = tid; d < p.dim_pad; d += 256) gn[d] = n[d];
  if (tid == 0) *gm = m;
}

constexpr int kChunk = 64;
constexpr int kPStride = kChunk + 8;          // bf16 per row of the decayed scores
constexpr int kVStride = kStateCols + 8;      // bf16 per row of a value tile
constexpr int kRedStride = kStateCols + 1;
// What the gates of one (chunk, head) come to, as the chunk kernel wants it: five rows of 64 values and four scalars.
//   [0] e_t = (F_t - m_t) log2(e)   [1] a_s = (i_s - F_s) log2(e)   [2] weight of key s in the state after the chunk
//   [3] q_scale exp(F_t + m0 - m_t)  [4] exp(-m_t)                   scalars: factor on the old state, m after the chunk
constexpr int kGateFloats = 5 * kChunk + 4;

// One block per head: the gates of every chunk, then the maxima from chunk to chunk.
__global__ void __launch_bounds__(1024) mlstm_gates_kernel(ds41_mlstm_args p) {
  extern __shared__ float mg_smem[];          // [n_chunks][3]: F at the end, largest i - F, m before the chunk
  const int h = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[0];
  if (slot < 0 || slot >= p.slots) return;
  const int n_chunks = (p.rows + kChunk - 1) / kChunk;
  constexpr float kLog2e = 1.4426950408889634f;
  float F[2], a[2], top[2];
  auto scan = [&](int c) {
    float gi[2], gf[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int r = c * kChunk + 2 * lane + u;
      gi[u] = -INFINITY;
      gf[u] = 0.f;
      if (r < p.rows) {
        const GateValues g = mlstm_gates(p, r, h);
        gi[u] = g.i;
        gf[u] = g.f;
      }
    }
    F[1] = gf[0] + gf[1];                     // running sum up to row 2 lane + 1
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, F[1], o);
      if (lane >= o) F[1] += x;
    }
    F[0] = __shfl_up_sync(0xffffffffu, F[1], 1);
    F[0] = (lane == 0 ? 0.f : F[0]) + gf[0];
    a[0] = gi[0] - F[0];
    a[1] = gi[1] - F[1];
    top[1] = fmaxf(a[0], a[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, top[1], o);
      if (lane >= o) top[1] = fmaxf(top[1], x);
    }
    top[0] = __shfl_up_sync(0xffffffffu, top[1], 1);
    top[0] = fmaxf(lane == 0 ? -INFINITY : top[0], a[0]);
  };
  for (int c = warp; c < n_chunks; c += 32) {
    scan(c);
    if (lane == 31) {
      mg_smem[3 * c] = F[1];
      mg_smem[3 * c + 1] = top[1];
    }
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    const int nb = (p.vdim_pad + kStateCols - 1) / kStateCols;
    float m = p.row_pos[0] == 0 ? 0.f : p.state_m[(1ll * slot * p.heads + h) * nb];
    for (int c = 0; c < n_chunks; ++c) {
      mg_smem[3 * c + 2] = m;
      m = mg_smem[3 * c] + fmaxf(m, mg_smem[3 * c + 1]);
    }
  }
  __syncthreads();
  for (int c = warp; c < n_chunks; c += 32) {
    if (n_chunks > 32) scan(c);               // one chunk per warp keeps its values
    const float F_end = mg_smem[3 * c], m0 = mg_smem[3 * c + 2], end = fmaxf(m0, mg_smem[3 * c + 1]);
    float* out = p.work + (1ll * c * p.heads + h) * kGateFloats;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int t = 2 * lane + u;
      const float mx = fmaxf(top[u], m0);     // m_t - F_t
      out[t] = -mx * kLog2e;
      out[kChunk + t] = a[u] * kLog2e;
      out[2 * kChunk + t] = expf(a[u] - end);
      out[3 * kChunk + t] = p.q_scale * expf(m0 - mx);
      out[4 * kChunk + t] = expf(-(F[u] + mx));
    }
    if (lane == 0) {
      out[5 * kChunk] = expf(m0 - end);
      out[5 * kChunk + 1] = F_end + end;
    }
  }
}

template <int NTD>
struct ChunkSmem {
  static constexpr int D = NTD * 32;
  static constexpr int kStride = D + 8;                            // bf16 per row of a q / k tile
  static constexpr int kTile = kChunk * kStride * 2;               // bytes
  static constexpr int kStage = 2 * kTile + kChunk * kVStride * 2 + kGateFloats * 4;
  static constexpr int kFixed = 2 * kChunk * kPStride * 2 + 2 * kChunk * kVStride * 2 + 8 * kStride * 2 +
                                4 * kChunk * kRedStride * 4 + D * 4 + 4 * kChunk * 4;
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
  __nv_bfloat16* n_rows = w_lo + kChunk * kVStride;                    // [8][D + 8]: n as high and low parts, zero rows
  float* red = reinterpret_cast<float*>(n_rows + 8 * Sm::kStride);     // [4][64][33]
  float* nv = red + 4 * kChunk * kRedStride;                           // [D]
  float* nq = nv + D;                  // n . q_t before the chunk
  float* rs = nq + kChunk;             // [2][64] sums of the decayed scores
  float* inv = rs + 2 * kChunk;        // 1 / denominator
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

  const __nv_bfloat16* gq = static_cast<const __nv_bfloat16*>(p.q.data) + p.q.col + h * p.dim_pad;
  const __nv_bfloat16* gk = static_cast<const __nv_bfloat16*>(p.k.data) + p.k.col + h * p.dim_pad;
  const __nv_bfloat16* gv = static_cast<const __nv_bfloat16*>(p.v.data) + p.v.col + h * p.vdim_pad + col0;
  const int n_chunks = (p.rows + kChunk - 1) / kChunk;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  auto load = [&](int c, int stage) {
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(mc_smem + stage * Sm::kStage);
    __nv_bfloat16* sk = sq + kChunk * Sm::kStride;
    __nv_bfloat16* sv = sk + kChunk * Sm::kStride;
    const int live = p.rows - c * kChunk;
    constexpr int kPer = D / 8;                       // 16-byte pieces of a row
    constexpr int kRows = kPer <= 256 ? 256 / kPer : 1;
    if (kPer * kRows == 256 || tid < kPer * kRows) {
      const int d = (tid % kPer) * 8;
      const __nv_bfloat16* q = gq + (1ll * c * kChunk + tid / kPer) * p.q.ld + d;
      const __nv_bfloat16* k = gk + (1ll * c * kChunk + tid / kPer) * p.k.ld + d;
      for (int t = tid / kPer; t < kChunk; t += kRows, q += 1ll * kRows * p.q.ld, k += 1ll * kRows * p.k.ld) {
        if (t < live && d < p.dim_pad) {
          cp_async_16(sq + t * Sm::kStride + d, q);
          cp_async_16(sk + t * Sm::kStride + d, k);
        } else {
          *reinterpret_cast<uint4*>(sq + t * Sm::kStride + d) = zero;
          *reinterpret_cast<uint4*>(sk + t * Sm::kStride + d) = zero;
        }
      }
    }
    {
      const int t = tid >> 2, d = (tid & 3) * 8;
      if (t < live && col0 + d < p.vdim_pad) cp_async_16(sv + t * kVStride + d, gv + (1ll * c * kChunk + t) * p.v.ld + d);
      else *reinterpret_cast<uint4*>(sv + t * kVStride + d) = zero;
    }
    if (tid < kGateFloats / 4)
      cp_async_16(reinterpret_cast<float*>(sv + kChunk * kVStride) + 4 * tid,
                  p.work + (1ll * c * p.heads + h) * kGateFloats + 4 * tid);
    cp_async_commit();
  };
  load(0, 0);
  // transposed state: tile j holds columns d = dq DQ + 8 j + q2 + {0, 1} of rows nt 16 + g and + 8
  float st[NTD][4];
#pragma unroll
  for (int j = 0; j < NTD; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = dq * DQ + 8 * j + q2 + (e & 1), c = col0 + nt * 16 + g + (e >> 1) * 8;
      st[j][e] = !fresh && d < p.dim_pad && c < p.vdim_pad ? gS[1ll * d * p.vdim_pad + c] : 0.f;
    }
  for (int i = tid; i < 8 * Sm::kStride; i += 256) n_rows[i] = __float2bfloat16_rn(0.f);
  __syncthreads();
  for (int d = tid; d < D; d += 256) {
    const float x = !fresh && d < p.dim_pad ? gn[d] : 0.f;
    const __nv_bfloat16 hi = __float2bfloat16_rn(x);
    nv[d] = x;
    n_rows[d] = hi;
    n_rows[Sm::kStride + d] = __float2bfloat16_rn(x - __bfloat162float(hi));
  }
  float m_end = 0.f;
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
    const float* gates = reinterpret_cast<const float*>(sv + kChunk * kVStride);
    __syncthreads();

    // ---- decayed scores, 16 rows x 32 keys per warp; the warps of the first keys also take n . q_t
    {
      const int tm = warp >> 1, sh = warp & 1;
      float acc[4][4] = {}, na[4] = {};
      const __nv_bfloat16* arow = sq + (tm * 16 + (lane & 15)) * Sm::kStride + (lane >> 4) * 8;
      const __nv_bfloat16* brow = sk + (sh * 32 + (lane & 7) + (lane >> 4) * 8) * Sm::kStride + ((lane >> 3) & 1) * 8;
      const __nv_bfloat16* nrow = n_rows + (lane & 7) * Sm::kStride + (lane >> 3) * 8;
      if (sh * 32 <= tm * 16 + 15) {
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
      if (sh == 0) {
#pragma unroll 2
        for (int k = 0; k < D; k += 32) {
          uint32_t a[4], b[4];
          ldmatrix_x4(b[0], b[1], b[2], b[3], nrow + k);
          ldmatrix_x4(a[0], a[1], a[2], a[3], arow + k);
          mma_bf16_16816(na, a, b[0], b[1]);
          ldmatrix_x4(a[0], a[1], a[2], a[3], arow + k + 16);
          mma_bf16_16816(na, a, b[2], b[3]);
        }
        if ((lane & 3) == 0) {
          nq[tm * 16 + g] = na[0] + na[1];
          nq[tm * 16 + g + 8] = na[2] + na[3];
        }
      }
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int t = tm * 16 + g + 8 * u;
        const float e = gates[t];
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int s = sh * 32 + 8 * j + q2;
          const float2 as = *reinterpret_cast<const float2*>(gates + kChunk + s);
          const float x = s <= t ? acc[j][2 * u] * p.q_scale * ex2_approx(e + as.x) : 0.f;
          const float y = s + 1 <= t ? acc[j][2 * u + 1] * p.q_scale * ex2_approx(e + as.y) : 0.f;
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
    // ---- decayed values
    {
      const int s = tid >> 2, d = (tid & 3) * 8;
      const float w = gates[2 * kChunk + s];
      const uint4 v4 = *reinterpret_cast<const uint4*>(sv + s * kVStride + d);
      const uint32_t v[4] = {v4.x, v4.y, v4.z, v4.w};
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float x = __uint_as_float(v[i] << 16) * w, y = __uint_as_float(v[i] & 0xffff0000u) * w;
        hi[i] = pack_bf16(x, y);
        lo[i] = pack_bf16_rest(x, y, hi[i]);
      }
      *reinterpret_cast<uint4*>(w_hi + s * kVStride + d) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(w_lo + s * kVStride + d) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
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
        const float2 f = *reinterpret_cast<const float2*>(gates + 3 * kChunk + 8 * j + q2);
        o[j][0] *= f.x;
        o[j][1] *= f.y;
        o[j][2] *= f.x;
        o[j][3] *= f.y;
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
    if (tid < kChunk)
      inv[tid] = 1.0f / (fmaxf(fabsf(gates[3 * kChunk + tid] * nq[tid] + rs[tid] + rs[kChunk + tid]), gates[4 * kChunk + tid]) +
                         p.den_eps);
    // ---- state after the chunk
    {
      const float keep = gates[5 * kChunk];
      m_end = gates[5 * kChunk + 1];
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
      // n: one row of weights (high parts in row 0, low parts in row 1 of the left operand) times the keys; the two warps
      // of a quarter take half of its columns each
      uint32_t wf[4][2];
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float2 w = *reinterpret_cast<const float2*>(gates + 2 * kChunk + 16 * k + 8 * e + q2);
          const uint32_t hi = pack_bf16(w.x, w.y);
          wf[k][e] = g == 0 ? hi : (g == 1 ? pack_bf16_rest(w.x, w.y, hi) : 0u);
        }
#pragma unroll
      for (int j = nt; j < NTD / 2; j += 2) {
        float x[4] = {}, y[4] = {};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          uint32_t b[4];
          const uint32_t a[4] = {wf[k][0], 0u, wf[k][1], 0u};
          ldmatrix_x4_trans(b[0], b[1], b[2], b[3], brow + 16 * k * Sm::kStride + 16 * j);
          mma_bf16_16816(x, a, b[0], b[1]);
          mma_bf16_16816(y, a, b[2], b[3]);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          x[e] += __shfl_down_sync(0xffffffffu, x[e], 4);       // rows 0 and 1 of a column meet in row 0's lanes
          y[e] += __shfl_down_sync(0xffffffffu, y[e], 4);
        }
        if (g == 0) {
          const int d = dq * DQ + 16 * j + q2;
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int at = d + 8 * u;
            const float n0 = nv[at] * keep + (u == 0 ? x[0] : y[0]), n1 = nv[at + 1] * keep + (u == 0 ? x[1] : y[1]);
            nv[at] = n0;
            nv[at + 1] = n1;
            const uint32_t hi = pack_bf16(n0, n1);
            *reinterpret_cast<uint32_t*>(n_rows + at) = hi;
            *reinterpret_cast<uint32_t*>(n_rows + Sm::kStride + at) = pack_bf16_rest(n0, n1, hi);
          }
        }
      }
    }
    __syncthreads();
    if (col0 + lane < p.vdim_pad) {
      const int t0 = warp * 8, live = min(8, p.rows - c * kChunk - t0);
      float* dst = p.out + (1ll * c * kChunk + t0) * p.ld_out + h * p.vdim_pad + col0 + lane;
      const float* src = red + t0 * kRedStride + lane;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float x = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) x += src[(w * kChunk + i) * kRedStride];
        if (i < live) dst[1ll * i * p.ld_out] = x * inv[t0 + i];
      }
    }
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
  if (tid == 0) p.state_m[head * nb + vb] = m_end;
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
  const size_t gate_smem = 3ull * ((a.rows + kChunk - 1) / kChunk) * sizeof(float);
  if (gate_smem > 48 * 1024) return cudaErrorInvalidValue;
  const cudaError_t e = launch_pdl(mlstm_gates_kernel, dim3(a.heads), dim3(1024), gate_smem, st, a);
  if (e != cudaSuccess) return e;
  const dim3 grid((a.vdim_pad + kStateCols - 1) / kStateCols, a.heads);
  return launch_pdl(mlstm_chunk_kernel<NTD>, grid, dim3(256), ChunkSmem<NTD>::kBytes, st, a);
}

}  // namespace ds41

using namespace ds41;

static bool mlstm_args_ok(const ds41_mlstm_args* a) {
  return a != nullptr && a->rows > 0 && a->rows <= 65535 && a->heads > 0 && a->heads <= 65535 && a->dim_pad > 0 &&
         a->vdim_pad > 0 && a->slots > 0 && a->gate_cap > 0.f && proj_ok(a->q) && proj_ok(a->k) && proj_ok(a->v) &&
         proj_ok(a->gate_i) && proj_ok(a->gate_f) && a->bias_i != nullptr && a->bias_f != nullptr &&
         a->row_pos != nullptr && a->row_slot != nullptr && a->state_s != nullptr && a->state_n != nullptr &&
         a->state_m != nullptr && a->out != nullptr && a->ld_out >= a->heads * a->vdim_pad;
}

extern "C" int ds41_mlstm_step(const ds41_mlstm_args* a, void* stream) {
  if (!mlstm_args_ok(a)) return cudaErrorInvalidValue;
  if (!(a->vdim_pad & 3) && a->dim_pad <= 512 && !(reinterpret_cast<uintptr_t>(a->state_s) & 15)) {
    const dim3 grid((a->vdim_pad + kStateCols - 1) / kStateCols, a->heads, a->rows);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a->dim_pad <= 32) return launch_pdl(mlstm_walk_kernel<1>, grid, dim3(256), 0, st, *a);
    if (a->dim_pad <= 64) return launch_pdl(mlstm_walk_kernel<2>, grid, dim3(256), 0, st, *a);
    if (a->dim_pad <= 128) return launch_pdl(mlstm_walk_kernel<4>, grid, dim3(256), 0, st, *a);
    if (a->dim_pad <= 256) return launch_pdl(mlstm_walk_kernel<8>, grid, dim3(256), 0, st, *a);
    return launch_pdl(mlstm_walk_kernel<16>, grid, dim3(256), 0, st, *a);
  }
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
  if ((a->dim_pad & 15) || (a->vdim_pad & 15) || a->work == nullptr || (reinterpret_cast<uintptr_t>(a->work) & 15)) return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->dim_pad <= 64) return launch_chunk<2>(*a, st);
  if (a->dim_pad <= 128) return launch_chunk<4>(*a, st);
  if (a->dim_pad <= 192) return launch_chunk<6>(*a, st);
  if (a->dim_pad <= 256) return launch_chunk<8>(*a, st);
  if (a->dim_pad <= 384) return launch_chunk<12>(*a, st);
  if (a->dim_pad <= 512) return launch_chunk<16>(*a, st);
  return cudaErrorInvalidValue;
}

extern "C" long long ds41_mlstm_chunk_work(int rows, int heads) {
  return rows <= 0 || heads <= 0 ? 0 : 4ll * kGateFloats * heads * ((rows + kChunk - 1) / kChunk);
}
