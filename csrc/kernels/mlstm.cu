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
//  mlstm_chunk: one request's rows, 64 at a time, on the tensor cores, in three launches: the gates of every chunk; the
//               states from chunk to chunk; the outputs of all chunks side by side.  With F the running sum of f inside a chunk and m0
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

// Layout of the workspace, in bytes from its start.
struct ChunkWork {
  long long gates, n, state, total;
};
__host__ __device__ inline int chunk_tiles(int dim_pad) {        // NTD of the kernels that take this key width
  return dim_pad <= 64 ? 2 : dim_pad <= 128 ? 4 : dim_pad <= 192 ? 6 : dim_pad <= 256 ? 8 : dim_pad <= 384 ? 12 : 16;
}
__host__ __device__ inline ChunkWork chunk_work(int rows, int heads, int dim_pad, int vdim_pad) {
  const long long chunks = (rows + kChunk - 1) / kChunk, per = chunks * heads;
  const long long D = chunk_tiles(dim_pad) * 32, nb = (vdim_pad + kStateCols - 1) / kStateCols;
  ChunkWork w;
  w.gates = 0;
  w.n = per * kGateFloats * 4;
  w.state = w.n + per * D * 4;
  w.total = w.state + per * nb * D * kStateCols * 4;
  return w;
}

// ---- states: walks the chunks of one head and 32 value columns and leaves the state before every chunk in the workspace
// The key dimension is shared by kSplit CTAs, whose warps take slices of a quarter each.
template <int NTD>
struct StateSmem {
  static constexpr int kSplit = NTD % 4 == 0 ? 2 : 1;
  static constexpr int D = NTD * 32 / kSplit;                      // key columns of this CTA
  static constexpr int NT = NTD / kSplit;                          // state tiles of 8 key columns per warp
  static constexpr int kStride = D + 8;                            // bf16 per row of a key tile
  static constexpr int kStage = kChunk * kStride * 2 + kChunk * kVStride * 2 + (kChunk + 4) * 4;
  static constexpr int kFixed = 2 * kChunk * kVStride * 2 + D * 4;
  static constexpr int kStages = 2 * (4 * kStage + kFixed) <= 224 * 1024 ? 4 : 3;      // two CTAs per SM where they fit
  static constexpr int kBytes = kStages * kStage + kFixed;
};

// 256 threads; warp w owns value columns 16 (w & 1) .. +16 and the (w >> 1)-th quarter of this CTA's key columns, whose slice
// of the transposed state it keeps in registers.
template <int NTD>
__global__ void __launch_bounds__(256) mlstm_state_kernel(ds41_mlstm_args p) {
  using Sm = StateSmem<NTD>;
  constexpr int D = Sm::D, DQ = D / 4, S = Sm::kStages, NT = Sm::NT;
  extern __shared__ __align__(16) uint8_t ms_raw[];
  __nv_bfloat16* w_hi = reinterpret_cast<__nv_bfloat16*>(ms_raw + S * Sm::kStage);
  __nv_bfloat16* w_lo = w_hi + kChunk * kVStride;
  float* nv = reinterpret_cast<float*>(w_lo + kChunk * kVStride);      // [D]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int vb = blockIdx.x, h = blockIdx.y, d_base = blockIdx.z * D;
  const int nt = warp & 1, dq = warp >> 1, g = lane >> 2, q2 = 2 * (lane & 3);
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[0];
  if (slot < 0 || slot >= p.slots) return;
  const bool fresh = p.row_pos[0] == 0;
  const int nb = gridDim.x, col0 = vb * kStateCols;
  const long long head = 1ll * slot * p.heads + h;
  float* gS = p.state_s + head * p.dim_pad * p.vdim_pad;
  float* gn = p.state_n + head * nb * p.dim_pad;
  const ChunkWork wk = chunk_work(p.rows, p.heads, p.dim_pad, p.vdim_pad);
  uint8_t* work = reinterpret_cast<uint8_t*>(p.work);

  const __nv_bfloat16* gk = static_cast<const __nv_bfloat16*>(p.k.data) + p.k.col + h * p.dim_pad + d_base;
  const __nv_bfloat16* gv = static_cast<const __nv_bfloat16*>(p.v.data) + p.v.col + h * p.vdim_pad + col0;
  const int n_chunks = (p.rows + kChunk - 1) / kChunk;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  auto load = [&](int c) {
    if (c < n_chunks) {
      __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(ms_raw + (c % S) * Sm::kStage);
      __nv_bfloat16* sv = sk + kChunk * Sm::kStride;
      const int live = p.rows - c * kChunk;
      constexpr int kPer = D / 8, kRows = 256 / kPer;                  // 16-byte pieces of a row, rows per sweep
      if (kPer * kRows == 256 || tid < kPer * kRows) {
        const int d = (tid % kPer) * 8;
        const __nv_bfloat16* k = gk + (1ll * c * kChunk + tid / kPer) * p.k.ld + d;
        for (int t = tid / kPer; t < kChunk; t += kRows, k += 1ll * kRows * p.k.ld) {
          if (t < live && d_base + d < p.dim_pad) cp_async_16(sk + t * Sm::kStride + d, k);
          else *reinterpret_cast<uint4*>(sk + t * Sm::kStride + d) = zero;
        }
      }
      const int t = tid >> 2, d = (tid & 3) * 8;
      if (t < live && col0 + d < p.vdim_pad) cp_async_16(sv + t * kVStride + d, gv + (1ll * c * kChunk + t) * p.v.ld + d);
      else *reinterpret_cast<uint4*>(sv + t * kVStride + d) = zero;
      // the weights of the keys and the scalars
      const float* gates = p.work + (1ll * c * p.heads + h) * kGateFloats;
      float* sg = reinterpret_cast<float*>(sv + kChunk * kVStride);
      if (tid < kChunk / 4) cp_async_16(sg + 4 * tid, gates + 2 * kChunk + 4 * tid);
      else if (tid == kChunk / 4) cp_async_16(sg + kChunk, gates + 5 * kChunk);
    }
    cp_async_commit();                 // one group per call, so that the waits count calls
  };
#pragma unroll
  for (int i = 0; i < S - 1; ++i) load(i);
  // transposed state: tile j holds columns d = d_base + dq DQ + 8 j + q2 + {0, 1} of rows nt 16 + g and + 8
  float st[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d_base + dq * DQ + 8 * j + q2 + (e & 1), c = col0 + nt * 16 + g + (e >> 1) * 8;
      st[j][e] = !fresh && d < p.dim_pad && c < p.vdim_pad ? gS[1ll * d * p.vdim_pad + c] : 0.f;
    }
  if (vb == 0)
    for (int d = tid; d < D; d += 256) nv[d] = !fresh && d_base + d < p.dim_pad ? gn[d_base + d] : 0.f;
  float m_end = 0.f;
  for (int c = 0; c < n_chunks; ++c) {
    cp_async_wait<S - 2>();
    __syncthreads();                   // chunk c is here; every warp is done with chunk c - 1
    load(c + S - 1);
    const __nv_bfloat16* sk = reinterpret_cast<const __nv_bfloat16*>(ms_raw + (c % S) * Sm::kStage);
    const __nv_bfloat16* sv = sk + kChunk * Sm::kStride;
    const float* sg = reinterpret_cast<const float*>(sv + kChunk * kVStride);
    // ---- decayed values
    {
      const int s = tid >> 2, d = (tid & 3) * 8;
      const float w = sg[s];
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
    // ---- the state before this chunk, as the output kernel's left operand wants it: high and low parts per fragment
    {
      const long long cell = (1ll * c * p.heads + h) * nb + vb;
      // the output kernel's warp and its first fragment that these columns belong to
      const int slice = blockIdx.z * 4 + dq, quarter = slice / Sm::kSplit, first = slice % Sm::kSplit * (NT / 2);
      uint4* dst = reinterpret_cast<uint4*>(work + wk.state) + (cell * 8 + quarter * 2 + nt) * NTD * 32 + first * 64 + lane;
#pragma unroll
      for (int k = 0; k < NT / 2; ++k) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = st[2 * k + (e >> 1)][2 * (e & 1)], y = st[2 * k + (e >> 1)][2 * (e & 1) + 1];
          hi[e] = pack_bf16(x, y);
          lo[e] = pack_bf16_rest(x, y, hi[e]);
        }
        dst[(2 * k) * 32] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        dst[(2 * k + 1) * 32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      if (vb == 0) {
        float* gw = reinterpret_cast<float*>(work + wk.n) + (1ll * c * p.heads + h) * NTD * 32 + d_base;
        for (int d = tid; d < D; d += 256) gw[d] = nv[d];
      }
    }
    __syncthreads();
    const float keep = sg[kChunk];
    m_end = sg[kChunk + 1];
#pragma unroll
    for (int j = 0; j < NT; ++j)
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
      for (int j = 0; j < NT / 2; ++j) {
        uint32_t b[4];
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], brow + k * Sm::kStride + 16 * j);
        mma_bf16_16816(st[2 * j], hi, b[0], b[1]);
        mma_bf16_16816(st[2 * j + 1], hi, b[2], b[3]);
        mma_bf16_16816(st[2 * j], lo, b[0], b[1]);
        mma_bf16_16816(st[2 * j + 1], lo, b[2], b[3]);
      }
    }
    if (vb == 0) {
      // n: one row of weights (high parts in row 0, low parts in row 1 of the left operand) times the keys; the two warps
      // of a quarter take half of its columns each
      uint32_t wf[4][2];
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float2 w = *reinterpret_cast<const float2*>(sg + 16 * k + 8 * e + q2);
          const uint32_t hi = pack_bf16(w.x, w.y);
          wf[k][e] = g == 0 ? hi : (g == 1 ? pack_bf16_rest(w.x, w.y, hi) : 0u);
        }
#pragma unroll
      for (int j = nt; j < NT / 2; j += 2) {
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
            nv[d + 8 * u] = nv[d + 8 * u] * keep + (u == 0 ? x[0] : y[0]);
            nv[d + 8 * u + 1] = nv[d + 8 * u + 1] * keep + (u == 0 ? x[1] : y[1]);
          }
        }
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d_base + dq * DQ + 8 * j + q2 + (e & 1), c = col0 + nt * 16 + g + (e >> 1) * 8;
      if (d < p.dim_pad && c < p.vdim_pad) gS[1ll * d * p.vdim_pad + c] = st[j][e];
    }
  if (vb == 0)                         // every column block's copy of n
    for (int b = 0; b < nb; ++b)
      for (int d = tid; d < D; d += 256)
        if (d_base + d < p.dim_pad) gn[1ll * b * p.dim_pad + d_base + d] = nv[d];
  if (tid == 0 && blockIdx.z == 0) p.state_m[head * nb + vb] = m_end;
}

// ---- outputs: every (chunk, head, pair of value blocks) on its own, from the state before the chunk
constexpr int kOutCols = 2 * kStateCols;
constexpr int kOStride = kOutCols + 8;        // bf16 per row of the value tile

template <int NTD>
struct OutSmem {
  static constexpr int D = NTD * 32;
  static constexpr int kStride = D + 8;
  static constexpr int kTile = kChunk * kStride * 2;
  static constexpr int kRed = 4 * kChunk * kRedStride * 4;             // takes the key tile's place once it has been used
  static constexpr int kKeys = kTile > kRed ? kTile : kRed;
  static constexpr int kBytes = kTile + kKeys + kChunk * kOStride * 2 + kGateFloats * 4 + 2 * kChunk * kPStride * 2 +
                                8 * kStride * 2 + 4 * kChunk * 4;
};

// 256 threads.  Q K^T: warp w owns 16 rows x 32 keys; outputs: as in the state kernel, one 32-column block after the other.
template <int NTD>
__global__ void __launch_bounds__(256, NTD <= 8 ? 2 : 1) mlstm_output_kernel(ds41_mlstm_args p) {
  using Sm = OutSmem<NTD>;
  constexpr int D = Sm::D, DQ = D / 4;
  extern __shared__ __align__(16) uint8_t mo_raw[];
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(mo_raw);
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(mo_raw + Sm::kTile);
  float* red = reinterpret_cast<float*>(sk);                           // [4][64][33]
  __nv_bfloat16* sv = reinterpret_cast<__nv_bfloat16*>(mo_raw + Sm::kTile + Sm::kKeys);
  float* gates = reinterpret_cast<float*>(sv + kChunk * kOStride);
  __nv_bfloat16* p_hi = reinterpret_cast<__nv_bfloat16*>(gates + kGateFloats);
  __nv_bfloat16* p_lo = p_hi + kChunk * kPStride;
  __nv_bfloat16* n_rows = p_lo + kChunk * kPStride;                    // [8][D + 8]: n as high and low parts, zero rows
  float* nq = reinterpret_cast<float*>(n_rows + 8 * Sm::kStride);      // n . q_t before the chunk
  float* rs = nq + kChunk;             // [2][64] sums of the decayed scores
  float* inv = rs + 2 * kChunk;        // 1 / denominator
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pair = blockIdx.x, h = blockIdx.y, c = blockIdx.z;
  const int nt = warp & 1, dq = warp >> 1, g = lane >> 2, q2 = 2 * (lane & 3);
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[0];
  if (slot < 0 || slot >= p.slots) return;
  const int nb = (p.vdim_pad + kStateCols - 1) / kStateCols, col0 = pair * kOutCols, live = p.rows - c * kChunk;
  const ChunkWork wk = chunk_work(p.rows, p.heads, p.dim_pad, p.vdim_pad);
  const uint8_t* work = reinterpret_cast<const uint8_t*>(p.work);
  const long long cell = 1ll * c * p.heads + h;
  {
    const __nv_bfloat16* gq = static_cast<const __nv_bfloat16*>(p.q.data) + p.q.col + h * p.dim_pad;
    const __nv_bfloat16* gk = static_cast<const __nv_bfloat16*>(p.k.data) + p.k.col + h * p.dim_pad;
    const __nv_bfloat16* gv = static_cast<const __nv_bfloat16*>(p.v.data) + p.v.col + h * p.vdim_pad + col0;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    constexpr int kPer = D / 8, kRows = 256 / kPer;
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
#pragma unroll
    for (int i = tid; i < kChunk * kOutCols / 8; i += 256) {
      const int t = i >> 3, d = (i & 7) * 8;
      if (t < live && col0 + d < p.vdim_pad) cp_async_16(sv + t * kOStride + d, gv + (1ll * c * kChunk + t) * p.v.ld + d);
      else *reinterpret_cast<uint4*>(sv + t * kOStride + d) = zero;
    }
    if (tid < kGateFloats / 4) cp_async_16(gates + 4 * tid, p.work + cell * kGateFloats + 4 * tid);
    cp_async_commit();
    const float* gw = reinterpret_cast<const float*>(work + wk.n) + cell * D;
    for (int d = tid; d < D; d += 256) {
      const float x = gw[d];
      const __nv_bfloat16 hi = __float2bfloat16_rn(x);
      n_rows[d] = hi;
      n_rows[Sm::kStride + d] = __float2bfloat16_rn(x - __bfloat162float(hi));
    }
    for (int i = tid; i < 6 * Sm::kStride; i += 256) n_rows[2 * Sm::kStride + i] = __float2bfloat16_rn(0.f);
  }
  // the state fragments of the first value block travel while the scores are computed
  constexpr bool kAhead = NTD <= 8;
  constexpr int kFrags = kAhead ? NTD : 2;
  const uint4* frag = reinterpret_cast<const uint4*>(work + wk.state) + ((cell * nb + 2 * pair) * 8 + warp) * NTD * 32 + lane;
  uint4 ahead[kFrags];
  if (kAhead)
#pragma unroll
    for (int k = 0; k < kFrags; ++k) ahead[k] = __ldcg(frag + k * 32);
  cp_async_wait<0>();
  __syncthreads();
  // ---- decayed scores, 16 rows x 32 keys per warp; one warp per row tile also takes n . q_t
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
    if ((sh == 1) == (tm < 2)) {        // of the first row tiles the warps that have no visible keys
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
  __syncthreads();
  if (tid < kChunk)
    inv[tid] = 1.0f / (fmaxf(fabsf(gates[3 * kChunk + tid] * nq[tid] + rs[tid] + rs[kChunk + tid]), gates[4 * kChunk + tid]) +
                       p.den_eps);
  // ---- outputs, transposed: 16 value columns x 64 rows per warp, this warp's quarter of d and of the keys
#pragma unroll 1
  for (int half = 0; half < 2; ++half) {
    const int vb = 2 * pair + half;
    if (vb >= nb) break;
    float o[8][4] = {};
    const __nv_bfloat16* brow = sq + ((lane & 7) + (lane >> 4) * 8) * Sm::kStride + dq * DQ + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int k = 0; k < NTD / 2; ++k) {
      const uint4 fh = kAhead ? ahead[(2 * k) % kFrags] : __ldcg(frag + (2 * k) * 32);
      const uint4 fl = kAhead ? ahead[(2 * k + 1) % kFrags] : __ldcg(frag + (2 * k + 1) * 32);
      const uint32_t hi[4] = {fh.x, fh.y, fh.z, fh.w}, lo[4] = {fl.x, fl.y, fl.z, fl.w};
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
    frag += 8 * NTD * 32;               // the next value block's
    if (kAhead && half == 0 && vb + 1 < nb)
#pragma unroll
      for (int k = 0; k < kFrags; ++k) ahead[k] = __ldcg(frag + k * 32);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float2 f = *reinterpret_cast<const float2*>(gates + 3 * kChunk + 8 * j + q2);
      o[j][0] *= f.x;
      o[j][1] *= f.y;
      o[j][2] *= f.x;
      o[j][3] *= f.y;
    }
    uint32_t a[4];
    ldmatrix_x4_trans(a[0], a[1], a[2], a[3], sv + (dq * 16 + (lane & 7) + (lane >> 4) * 8) * kOStride +
                                                  half * kStateCols + nt * 16 + ((lane >> 3) & 1) * 8);
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
    float* part = red + dq * kChunk * kRedStride + nt * 16 + g;
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) part[(8 * j + q2 + (e & 1)) * kRedStride + (e >> 1) * 8] = o[j][e];
    __syncthreads();
    const int col = vb * kStateCols + lane;
    if (col < p.vdim_pad) {
      const int t0 = warp * 8;
      float* dst = p.out + (1ll * c * kChunk + t0) * p.ld_out + h * p.vdim_pad + col;
      const float* src = red + t0 * kRedStride + lane;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float x = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) x += src[(w * kChunk + i) * kRedStride];
        if (t0 + i < live) dst[1ll * i * p.ld_out] = x * inv[t0 + i];
      }
    }
    __syncthreads();
  }
}

template <int NTD>
static int launch_chunk(const ds41_mlstm_args& a, cudaStream_t st) {
  static bool ready = false;
  cudaError_t e = cudaSuccess;
  if (!ready) {
    e = cudaFuncSetAttribute(mlstm_state_kernel<NTD>, cudaFuncAttributeMaxDynamicSharedMemorySize, StateSmem<NTD>::kBytes);
    if (e != cudaSuccess) return e;
    e = cudaFuncSetAttribute(mlstm_output_kernel<NTD>, cudaFuncAttributeMaxDynamicSharedMemorySize, OutSmem<NTD>::kBytes);
    if (e != cudaSuccess) return e;
    ready = true;
  }
  const int n_chunks = (a.rows + kChunk - 1) / kChunk, nb = (a.vdim_pad + kStateCols - 1) / kStateCols;
  const size_t gate_smem = 3ull * n_chunks * sizeof(float);
  if (gate_smem > 48 * 1024) return cudaErrorInvalidValue;
  e = launch_pdl(mlstm_gates_kernel, dim3(a.heads), dim3(1024), gate_smem, st, a);
  if (e != cudaSuccess) return e;
  e = launch_pdl(mlstm_state_kernel<NTD>, dim3(nb, a.heads, StateSmem<NTD>::kSplit), dim3(256), StateSmem<NTD>::kBytes, st, a);
  if (e != cudaSuccess) return e;
  return launch_pdl(mlstm_output_kernel<NTD>, dim3((nb + 1) / 2, a.heads, n_chunks), dim3(256), OutSmem<NTD>::kBytes, st, a);
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
  if (a->dim_pad > 512) return cudaErrorInvalidValue;
  switch (chunk_tiles(a->dim_pad)) {
    case 2: return launch_chunk<2>(*a, st);
    case 4: return launch_chunk<4>(*a, st);
    case 6: return launch_chunk<6>(*a, st);
    case 8: return launch_chunk<8>(*a, st);
    case 12: return launch_chunk<12>(*a, st);
    default: return launch_chunk<16>(*a, st);
  }
}

extern "C" long long ds41_mlstm_chunk_work(int rows, int heads, int dim_pad, int vdim_pad) {
  return rows <= 0 || heads <= 0 || dim_pad <= 0 || vdim_pad <= 0 ? 0 : chunk_work(rows, heads, dim_pad, vdim_pad).total;
}
