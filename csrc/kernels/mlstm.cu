// Matrix-memory recurrence (mLSTM of xLSTM) with a running maximum.
//
// Per head the state is a dim x vdim matrix S, a vector n and a scalar m, all fp32, one set per request slot:
//   m' = max(f + m, i);  S' = exp(f + m - m') S + exp(i - m') k v^T;  n' the same with k alone
//   o  = S'^T q / (max(|n' . q|, exp(-m')) + den_eps)
// A block owns 32 value columns of one head.  Every column block carries its own copy of n and m, so blocks never wait for
// one another.  A request's state starts at zero where its rows start at position 0.
//
//  mlstm_step : one block walks the adjacent rows of a request token by token (decode rows, 32-bit passes)
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
