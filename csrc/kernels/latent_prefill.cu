// Causal attention of a long prompt pass over expanded keys and values: one request, adjacent rows.
//
// Head h's key is [K row: dim values | rotated part shared by all heads], its value a V row; the two query tiles of a CTA are
// neighbouring tiles of one head (ds41_prompt_attend.cuh).  The softmax denominator contains exp(sink) of the head; the
// output is multiplied by the sigmoid of its gate row before it leaves.
#include "ds41_prompt_attend.cuh"

namespace ds41 {

struct LatentForm {
  CUtensorMap q, kv, rot;
  const float* sinks;
  ds41_proj gates;
  static constexpr bool kLowerBound = false;

  __device__ PromptTiles tiles(const PromptParams& p, int block) const {
    PromptTiles t;
    const int n_pairs = (p.rows + 2 * kPreTile - 1) / (2 * kPreTile);
    const int pair = n_pairs - 1 - block / p.heads;                           // the longest walks first
    t.key0 = 0;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      t.head[i] = block % p.heads;
      t.row0[i] = (2 * pair + i) * kPreTile;
      const int last = min(t.row0[i] + kPreTile, p.rows) - 1;
      t.n[i] = t.row0[i] < p.rows ? min((p.pos0 + last) / kPreTile + 1, (p.n_keys + kPreTile - 1) / kPreTile) : 0;
    }
    return t;
  }
  __device__ void prefetch() const {
    tma_prefetch_desc(&q);
    tma_prefetch_desc(&kv);
  }
  __device__ void load_q(const PromptParams& p, uint8_t* dst, uint64_t* bar, int h, int row0) const {
    const int x = h * (p.dp + p.rp);
    for (int c = 0; c < p.kd; ++c) tma_load_3d(dst + c * kPreChunk, &q, bar, x + 64 * c, row0, 0);
    for (int c = 0; c < p.kr; ++c) tma_load_3d(dst + (p.kd + c) * kPreChunk, &q, bar, x + p.dp + 64 * c, row0, 0);
  }
  __device__ void load_k(const PromptParams& p, uint8_t* dst, uint64_t* bar, int h, int key) const {
    for (int c = 0; c < p.kd; ++c) tma_load_3d(dst + c * kPreChunk, &kv, bar, h * p.dp + 64 * c, key, 0);
    for (int c = 0; c < p.kr; ++c) tma_load_3d(dst + (p.kd + c) * kPreChunk, &rot, bar, 64 * c, key, 0);
  }
  __device__ void load_v(const PromptParams& p, uint8_t* dst, uint64_t* bar, int h, int key) const {
    const int x = p.heads * p.dp + h * p.vp;
    for (int c = 0; c < p.vc; ++c) tma_load_3d(dst + c * kPreChunk, &kv, bar, x + 64 * c, key, 0);
  }
  __device__ int first_key(int) const { return 0; }
  __device__ float sink(int h) const { return sinks != nullptr ? sinks[h] * 1.4426950408889634f : -INFINITY; }
  __device__ void gate(const PromptParams& p, int row, int h, int c, float (&f)[16]) const {
    if (gates.data == nullptr) {
#pragma unroll
      for (int i = 0; i < 16; ++i) f[i] = 1.f;
      return;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float4 x = proj_at4(gates, row, h * p.vp + c + 4 * i);
      f[4 * i] = sigmoid_f32(x.x);
      f[4 * i + 1] = sigmoid_f32(x.y);
      f[4 * i + 2] = sigmoid_f32(x.z);
      f[4 * i + 3] = sigmoid_f32(x.w);
    }
  }
};

}  // namespace ds41

using namespace ds41;

extern "C" int ds41_latent_prefill(const ds41_latent_prefill_args* a, void* stream) {
  if (a == nullptr || a->rows <= 0 || a->heads <= 0 || a->n_keys <= 0 || a->pos0 < 0 || a->pos0 + a->rows > a->n_keys ||
      a->dim_pad < 0 || a->rot_pad < 0 || a->dim_pad + a->rot_pad <= 0 || a->vdim_pad <= 0 || (a->dim_pad & 15) ||
      (a->rot_pad & 15) || (a->vdim_pad & 15) || a->vdim_pad > 128 || a->q == nullptr || a->kv == nullptr ||
      (a->rot_pad > 0 && a->rot == nullptr) || a->out == nullptr || (a->ld_out & 7) || a->ld_out < a->heads * a->vdim_pad)
    return cudaErrorInvalidValue;
  if (a->gate.data != nullptr &&
      (a->gate.splits != 1 || (a->gate.ld & 7) || (a->gate.col & 7) || (reinterpret_cast<uintptr_t>(a->gate.data) & 15)))
    return cudaErrorInvalidValue;
  PromptParams p{};
  p.rows = a->rows; p.heads = a->heads; p.dp = a->dim_pad; p.rp = a->rot_pad; p.vp = a->vdim_pad;
  p.n_keys = a->n_keys; p.pos0 = a->pos0;
  p.scale_log2 = a->scale * 1.4426950408889634f;
  p.out = static_cast<__nv_bfloat16*>(a->out); p.ld_out = a->ld_out;
  p.status = a->status;
  const int smem = prompt_smem(p);
  if (smem == 0) return cudaErrorInvalidValue;
  LatentForm f{};
  f.sinks = a->sink;
  f.gates = a->gate;
  const int hs = p.dp + p.rp;
  cudaError_t e = make_tensor_map_3d(&f.q, a->q, TmaDtype::kBF16, 1ull * p.heads * hs, p.rows, 1, a->ld_q * 2, 0, 64, kPreTile, true);
  if (e != cudaSuccess) return e;
  e = make_tensor_map_3d(&f.kv, a->kv, TmaDtype::kBF16, 1ull * p.heads * (p.dp + p.vp), p.n_keys, 1, a->ld_kv * 2, 0, 64,
                         kPreTile, true);
  if (e != cudaSuccess) return e;
  f.rot = f.kv;
  if (p.rp > 0) {
    e = make_tensor_map_3d(&f.rot, a->rot, TmaDtype::kBF16, p.rp, p.n_keys, 1, 2ull * p.rp, 0, 64, kPreTile, true);
    if (e != cudaSuccess) return e;
  }
  const int pairs = (p.rows + 2 * kPreTile - 1) / (2 * kPreTile);
  return launch_prompt_attend(f, p, p.heads * pairs, smem, static_cast<cudaStream_t>(stream));
}
