// What the kernels of grouped-query attention share (group_attn.cu, group_prefill.cu).
#pragma once
#include "ds41_stack.cuh"

namespace ds41 {

// First position that `pos` sees.
__host__ __device__ __forceinline__ int chunk_start(int pos, int chunk) { return chunk > 0 ? pos - pos % chunk : 0; }

// If row r is one of the last taps - 1 rows of its request in this pass, its share of the convolution's inputs goes into the
// request's ring.  `part` of `parts` blocks works on the row, with `threads` threads each.
__device__ __forceinline__ void keep_inputs(const ds41_group_attend_args& p, int r, int slot, int pos, int part, int parts,
                                            int thread, int threads) {
  const int back = p.taps - 1;
  if (back <= 0 || (r + back < p.rows && p.row_slot[r + back] == slot)) return;
  const int C = (p.heads + p.kv_heads) * p.dim_pad + p.kv_heads * p.vdim_pad;
  float* ring = p.state + (1ll * slot * back + pos % back) * C;
  for (int c = 4 * (part * threads + thread); c < C; c += 4 * parts * threads)
    *reinterpret_cast<float4*>(ring + c) = proj_at4(p.u, r, c);
}

inline bool group_attend_ok(const ds41_group_attend_args* a) {
  return a != nullptr && a->rows > 0 && a->heads > 0 && a->kv_heads > 0 && a->heads % a->kv_heads == 0 && a->heads <= 65535 &&
         a->dim_pad > 0 && !(a->dim_pad & 15) && a->vdim_pad > 0 && !(a->vdim_pad & 15) && a->chunk >= 0 && a->taps >= 1 &&
         a->slots > 0 && a->max_pages > 0 && a->page_tokens > 0 && a->q != nullptr && a->pool != nullptr && a->out != nullptr &&
         a->page_table != nullptr && a->row_pos != nullptr && a->row_slot != nullptr && a->ld_q >= a->heads * a->dim_pad &&
         a->ld_out >= a->heads * a->vdim_pad && (a->gate.data == nullptr || proj_ok(a->gate)) &&
         (a->taps == 1 || (proj_ok(a->u) && proj_vec4(a->u) && a->state != nullptr));
}

}  // namespace ds41
