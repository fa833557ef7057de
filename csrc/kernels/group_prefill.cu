// Grouped-query attention of a long prompt pass (one request, adjacent rows) straight from the paged cache.
//
// The two query tiles of a CTA (ds41_prompt_attend.cuh) are the same 128 rows of two query heads that share a key/value head;
// with one query head per key/value head they are neighbouring row tiles.  Key and value tiles are fetched page by page, so
// nothing is gathered first.  A walk starts at the page that holds the first key its rows see.
#include "ds41_group.cuh"
#include "ds41_prompt_attend.cuh"

namespace ds41 {

struct GroupForm {
  CUtensorMap q, pool;
  const int* page_table;
  const int* row_slot;
  ds41_proj gates;           // one column per head
  int kv_heads, per_group, chunk, max_pages, page_tokens, n_rows_pool;
  static constexpr bool kLowerBound = true;

  __device__ PromptTiles tiles(const PromptParams& p, int block) const {
    PromptTiles t;
    const int row_tiles = (p.rows + kPreTile - 1) / kPreTile;
    const bool pair_heads = per_group > 1;
    const int lanes = kv_heads * (pair_heads ? (per_group + 1) / 2 : 1);      // head pairs, or heads
    const int steps = pair_heads ? row_tiles : (row_tiles + 1) / 2;
    const int step = steps - 1 - block / lanes, lane = block % lanes;         // the last rows first
    const int g = pair_heads ? lane / ((per_group + 1) / 2) : lane, i = pair_heads ? 2 * (lane % ((per_group + 1) / 2)) : 0;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      t.head[k] = g * per_group + (pair_heads ? i + k : 0);
      t.row0[k] = (pair_heads ? step : 2 * step + k) * kPreTile;
    }
    const int first = first_key(p.pos0 + t.row0[0]);
    t.key0 = first - first % page_tokens;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int last = p.pos0 + min(t.row0[k] + kPreTile, p.rows) - 1;
      const bool live = pair_heads ? i + k < per_group : t.row0[k] < p.rows;
      t.n[k] = live ? (last - t.key0) / kPreTile + 1 : 0;
    }
    return t;
  }
  __device__ void prefetch() const {
    tma_prefetch_desc(&q);
    tma_prefetch_desc(&pool);
  }
  __device__ void load_q(const PromptParams& p, uint8_t* dst, uint64_t* bar, int h, int row0) const {
    for (int c = 0; c < p.kd; ++c) tma_load_3d(dst + c * kPreChunk, &q, bar, h * p.dp + 64 * c, row0, 0);
  }
  // one tile of 128 keys, page by page; a page that is not leased reads as zeros (rows beyond the pool)
  __device__ void load_pages(uint8_t* dst, uint64_t* bar, int x, int chunks, int key) const {
    const int slot = row_slot[0];
    for (int i = 0; i < kPreTile; i += page_tokens) {
      const int pg = (key + i) / page_tokens;
      const int id = slot >= 0 && pg < max_pages ? __ldg(page_table + 1ll * slot * max_pages + pg) : -1;
      const int row = id >= 0 ? id * page_tokens : n_rows_pool;
      for (int c = 0; c < chunks; ++c) tma_load_3d(dst + c * kPreChunk + i * 128, &pool, bar, x + 64 * c, row, 0);
    }
  }
  __device__ void load_k(const PromptParams& p, uint8_t* dst, uint64_t* bar, int h, int key) const {
    load_pages(dst, bar, h / per_group * p.dp, p.kd, key);
  }
  __device__ void load_v(const PromptParams& p, uint8_t* dst, uint64_t* bar, int h, int key) const {
    load_pages(dst, bar, kv_heads * p.dp + h / per_group * p.vp, p.vc, key);
  }
  __device__ int first_key(int pos) const { return chunk_start(pos, chunk); }
  __device__ float sink(int) const { return -INFINITY; }
  __device__ void gate(const PromptParams&, int row, int h, int, float (&f)[16]) const {
    const float v = gates.data != nullptr ? sigmoid_f32(proj_at(gates, row, h)) : 1.f;
#pragma unroll
    for (int i = 0; i < 16; ++i) f[i] = v;
  }
};

// the convolution's last inputs of a long pass
__global__ void __launch_bounds__(256) keep_inputs_kernel(ds41_group_attend_args p) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = p.rows - 1 - static_cast<int>(blockIdx.y);
  if (r < 0 || p.row_slot[r] < 0) return;
  keep_inputs(p, r, p.row_slot[r], p.row_pos[r], blockIdx.x, gridDim.x, threadIdx.x, blockDim.x);
}

}  // namespace ds41

using namespace ds41;

extern "C" int ds41_group_prefill(const ds41_group_attend_args* a, void* stream) {
  if (!group_attend_ok(a) || a->f32 || a->pos0 < 0 || a->n_pages <= 0 || (a->ld_out & 7) || (a->ld_q & 7) ||
      (a->page_tokens != 32 && a->page_tokens != 64 && a->page_tokens != 128) || a->vdim_pad > 128 ||
      ((reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->pool) | reinterpret_cast<uintptr_t>(a->out)) & 15))
    return cudaErrorInvalidValue;
  if (a->pos0 + a->rows > 1ll * a->max_pages * a->page_tokens) return cudaErrorInvalidValue;
  PromptParams p{};
  p.rows = a->rows; p.heads = a->heads; p.dp = a->dim_pad; p.rp = 0; p.vp = a->vdim_pad;
  p.n_keys = a->pos0 + a->rows; p.pos0 = a->pos0;
  p.scale_log2 = a->scale * 1.4426950408889634f;
  p.out = static_cast<__nv_bfloat16*>(a->out); p.ld_out = a->ld_out;
  p.status = a->status;
  const int smem = prompt_smem(p);
  if (smem == 0) return cudaErrorInvalidValue;
  GroupForm f{};
  f.page_table = a->page_table; f.row_slot = a->row_slot; f.gates = a->gate;
  f.kv_heads = a->kv_heads; f.per_group = a->heads / a->kv_heads; f.chunk = a->chunk;
  f.max_pages = a->max_pages; f.page_tokens = a->page_tokens; f.n_rows_pool = a->n_pages * a->page_tokens;
  const int row_len = a->kv_heads * (p.dp + p.vp);
  cudaError_t e = make_tensor_map_3d(&f.q, a->q, TmaDtype::kBF16, 1ull * p.heads * p.dp, p.rows, 1, a->ld_q * 2, 0, 64,
                                     kPreTile, true);
  if (e != cudaSuccess) return e;
  e = make_tensor_map_3d(&f.pool, a->pool, TmaDtype::kBF16, row_len, f.n_rows_pool, 1, 2ull * row_len, 0, 64, a->page_tokens, true);
  if (e != cudaSuccess) return e;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->taps > 1) {
    e = launch_pdl(keep_inputs_kernel, dim3(4, a->taps - 1), dim3(256), 0, st, *a);
    if (e != cudaSuccess) return e;
  }
  const int row_tiles = (p.rows + kPreTile - 1) / kPreTile;
  const int blocks = f.per_group > 1 ? row_tiles * f.kv_heads * ((f.per_group + 1) / 2) : (row_tiles + 1) / 2 * f.kv_heads;
  return launch_prompt_attend(f, p, blocks, smem, st);
}
