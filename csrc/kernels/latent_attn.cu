// Latent attention: every head's keys and values are linear maps of one cached latent row per token, beside one rotated
// key part that all heads share.  A cache row is [latent (kv_pad) | rotated key part (rot_pad)], zero in the padding.
//
//  latent_post   : RMS norm of the query latent; RMS norm of the key/value latent and rotation of the shared key part into
//                  the request's cache pages
//  latent_query  : per-head queries [dim | rotated part] from a projection, the rotated part turned by the row's position
//  latent_gather : one request's cache rows as two contiguous matrices (prompt passes expand keys and values from them)
//  latent_attend : causal attention over the cache with absorbed queries (q W_uk, so that the latent row itself is key and
//                  value), partial results per key split
//  latent_merge  : sums the splits; the softmax denominator also contains exp(sink) per head
#include "ds41_stack.cuh"

namespace ds41 {

__device__ __forceinline__ void rotate_pair(float u, float v, int pos, float freq, float mag, float& ru, float& rv) {
  float s, c;
  sincosf(static_cast<float>(pos) * freq, &s, &c);
  c *= mag;
  s *= mag;
  ru = u * c - v * s;
  rv = v * c + u * s;
}

// Cache row of position `pos` of a request, or null when its page is not leased.
template <typename T>
__device__ __forceinline__ T* cache_row(T* pool, const int* page_table, int max_pages, int page_tokens, int row_len,
                                        int slot, int pos) {
  const int pg = pos / page_tokens;
  if (pg < 0 || pg >= max_pages) return nullptr;
  const int id = page_table[1ll * slot * max_pages + pg];
  if (id < 0) return nullptr;
  return pool + (1ll * id * page_tokens + (pos - pg * page_tokens)) * row_len;
}

template <typename T>
__global__ void __launch_bounds__(256) latent_post_kernel(ds41_latent_post_args p) {
  __shared__ float red[33];
  const int r = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  if (blockIdx.y == 0) {
    float q = 0.f;
    for (int i = threadIdx.x; i < p.q_rank; i += blockDim.x) {
      const float v = proj_at(p.dq, r, i);
      q += v * v;
    }
    const float s = 1.0f / sqrtf(block_sum(q, red) / p.q_rank + p.eps);
    T* out = static_cast<T*>(p.cq) + 1ll * r * p.ld_cq;
    for (int i = threadIdx.x; i < p.q_rank; i += blockDim.x) out[i] = from_f32<T>(proj_at(p.dq, r, i) * s * p.dq_norm[i]);
    return;
  }
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  if (slot < 0) return;
  T* row = cache_row(static_cast<T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, p.row_len, slot, pos);
  if (row == nullptr) return;
  float q = 0.f;
  for (int i = threadIdx.x; i < p.kv_rank; i += blockDim.x) {
    const float v = proj_at(p.kv, r, i);
    q += v * v;
  }
  const float s = 1.0f / sqrtf(block_sum(q, red) / p.kv_rank + p.eps);
  for (int i = threadIdx.x; i < p.kv_rank; i += blockDim.x) row[i] = from_f32<T>(proj_at(p.kv, r, i) * s * p.kv_norm[i]);
  for (int i = threadIdx.x; i < p.rot_dim / 2; i += blockDim.x) {
    float a, b;
    rotate_pair(proj_at(p.kr, r, 2 * i), proj_at(p.kr, r, 2 * i + 1), pos, p.freq[i], p.magnitude, a, b);
    row[p.kv_pad + 2 * i] = from_f32<T>(a);
    row[p.kv_pad + 2 * i + 1] = from_f32<T>(b);
  }
}

// In place when q is the projection itself (q.data == out): then only the rotated parts change.
template <typename T>
__global__ void __launch_bounds__(256) latent_query_kernel(ds41_proj q, const int* row_pos, const float* freq,
                                                           float magnitude, int heads, int dim_pad, int rot_pad,
                                                           int rot_dim, T* out, int ld_out, int in_place) {
  const int r = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  const int hs = dim_pad + rot_pad;
  const int half = in_place ? rot_pad / 2 : hs / 2;
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= heads * half) return;
  const int h = i / half, j = 2 * (i - h * half) + (in_place ? dim_pad : 0), c = h * hs + j;
  float a = proj_at(q, r, c), b = proj_at(q, r, c + 1);
  const int t = j - dim_pad;
  if (t >= 0 && t < rot_dim) {
    const float u = a, v = b;
    rotate_pair(u, v, row_pos[r], freq[t / 2], magnitude, a, b);
  }
  out[1ll * r * ld_out + c] = from_f32<T>(a);
  out[1ll * r * ld_out + c + 1] = from_f32<T>(b);
}

template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* pool, const int* page_table, int max_pages,
                                                            int page_tokens, int row_len, int kv_pad, int slot_row,
                                                            const int* row_slot, int n_keys, T* lat, T* rot) {
  const int key = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  if (key >= n_keys) return;
  const int slot = row_slot[slot_row];
  const T* src = slot < 0 ? nullptr
                          : cache_row(const_cast<T*>(pool), page_table, max_pages, page_tokens, row_len, slot, key);
  const int rot_pad = row_len - kv_pad;
  // rows are multiples of 16 elements: whole 16-byte pieces
  constexpr int kPer = 16 / sizeof(T);
  for (int i = lane * kPer; i < row_len; i += 32 * kPer) {
    const uint4 v = src != nullptr ? *reinterpret_cast<const uint4*>(src + i) : make_uint4(0, 0, 0, 0);
    T* dst = i < kv_pad ? lat + 1ll * key * kv_pad + i : rot + 1ll * key * rot_pad + (i - kv_pad);
    *reinterpret_cast<uint4*>(dst) = v;
  }
}

// Plain form for every type and size: one block per (row, head, split), a tile of 32 keys at a time.
template <typename T>
__global__ void __launch_bounds__(128) latent_attend_plain_kernel(ds41_latent_attend_args p) {
  extern __shared__ float att_smem[];
  float* qs = att_smem;                  // [kv_pad + rot_pad] query, scaled
  float* os = qs + p.row_len;            // [kv_pad] running output
  float* sc = os + p.kv_pad;             // [32] scores
  const int h = blockIdx.x, split = blockIdx.y, r = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.row_slot[r], pos = p.row_pos[r];
  const int n_keys = slot < 0 ? 0 : pos + 1;
  int per = (n_keys + p.n_splits - 1) / p.n_splits;
  per = (per + 63) / 64 * 64;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  const long long cell = (1ll * r * p.n_splits + split) * p.heads + h;
  if (k0 >= k1) {
    if (tid == 0) {
      p.part_ml[2 * cell] = -INFINITY;
      p.part_ml[2 * cell + 1] = 0.f;
    }
    return;
  }
  const T* qa = static_cast<const T*>(p.q_abs) + r * p.ld_q_abs + 1ll * h * p.kv_pad;
  const T* qr = static_cast<const T*>(p.q_rot) + r * p.ld_q_rot + 1ll * h * p.q_rot_stride;
  for (int i = tid; i < p.row_len; i += 128) qs[i] = to_f32(i < p.kv_pad ? qa[i] : qr[i - p.kv_pad]);
  for (int i = tid; i < p.kv_pad; i += 128) os[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  __syncthreads();
  for (int t0 = k0; t0 < k1; t0 += 32) {
    for (int j = warp; j < 32; j += 4) {
      const int key = t0 + j;
      float s = -INFINITY;
      if (key < k1) {
        const T* kv = cache_row(static_cast<T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, p.row_len, slot, key);
        float a = 0.f;
        if (kv != nullptr)
          for (int i = lane; i < p.row_len; i += 32) a += qs[i] * to_f32(kv[i]);
        a = warp_sum(a);
        if (kv != nullptr) s = a * p.scale;
      }
      if (lane == 0) sc[j] = s;
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
    for (int i = tid; i < p.kv_pad; i += 128) {
      float a = os[i] * keep;
      for (int j = 0; j < 32 && t0 + j < k1; ++j) {
        const T* kv = cache_row(static_cast<T*>(p.pool), p.page_table, p.max_pages, p.page_tokens, p.row_len, slot, t0 + j);
        if (kv != nullptr) a += sc[j] * to_f32(kv[i]);
      }
      os[i] = a;
    }
    __syncthreads();
  }
  for (int i = tid; i < p.kv_pad; i += 128) p.part_o[cell * p.kv_pad + i] = os[i];
  if (tid == 0) {
    p.part_ml[2 * cell] = m;
    p.part_ml[2 * cell + 1] = l;
  }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* part_o, const float* part_ml, const float* sink,
                                                           int n_splits, int heads, int kv_pad, T* out, int ld_out) {
  const int h = blockIdx.x, r = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  const long long cell0 = 1ll * r * n_splits * heads + h;
  float m = sink != nullptr ? sink[h] : -INFINITY;
  for (int s = 0; s < n_splits; ++s) m = fmaxf(m, part_ml[2 * (cell0 + 1ll * s * heads)]);
  float den = sink != nullptr ? expf(sink[h] - m) : 0.f;
  for (int s = 0; s < n_splits; ++s) {
    const float* ml = part_ml + 2 * (cell0 + 1ll * s * heads);
    if (ml[1] > 0.f) den += ml[1] * expf(ml[0] - m);
  }
  const float inv = den > 0.f ? 1.0f / den : 0.f;
  for (int i = threadIdx.x; i < kv_pad; i += blockDim.x) {
    float a = 0.f;
    for (int s = 0; s < n_splits; ++s) {
      const long long c = cell0 + 1ll * s * heads;
      if (part_ml[2 * c + 1] > 0.f) a += part_o[c * kv_pad + i] * expf(part_ml[2 * c] - m);
    }
    out[1ll * r * ld_out + h * kv_pad + i] = from_f32<T>(a * inv);
  }
}

}  // namespace ds41

using namespace ds41;

static bool proj_ok(const ds41_proj& p) {
  return p.data != nullptr && p.ld > 0 && p.splits >= 1 && p.col >= 0 && (p.splits == 1 || (p.plane > 0 && !p.bf16));
}

extern "C" int ds41_latent_post(const ds41_latent_post_args* a, void* stream) {
  if (a == nullptr || a->rows <= 0 || !proj_ok(a->dq) || a->cq == nullptr || a->dq_norm == nullptr || a->q_rank <= 0 ||
      a->ld_cq < a->q_rank)
    return cudaErrorInvalidValue;
  const bool kv = a->pool != nullptr;       // a layer that reads another layer's rows writes none
  if (kv && (!proj_ok(a->kv) || !proj_ok(a->kr) || a->kv_norm == nullptr || a->freq == nullptr || a->kv_rank <= 0 ||
             a->kv_pad < a->kv_rank || a->row_len < a->kv_pad + a->rot_dim || (a->rot_dim & 1) || a->page_tokens <= 0 ||
             a->max_pages <= 0 || a->page_table == nullptr || a->row_pos == nullptr || a->row_slot == nullptr))
    return cudaErrorInvalidValue;
  const dim3 grid(a->rows, kv ? 2 : 1);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->f32 ? launch_pdl(latent_post_kernel<float>, grid, dim3(256), 0, st, *a)
                : launch_pdl(latent_post_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, *a);
}

extern "C" int ds41_latent_query(const ds41_proj* q, const int* row_pos, const float* freq, float magnitude, int rows,
                                 int heads, int dim_pad, int rot_pad, int rot_dim, void* out, int ld_out, int f32,
                                 void* stream) {
  if (q == nullptr || !proj_ok(*q) || row_pos == nullptr || freq == nullptr || rows <= 0 || rows > 65535 || heads <= 0 ||
      dim_pad < 0 || (dim_pad & 1) || (rot_pad & 1) || (rot_dim & 1) || rot_dim > rot_pad || out == nullptr ||
      ld_out < heads * (dim_pad + rot_pad))
    return cudaErrorInvalidValue;
  const int in_place = q->data == out ? 1 : 0;
  if (in_place && ((f32 != 0) == (q->bf16 != 0) || q->splits != 1 || q->col != 0 || q->ld != ld_out)) return cudaErrorInvalidValue;
  if (in_place && rot_pad == 0) return cudaSuccess;
  const int half = in_place ? rot_pad / 2 : (dim_pad + rot_pad) / 2;
  const dim3 grid((heads * half + 255) / 256, rows);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return launch_pdl(latent_query_kernel<float>, grid, dim3(256), 0, st, *q, row_pos, freq, magnitude, heads, dim_pad,
                      rot_pad, rot_dim, static_cast<float*>(out), ld_out, in_place);
  return launch_pdl(latent_query_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, *q, row_pos, freq, magnitude, heads,
                    dim_pad, rot_pad, rot_dim, static_cast<__nv_bfloat16*>(out), ld_out, in_place);
}

extern "C" int ds41_latent_gather(const void* pool, const int* page_table, int max_pages, int page_tokens, int row_len,
                                  int kv_pad, int slot_row, const int* row_slot, int n_keys, void* lat, void* rot,
                                  int f32, void* stream) {
  if (pool == nullptr || page_table == nullptr || lat == nullptr || row_slot == nullptr || slot_row < 0 || n_keys <= 0 ||
      page_tokens <= 0 || max_pages <= 0 || kv_pad <= 0 || (kv_pad & 15) || (row_len & 15) || row_len < kv_pad ||
      (row_len > kv_pad && rot == nullptr))
    return cudaErrorInvalidValue;
  const dim3 grid((n_keys + 7) / 8);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return launch_pdl(latent_gather_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(pool), page_table,
                      max_pages, page_tokens, row_len, kv_pad, slot_row, row_slot, n_keys, static_cast<float*>(lat),
                      static_cast<float*>(rot));
  return launch_pdl(latent_gather_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(pool),
                    page_table, max_pages, page_tokens, row_len, kv_pad, slot_row, row_slot, n_keys,
                    static_cast<__nv_bfloat16*>(lat), static_cast<__nv_bfloat16*>(rot));
}

extern "C" int ds41_latent_attend(const ds41_latent_attend_args* a, void* stream) {
  if (a == nullptr || a->rows <= 0 || a->rows > 65535 || a->heads <= 0 || a->n_splits <= 0 || a->n_splits > 65535 ||
      a->kv_pad <= 0 || a->row_len < a->kv_pad || a->page_tokens <= 0 || a->max_pages <= 0 || a->q_abs == nullptr ||
      (a->row_len > a->kv_pad && a->q_rot == nullptr) || a->pool == nullptr || a->page_table == nullptr ||
      a->row_pos == nullptr || a->row_slot == nullptr || a->part_o == nullptr || a->part_ml == nullptr)
    return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const size_t smem = (1ull * a->row_len + a->kv_pad + 32) * sizeof(float);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const dim3 grid(a->heads, a->n_splits, a->rows);
  return a->f32 ? launch_pdl(latent_attend_plain_kernel<float>, grid, dim3(128), smem, st, *a)
                : launch_pdl(latent_attend_plain_kernel<__nv_bfloat16>, grid, dim3(128), smem, st, *a);
}

extern "C" int ds41_latent_merge(const float* part_o, const float* part_ml, const float* sink, int n_splits, int rows,
                                 int heads, int kv_pad, void* out, int ld_out, int f32, void* stream) {
  if (part_o == nullptr || part_ml == nullptr || n_splits <= 0 || rows <= 0 || rows > 65535 || heads <= 0 ||
      kv_pad <= 0 || out == nullptr || ld_out < heads * kv_pad)
    return cudaErrorInvalidValue;
  const dim3 grid(heads, rows);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return launch_pdl(latent_merge_kernel<float>, grid, dim3(128), 0, st, part_o, part_ml, sink, n_splits, heads, kv_pad,
                      static_cast<float*>(out), ld_out);
  return launch_pdl(latent_merge_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, part_o, part_ml, sink, n_splits, heads,
                    kv_pad, static_cast<__nv_bfloat16*>(out), ld_out);
}
