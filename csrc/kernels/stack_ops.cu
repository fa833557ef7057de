// Row-wise steps of a layer stack whose residual stream is one fp32 row per token.
//
//  resid_step    : closes a sublayer and opens the next one.  result (of routed experts: the sum of the rows that the routes
//                  name) -> sigmoid gate -> norm -> added to the stream;
//                  optionally the stream becomes a weighted sum of the kept streams of all layers so far (depth average);
//                  then the norm that feeds the next sublayer.  With `tokens` the stream starts from the embedding.
//  polynorm      : activation a N(z) + b N(z^2) + c N(z^3) + e, N = division by the row's root mean square
//  gate_mul      : result x sigmoid(gate)
//  head_norm_gate: per-head RMS norm x weight x sigmoid(gate)
//  side_act      : gelu_tanh(projection) x a layer's part of the token's second embedding
//  softcap_rows  : cap tanh(x / cap) in place
//  gather_rows   : picks rows of an activation matrix by index
#include <cooperative_groups.h>

#include "ds41_stack.cuh"

namespace ds41 {

namespace cg = cooperative_groups;

// (mean, sum of squared deviations, count) of a set of values
struct Moments {
  float mean, m2, n;
};
__device__ __forceinline__ Moments merge(Moments a, Moments b) {
  const float n = a.n + b.n;
  if (n == 0.f) return a;
  const float d = b.mean - a.mean, f = b.n / n;
  return {a.mean + d * f, a.m2 + b.m2 + d * d * (a.n * f), n};
}
__device__ __forceinline__ Moments merge_lanes(Moments v) {          // result in lane 0, then in every lane
#pragma unroll
  for (int o = 16; o; o >>= 1)
    v = merge(v, {__shfl_down_sync(0xffffffffu, v.mean, o), __shfl_down_sync(0xffffffffu, v.m2, o),
                  __shfl_down_sync(0xffffffffu, v.n, o)});
  return {__shfl_sync(0xffffffffu, v.mean, 0), __shfl_sync(0xffffffffu, v.m2, 0), __shfl_sync(0xffffffffu, v.n, 0)};
}

// Subtrahend and factor of a row's norm - layer norm (subtract the mean) or RMS norm (mean of squares) - from the pieces of
// four columns that the threads hold; `n` columns of the row are in this CTA, piece i covers columns 4 (tid + i blockDim).
// Deviations are taken from each thread's own mean and merged pairwise, over the warp, the CTA and the cluster, in an order
// that is the same in every thread.  `slot` holds 3 x 32 floats; at most 32 warps (4 per CTA of a cluster of 8).
template <int CL, int NI>
__device__ __forceinline__ float2 row_norm(const float4 (&v)[NI], int n, int W, int kind, float eps, float* slot) {
  float cnt = 0.f, s = 0.f;              // columns beyond the row hold zeros
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int live = n - 4 * static_cast<int>(threadIdx.x + i * blockDim.x);
    cnt += static_cast<float>(max(0, min(4, live)));
    s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
  }
  const float mean = kind == 0 && cnt > 0.f ? s / cnt : 0.f;         // an RMS norm merges with zero means
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int live = n - 4 * static_cast<int>(threadIdx.x + i * blockDim.x);
    const float a = v[i].x - mean, b = v[i].y - mean, c = v[i].z - mean, d = v[i].w - mean;
    q += (live > 0 ? a * a : 0.f) + (live > 1 ? b * b : 0.f) + (live > 2 ? c * c : 0.f) + (live > 3 ? d * d : 0.f);
  }
  Moments t = merge_lanes({mean, q, cnt});
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  if (lane == 0) {
    slot[warp] = t.mean;
    slot[32 + warp] = t.m2;
    slot[64 + warp] = t.n;
  }
  t = {0.f, 0.f, 0.f};
  if constexpr (CL == 1) {
    __syncthreads();
    if (lane < n_warps) t = {slot[lane], slot[32 + lane], slot[64 + lane]};
  } else {
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    if (lane < CL * n_warps) {
      const float* far = cluster.map_shared_rank(slot, lane / n_warps);
      const int w = lane % n_warps;
      t = {far[w], far[32 + w], far[64 + w]};
    }
  }
  t = merge_lanes(t);
  return make_float2(t.mean, 1.0f / sqrtf(t.m2 / W + eps));
}

// Four columns of the sum of a row's routed results, in route order.
__device__ __forceinline__ float4 routed_at4(const ds41_resid_args& p, int r, int col) {
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int k = 0; k < p.y_top; ++k) {
    const int e = p.y_route[r * p.y_top + k];
    if (e < 0) continue;
    const float4 v = proj_at4(p.y, p.y_rows > 0 ? 1ll * e * p.y_rows + r : 1ll * r * p.y_top + k, col);
    s.x += v.x;
    s.y += v.y;
    s.z += v.z;
    s.w += v.w;
  }
  return s;
}

template <typename T, int CL, int NI>
__global__ void __launch_bounds__(CL == 8 ? 128 : (NI <= 4 ? 256 : 512)) resid_step_kernel(ds41_resid_args p) {
  __shared__ float slots[2][96];
  const int per = ((p.W + CL - 1) / CL + 3) / 4 * 4;
  const int part = CL > 1 ? blockIdx.x % CL : 0;
  const int r = CL > 1 ? blockIdx.x / CL : blockIdx.x;
  const int c0 = min(p.W, part * per), n = min(p.W, c0 + per) - c0;
  pdl_launch_dependents();
  pdl_wait();
  float4 x[NI];
  int at[NI], live[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    at[i] = 4 * (threadIdx.x + i * blockDim.x);
    live[i] = n - at[i];
    x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (p.tokens != nullptr) {
    const int tok = p.tokens[r];
    const ds41_proj e{p.embed, 0, static_cast<int>(p.embed_ld), 1, 1, c0};
    if (tok >= 0 && tok < p.vocab)
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (live[i] > 0) x[i] = proj_at4(e, tok, at[i]);
  } else {
    const float* in = p.x_in + r * p.ldx + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (live[i] > 0) x[i] = *reinterpret_cast<const float4*>(in + at[i]);
  }
  // Few rows (clusters): what does not depend on the sublayer is loaded first - the weighted sum of the older kept streams,
  // the norm weight - since the launch is a chain of latencies.  Many rows: the registers are worth more.
  constexpr bool kEarly = CL > 1;
  float4 older[NI], w_next[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    older[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (kEarly) w_next[i] = p.next_w != nullptr && live[i] > 0 ? load4(p.next_w + c0 + at[i], live[i]) : older[i];
  }
  auto add_older = [&]() {
    const float* k0 = p.kept + r * p.ldx + c0;
#pragma unroll 4
    for (int j = 0; j < p.n_mix - 1; ++j) {
      const float c = p.mix[j];
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (live[i] > 0) {
          const float4 k = *reinterpret_cast<const float4*>(k0 + j * p.kept_stride + at[i]);
          older[i].x += c * k.x;
          older[i].y += c * k.y;
          older[i].z += c * k.z;
          older[i].w += c * k.w;
        }
    }
  };
  if (kEarly && p.mix != nullptr) add_older();
  auto clip = [&](float4& v, int i) {         // columns beyond the row hold zeros
    if (live[i] < 4) v.w = 0.f;
    if (live[i] < 3) v.z = 0.f;
    if (live[i] < 2) v.y = 0.f;
  };
  if (p.y.data != nullptr) {
    float4 y[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live[i] > 0) {
        y[i] = p.y_route != nullptr ? routed_at4(p, r, c0 + at[i]) : proj_at4(p.y, r, c0 + at[i]);
        if (p.gate.data != nullptr) {
          const float4 g = proj_at4(p.gate, r, c0 + at[i]), b = load4(p.gate_bias + c0 + at[i], live[i]);
          y[i].x *= sigmoid_f32(g.x + b.x);
          y[i].y *= sigmoid_f32(g.y + b.y);
          y[i].z *= sigmoid_f32(g.z + b.z);
          y[i].w *= sigmoid_f32(g.w + b.w);
        }
        clip(y[i], i);
      }
    }
    float2 s = make_float2(0.f, 1.f);
    if (p.post_w != nullptr) s = row_norm<CL, NI>(y, n, p.W, p.post_rms ? 1 : p.norm_kind, p.eps, slots[0]);
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (live[i] > 0) {
        const float4 w = p.post_w != nullptr ? load4(p.post_w + c0 + at[i], live[i]) : make_float4(1.f, 1.f, 1.f, 1.f);
        x[i].x += (y[i].x - s.x) * s.y * w.x;
        x[i].y += (y[i].y - s.x) * s.y * w.y;
        x[i].z += (y[i].z - s.x) * s.y * w.z;
        x[i].w += (y[i].w - s.x) * s.y * w.w;
      }
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) clip(x[i], i);
  if (p.x_out != nullptr) {
    float* o = p.x_out + r * p.ldx + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (live[i] > 0) store4(o + at[i], x[i]);
  }
  if (p.mix != nullptr) {
    if (!kEarly) add_older();
    const float last = p.mix[p.n_mix - 1];    // the newest kept stream is the row this block holds
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      x[i] = make_float4(older[i].x + last * x[i].x, older[i].y + last * x[i].y, older[i].z + last * x[i].z,
                         older[i].w + last * x[i].w);
      clip(x[i], i);
    }
    if (p.x_avg != nullptr) {
      float* o = p.x_avg + r * p.ldx + c0;
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (live[i] > 0) store4(o + at[i], x[i]);
    }
  }
  if (p.next_w != nullptr) {
    const float2 s = row_norm<CL, NI>(x, n, p.W, p.norm_kind, p.eps, slots[1]);
    T* h = static_cast<T*>(p.h) + 1ll * r * p.ldh + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (live[i] > 0) {
        const float4 w = kEarly ? w_next[i] : load4(p.next_w + c0 + at[i], live[i]);
        store4(h + at[i], make_float4((x[i].x - s.x) * s.y * w.x, (x[i].y - s.x) * s.y * w.y, (x[i].z - s.x) * s.y * w.z,
                                      (x[i].w - s.x) * s.y * w.w));
      }
  }
  if (p.next_w == nullptr && p.raw_h) {
    T* h = static_cast<T*>(p.h) + 1ll * r * p.ldh + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (live[i] > 0) store4(h + at[i], x[i]);
  }
  if constexpr (CL > 1) cg::this_cluster().sync();      // peers may still read this CTA's moments
}

template <typename T>
__global__ void __launch_bounds__(512) polynorm_kernel(ds41_proj z, const float* coef, int ff, int ld_out, float eps,
                                                       T* out) {
  extern __shared__ float zrow[];
  __shared__ float red[33];
  const int r = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto add = [&](float v) {
    const float q = v * v;
    s2 += q;
    s4 += q * q;
    s6 += q * q * q;
  };
#pragma unroll 4
  for (int i = 4 * threadIdx.x; i < ff; i += 4 * blockDim.x) {
    float4 v = proj_at4(z, r, i);
    if (i + 3 >= ff) v.w = 0.f;            // columns beyond ff add nothing to the sums
    if (i + 2 >= ff) v.z = 0.f;
    if (i + 1 >= ff) v.y = 0.f;
    *reinterpret_cast<float4*>(zrow + i) = v;
    add(v.x);
    add(v.y);
    add(v.z);
    add(v.w);
  }
  s2 = block_sum(s2, red);
  s4 = block_sum(s4, red);
  s6 = block_sum(s6, red);
  const float a = coef[0] / sqrtf(s2 / ff + eps), b = coef[1] / sqrtf(s4 / ff + eps), c = coef[2] / sqrtf(s6 / ff + eps);
  const float e = coef[3];
  auto act = [&](float v) { return ((c * v + b) * v + a) * v + e; };
  for (int i = 4 * threadIdx.x; i < ff; i += 4 * blockDim.x) {
    const float4 v = *reinterpret_cast<const float4*>(zrow + i);
    store4(out + 1ll * r * ld_out + i, make_float4(act(v.x), act(v.y), act(v.z), act(v.w)));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) gate_mul_kernel(ds41_proj y, ds41_proj gate, int n, T* out, int ld_out) {
  const int r = blockIdx.y, i = 4 * (blockIdx.x * blockDim.x + threadIdx.x);
  pdl_launch_dependents();
  pdl_wait();
  if (i >= n) return;
  const float4 v = proj_at4(y, r, i), g = proj_at4(gate, r, i);
  store4(out + 1ll * r * ld_out + i, make_float4(v.x * sigmoid_f32(g.x), v.y * sigmoid_f32(g.y), v.z * sigmoid_f32(g.z),
                                                 v.w * sigmoid_f32(g.w)));
}

// one block per (row, head); columns [width, stride) of a head are padding and are written as zeros
template <typename T>
__global__ void __launch_bounds__(128) head_norm_gate_kernel(const float* o, int ld_o, ds41_proj gate, const float* w,
                                                             int width, int stride, float eps, T* out, int ld_out) {
  __shared__ float red[4];
  const int h = blockIdx.x, r = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  const float* src = o + 1ll * r * ld_o + h * stride;
  T* dst = out + 1ll * r * ld_out + h * stride;
  float q = 0.f;
  float4 v0 = make_float4(0.f, 0.f, 0.f, 0.f), g0 = v0, w0 = v0;       // the thread's first piece stays in registers
  for (int i = 4 * threadIdx.x; i < stride; i += 4 * blockDim.x) {
    const float4 v = load4(src + i, width - i);
    if (i < 4 * static_cast<int>(blockDim.x)) {
      v0 = v;
      g0 = proj_at4(gate, r, h * stride + i);
      w0 = load4(w + h * stride + i, width - i);
    }
    q += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  q = warp_sum(q);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = q;
  __syncthreads();
  q = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) q += red[i];
  const float s = 1.0f / sqrtf(q / width + eps);
  for (int i = 4 * threadIdx.x; i < stride; i += 4 * blockDim.x) {
    const bool first = i < 4 * static_cast<int>(blockDim.x);
    const float4 v = first ? v0 : load4(src + i, width - i), ww = first ? w0 : load4(w + h * stride + i, width - i);
    const float4 g = first ? g0 : proj_at4(gate, r, h * stride + i);
    store4(dst + i, make_float4(i < width ? v.x * s * ww.x * sigmoid_f32(g.x) : 0.f,
                                i + 1 < width ? v.y * s * ww.y * sigmoid_f32(g.y) : 0.f,
                                i + 2 < width ? v.z * s * ww.z * sigmoid_f32(g.z) : 0.f,
                                i + 3 < width ? v.w * s * ww.w * sigmoid_f32(g.w) : 0.f));
  }
}

// many (row, head) pairs of at most 512 columns: one warp each
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_warp_kernel(const float* o, int ld_o, ds41_proj gate, const float* w,
                                                                  int items, int heads, int width, int stride, float eps,
                                                                  T* out, int ld_out) {
  const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  if (item >= items) return;
  const int r = item / heads, h = item - r * heads;
  const float* src = o + 1ll * r * ld_o + h * stride;
  T* dst = out + 1ll * r * ld_out + h * stride;
  float4 v[4], g[4];
  float q = 0.f;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int i = 4 * (lane + 32 * k);
    v[k] = g[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < stride) {
      v[k] = load4(src + i, width - i);
      g[k] = proj_at4(gate, r, h * stride + i);
    }
    q += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
  }
  const float s = 1.0f / sqrtf(warp_sum(q) / width + eps);
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int i = 4 * (lane + 32 * k);
    if (i >= stride) break;
    const float4 ww = load4(w + h * stride + i, width - i);
    store4(dst + i, make_float4(i < width ? v[k].x * s * ww.x * sigmoid_f32(g[k].x) : 0.f,
                                i + 1 < width ? v[k].y * s * ww.y * sigmoid_f32(g[k].y) : 0.f,
                                i + 2 < width ? v[k].z * s * ww.z * sigmoid_f32(g[k].z) : 0.f,
                                i + 3 < width ? v[k].w * s * ww.w * sigmoid_f32(g[k].w) : 0.f));
  }
}

// one block per row; columns [n, ld_out) are written as zeros
template <typename T>
__global__ void __launch_bounds__(128) side_act_kernel(ds41_proj z, const int* tokens, const __nv_bfloat16* embed,
                                                       long long embed_ld, int col, int vocab, int n, T* out, int ld_out) {
  const int r = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  const int tok = tokens[r];
  const bool known = tok >= 0 && tok < vocab;
  for (int j = threadIdx.x; j < ld_out; j += blockDim.x) {
    float v = 0.f;
    if (j < n) {
      const float a = proj_at(z, r, j);
      const float e = known ? __bfloat162float(embed[tok * embed_ld + col + j]) : 0.f;
      v = 0.5f * a * (1.0f + tanhf(0.7978845608028654f * (a + 0.044715f * a * a * a))) * e;
    }
    out[1ll * r * ld_out + j] = from_f32<T>(v);
  }
}

__global__ void __launch_bounds__(256) softcap_kernel(float* x, long long n, float cap) {
  const long long i = 1ll * blockIdx.x * blockDim.x + threadIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  if (i < n) x[i] = cap * tanhf(x[i] / cap);
}

template <typename T>
__global__ void __launch_bounds__(256) gather_rows_kernel(const T* src, int ld, const int* index, int n_src, int W, T* dst) {
  const int r = blockIdx.y, i = blockIdx.x * blockDim.x + threadIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  if (i >= W) return;
  const int s = index[r];
  dst[1ll * r * ld + i] = s >= 0 && s < n_src ? src[1ll * s * ld + i] : from_f32<T>(0.f);
}

template <typename T, int CL, int NI>
static cudaError_t launch_resid_ni(const ds41_resid_args& a, int threads, cudaStream_t st) {
  if constexpr (CL == 1) return launch_pdl(resid_step_kernel<T, CL, NI>, dim3(a.rows), dim3(threads), 0, st, a);
  else return launch_pdl_cluster(resid_step_kernel<T, CL, NI>, dim3(a.rows * CL), dim3(threads), CL, 0, st, a);
}

template <typename T, int CL>
static cudaError_t launch_resid(const ds41_resid_args& a, cudaStream_t st) {
  const int pieces = ((a.W + CL - 1) / CL + 3) / 4;
  const auto width = [&](int ni) { return ((pieces + ni - 1) / ni + 31) / 32 * 32; };
  constexpr int kMost = CL == 8 ? 128 : 256;        // the moments of a cluster's warps fit one warp
  if (width(1) <= kMost) return launch_resid_ni<T, CL, 1>(a, width(1), st);
  if (width(2) <= kMost) return launch_resid_ni<T, CL, 2>(a, width(2), st);
  if (width(4) <= kMost) return launch_resid_ni<T, CL, 4>(a, width(4), st);
  if (width(8) <= (CL == 8 ? 128 : 512)) return launch_resid_ni<T, CL, 8>(a, width(8), st);
  return cudaErrorInvalidValue;
}

}  // namespace ds41

using namespace ds41;

extern "C" int ds41_resid_step(const ds41_resid_args* a, void* stream) {
  if (a == nullptr || a->rows <= 0 || a->W <= 0 || a->ldx < a->W) return cudaErrorInvalidValue;
  if (a->tokens != nullptr ? (a->embed == nullptr || a->embed_ld < a->W || a->vocab <= 0) : a->x_in == nullptr)
    return cudaErrorInvalidValue;
  if (a->y.data != nullptr && !proj_ok(a->y)) return cudaErrorInvalidValue;
  if (a->gate.data != nullptr && (!proj_ok(a->gate) || a->gate_bias == nullptr)) return cudaErrorInvalidValue;
  if (a->mix != nullptr && (a->n_mix < 1 || (a->n_mix > 1 && a->kept == nullptr))) return cudaErrorInvalidValue;
  if (a->y_route != nullptr && (a->y.data == nullptr || a->y_top <= 0 || a->y_rows < 0)) return cudaErrorInvalidValue;
  if ((a->next_w != nullptr || a->raw_h) && (a->h == nullptr || a->ldh < a->W || (a->ldh & 3))) return cudaErrorInvalidValue;
  // rows are walked in pieces of four columns
  if ((a->ldx & 3) || (a->kept_stride & 3) || (a->tokens != nullptr && (a->embed_ld & 3)) ||
      (a->y.data != nullptr && !proj_vec4(a->y)) || (a->gate.data != nullptr && !proj_vec4(a->gate)))
    return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  // few rows: a cluster of eight CTAs shares a row, so that its loads do not queue on one SM
  const bool wide = (a->rows <= 32 && a->W >= 1024) || a->W > 16384;
  if (a->f32) return wide ? launch_resid<float, 8>(*a, st) : launch_resid<float, 1>(*a, st);
  return wide ? launch_resid<__nv_bfloat16, 8>(*a, st) : launch_resid<__nv_bfloat16, 1>(*a, st);
}

template <typename T>
static int launch_polynorm(const ds41_proj& z, const float* coef, int rows, int ff, int ld_out, float eps, void* out,
                           cudaStream_t st) {
  const size_t smem = (1ull * ff + 3) / 4 * 16;
  static size_t allowed = 48 * 1024 - 512;
  if (smem > allowed) {
    if (smem > 226 * 1024) return cudaErrorInvalidValue;
    const cudaError_t e = cudaFuncSetAttribute(polynorm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem));
    if (e != cudaSuccess) return e;
    allowed = smem;
  }
  return launch_pdl(polynorm_kernel<T>, dim3(rows), dim3(ff >= 2048 ? 512 : 256), smem, st, z, coef, ff, ld_out, eps,
                    static_cast<T*>(out));
}

extern "C" int ds41_polynorm(const ds41_proj* z, const float* coef, int rows, int ff, float eps, void* out, int ld_out,
                             int f32, void* stream) {
  if (z == nullptr || !proj_ok(*z) || !proj_vec4(*z) || coef == nullptr || out == nullptr || rows <= 0 || ff <= 0 ||
      ld_out < ff || (ld_out & 3) || z->ld < z->col + (ff + 3) / 4 * 4)
    return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_polynorm<float>(*z, coef, rows, ff, ld_out, eps, out, st)
             : launch_polynorm<__nv_bfloat16>(*z, coef, rows, ff, ld_out, eps, out, st);
}

extern "C" int ds41_gate_mul(const ds41_proj* y, const ds41_proj* gate, int rows, int n, void* out, int ld_out, int f32,
                             void* stream) {
  if (y == nullptr || gate == nullptr || !proj_ok(*y) || !proj_ok(*gate) || out == nullptr || rows <= 0 || n <= 0 ||
      ld_out < n || rows > 65535 || (n & 3) || (ld_out & 3) || !proj_vec4(*y) || !proj_vec4(*gate))
    return cudaErrorInvalidValue;
  const dim3 grid((n + 1023) / 1024, rows);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) return launch_pdl(gate_mul_kernel<float>, grid, dim3(256), 0, st, *y, *gate, n, static_cast<float*>(out), ld_out);
  return launch_pdl(gate_mul_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, *y, *gate, n,
                    static_cast<__nv_bfloat16*>(out), ld_out);
}

extern "C" int ds41_head_norm_gate(const float* o, int ld_o, const ds41_proj* gate, const float* w, int rows, int heads,
                                   int width, int stride, float eps, void* out, int ld_out, int f32, void* stream) {
  if (o == nullptr || gate == nullptr || !proj_ok(*gate) || w == nullptr || out == nullptr || rows <= 0 || heads <= 0 ||
      width <= 0 || stride < width || (stride & 3) || ld_o < heads * stride || (ld_o & 3) || ld_out < heads * stride ||
      (ld_out & 3) || !proj_vec4(*gate) || rows > 65535)
    return cudaErrorInvalidValue;
  const dim3 grid(heads, rows), block(stride >= 512 ? 128 : (stride + 127) / 128 * 32);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (stride <= 512 && rows * heads >= 1024) {
    const dim3 warps((rows * heads + 7) / 8);
    if (f32)
      return launch_pdl(head_norm_gate_warp_kernel<float>, warps, dim3(256), 0, st, o, ld_o, *gate, w, rows * heads, heads,
                        width, stride, eps, static_cast<float*>(out), ld_out);
    return launch_pdl(head_norm_gate_warp_kernel<__nv_bfloat16>, warps, dim3(256), 0, st, o, ld_o, *gate, w, rows * heads,
                      heads, width, stride, eps, static_cast<__nv_bfloat16*>(out), ld_out);
  }
  if (f32)
    return launch_pdl(head_norm_gate_kernel<float>, grid, block, 0, st, o, ld_o, *gate, w, width, stride, eps,
                      static_cast<float*>(out), ld_out);
  return launch_pdl(head_norm_gate_kernel<__nv_bfloat16>, grid, block, 0, st, o, ld_o, *gate, w, width, stride, eps,
                    static_cast<__nv_bfloat16*>(out), ld_out);
}

extern "C" int ds41_side_act(const ds41_proj* z, const int* tokens, const void* embed, long long embed_ld, int col, int vocab,
                             int rows, int n, void* out, int ld_out, int f32, void* stream) {
  if (z == nullptr || !proj_ok(*z) || tokens == nullptr || embed == nullptr || out == nullptr || rows <= 0 || n <= 0 ||
      ld_out < n || col < 0 || embed_ld < col + n || vocab <= 0 || z->ld < z->col + n)
    return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const __nv_bfloat16* e = static_cast<const __nv_bfloat16*>(embed);
  if (f32)
    return launch_pdl(side_act_kernel<float>, dim3(rows), dim3(128), 0, st, *z, tokens, e, embed_ld, col, vocab, n,
                      static_cast<float*>(out), ld_out);
  return launch_pdl(side_act_kernel<__nv_bfloat16>, dim3(rows), dim3(128), 0, st, *z, tokens, e, embed_ld, col, vocab, n,
                    static_cast<__nv_bfloat16*>(out), ld_out);
}

extern "C" int ds41_softcap_rows(float* x, long long n, float cap, void* stream) {
  if (x == nullptr || n <= 0 || !(cap > 0.f) || (n + 255) / 256 > 0x7fffffffll) return cudaErrorInvalidValue;
  return launch_pdl(softcap_kernel, dim3(static_cast<unsigned>((n + 255) / 256)), dim3(256), 0,
                    static_cast<cudaStream_t>(stream), x, n, cap);
}

extern "C" int ds41_gather_rows(const void* src, int ld, const int* index, int n_src, int rows, int W, void* dst, int f32,
                                void* stream) {
  if (src == nullptr || index == nullptr || dst == nullptr || rows <= 0 || W <= 0 || ld < W || rows > 65535)
    return cudaErrorInvalidValue;
  const dim3 grid((W + 255) / 256, rows);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return launch_pdl(gather_rows_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(src), ld, index, n_src,
                      W, static_cast<float*>(dst));
  return launch_pdl(gather_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(src), ld,
                    index, n_src, W, static_cast<__nv_bfloat16*>(dst));
}
