// Row-wise steps of a layer stack whose residual stream is one fp32 row per token.
//
//  resid_step    : closes a sublayer and opens the next one.  result -> sigmoid gate -> norm -> added to the stream;
//                  optionally the stream becomes a weighted sum of the kept streams of all layers so far (depth average);
//                  then the norm that feeds the next sublayer.  With `tokens` the stream starts from the embedding.
//  polynorm      : activation a N(z) + b N(z^2) + c N(z^3) + e, N = division by the row's root mean square
//  gate_mul      : result x sigmoid(gate)
//  head_norm_gate: per-head RMS norm x weight x sigmoid(gate)
//  gather_rows   : picks rows of an activation matrix by index
#include <cooperative_groups.h>

#include "ds41_stack.cuh"

namespace ds41 {

namespace cg = cooperative_groups;

// (mean, sum of squared deviations, count) of the part of a row that one CTA holds, merged over the CTAs of a cluster
struct Moments {
  float mean, m2, n;
};

template <int CL>
__device__ __forceinline__ Moments merge_moments(Moments own, float* slot) {
  if constexpr (CL == 1) {
    return own;
  } else {
    cg::cluster_group cluster = cg::this_cluster();
    if (threadIdx.x == 0) {
      slot[0] = own.mean;
      slot[1] = own.m2;
      slot[2] = own.n;
    }
    cluster.sync();
    Moments t{0.f, 0.f, 0.f};
#pragma unroll
    for (int c = 0; c < CL; ++c) {        // the same order in every CTA: all of them get the same numbers
      const float* s = cluster.map_shared_rank(slot, c);
      const float mean = s[0], m2 = s[1], n = s[2];
      if (n == 0.f) continue;
      const float total = t.n + n, d = mean - t.mean;
      t.mean += d * (n / total);
      t.m2 += m2 + d * d * (t.n * n / total);
      t.n = total;
    }
    return t;
  }
}

// Subtrahend and factor of a row's norm - layer norm (subtract the mean) or RMS norm (mean of squares) - from the pieces of
// four columns that the threads hold; `n` columns of the row are in this CTA, piece i covers columns 4 (tid + i blockDim).
template <int CL, int NI>
__device__ __forceinline__ float2 row_norm(const float4 (&v)[NI], int n, int W, int kind, float eps, float* red, float* slot) {
  float mean = 0.f;
  if (kind == 0) {
    float s = 0.f;                       // columns beyond the row hold zeros
#pragma unroll
    for (int i = 0; i < NI; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    mean = n > 0 ? block_sum(s, red) / n : 0.f;
  }
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int live = n - 4 * (threadIdx.x + i * blockDim.x);
    const float a = v[i].x - mean, b = v[i].y - mean, c = v[i].z - mean, d = v[i].w - mean;
    q += (live > 0 ? a * a : 0.f) + (live > 1 ? b * b : 0.f) + (live > 2 ? c * c : 0.f) + (live > 3 ? d * d : 0.f);
  }
  q = block_sum(q, red);
  // the means of squares add up: an RMS norm goes through the same exchange with zero means
  const Moments t = merge_moments<CL>({mean, q, static_cast<float>(n)}, slot);
  return make_float2(t.mean, 1.0f / sqrtf(t.m2 / W + eps));
}

template <typename T, int CL, int NI>
__global__ void __launch_bounds__(CL == 1 && NI <= 4 ? 256 : 1024) resid_step_kernel(ds41_resid_args p) {
  __shared__ float red[33];
  __shared__ float slots[2][3];
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
        y[i] = proj_at4(p.y, r, c0 + at[i]);
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
    if (p.post_w != nullptr) s = row_norm<CL, NI>(y, n, p.W, p.norm_kind, p.eps, red, slots[0]);
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
    // weighted sum of the kept streams; the newest one is the row this block holds
    const float* k0 = p.kept + r * p.ldx + c0;
    const float last = p.mix[p.n_mix - 1];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      x[i].x *= last;
      x[i].y *= last;
      x[i].z *= last;
      x[i].w *= last;
    }
#pragma unroll 4
    for (int j = 0; j < p.n_mix - 1; ++j) {
      const float c = p.mix[j];
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (live[i] > 0) {
          const float4 k = *reinterpret_cast<const float4*>(k0 + j * p.kept_stride + at[i]);
          x[i].x += c * k.x;
          x[i].y += c * k.y;
          x[i].z += c * k.z;
          x[i].w += c * k.w;
        }
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) clip(x[i], i);
    if (p.x_avg != nullptr) {
      float* o = p.x_avg + r * p.ldx + c0;
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (live[i] > 0) store4(o + at[i], x[i]);
    }
  }
  if (p.next_w != nullptr) {
    const float2 s = row_norm<CL, NI>(x, n, p.W, p.norm_kind, p.eps, red, slots[1]);
    T* h = static_cast<T*>(p.h) + 1ll * r * p.ldh + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (live[i] > 0) {
        const float4 w = load4(p.next_w + c0 + at[i], live[i]);
        store4(h + at[i], make_float4((x[i].x - s.x) * s.y * w.x, (x[i].y - s.x) * s.y * w.y, (x[i].z - s.x) * s.y * w.z,
                                      (x[i].w - s.x) * s.y * w.w));
      }
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
  const int r = blockIdx.y, i = blockIdx.x * blockDim.x + threadIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  if (i < n) out[1ll * r * ld_out + i] = from_f32<T>(proj_at(y, r, i) * sigmoid_f32(proj_at(gate, r, i)));
}

// one warp per (row, head); columns [width, stride) of a head are padding and are written as zeros
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* o, int ld_o, ds41_proj gate, const float* w,
                                                             int rows, int heads, int width, int stride, float eps,
                                                             T* out, int ld_out) {
  const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  if (item >= rows * heads) return;
  const int r = item / heads, h = item - r * heads;
  const float* src = o + 1ll * r * ld_o + h * stride;
  float q = 0.f;
  for (int i = lane; i < width; i += 32) q += src[i] * src[i];
  const float s = 1.0f / sqrtf(warp_sum(q) / width + eps);
  T* dst = out + 1ll * r * ld_out + h * stride;
  for (int i = lane; i < stride; i += 32) {
    const int c = h * stride + i;
    dst[i] = i < width ? from_f32<T>(src[i] * s * w[c] * sigmoid_f32(proj_at(gate, r, c))) : from_f32<T>(0.f);
  }
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
  if (width(1) <= 256) return launch_resid_ni<T, CL, 1>(a, width(1), st);
  if (width(2) <= 256) return launch_resid_ni<T, CL, 2>(a, width(2), st);
  if (width(4) <= 256) return launch_resid_ni<T, CL, 4>(a, width(4), st);
  if (width(8) <= 1024) return launch_resid_ni<T, CL, 8>(a, width(8), st);
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
  if (a->next_w != nullptr && (a->h == nullptr || a->ldh < a->W || (a->ldh & 3))) return cudaErrorInvalidValue;
  // rows are walked in pieces of four columns
  if ((a->ldx & 3) || (a->kept_stride & 3) || (a->tokens != nullptr && (a->embed_ld & 3)) ||
      (a->y.data != nullptr && !proj_vec4(a->y)) || (a->gate.data != nullptr && !proj_vec4(a->gate)))
    return cudaErrorInvalidValue;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  // few rows: a cluster of eight CTAs shares a row, so that its loads do not queue on one SM
  const bool wide = a->rows <= 32 && a->W >= 1024;
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
      ld_out < n || rows > 65535)
    return cudaErrorInvalidValue;
  const dim3 grid((n + 255) / 256, rows);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) return launch_pdl(gate_mul_kernel<float>, grid, dim3(256), 0, st, *y, *gate, n, static_cast<float*>(out), ld_out);
  return launch_pdl(gate_mul_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, *y, *gate, n,
                    static_cast<__nv_bfloat16*>(out), ld_out);
}

extern "C" int ds41_head_norm_gate(const float* o, int ld_o, const ds41_proj* gate, const float* w, int rows, int heads,
                                   int width, int stride, float eps, void* out, int ld_out, int f32, void* stream) {
  if (o == nullptr || gate == nullptr || !proj_ok(*gate) || w == nullptr || out == nullptr || rows <= 0 || heads <= 0 ||
      width <= 0 || stride < width || ld_o < heads * stride || ld_out < heads * stride)
    return cudaErrorInvalidValue;
  const dim3 grid((rows * heads + 7) / 8);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return launch_pdl(head_norm_gate_kernel<float>, grid, dim3(256), 0, st, o, ld_o, *gate, w, rows, heads, width, stride,
                      eps, static_cast<float*>(out), ld_out);
  return launch_pdl(head_norm_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, o, ld_o, *gate, w, rows, heads, width,
                    stride, eps, static_cast<__nv_bfloat16*>(out), ld_out);
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
