// Kernels of decoders that keep the residual stream in fp32 (independent of the activation type T, bf16 or fp32):
//
//   embed_norm           x = scale * E[token] (+ sinusoid(position));    h = T(rms_g(x) * w)
//   residual_norm        x += rms(y) * w_out;                            h = T(rms(x) * w_next)
//   residual_add_norm    x += mult * (y + sum of expert outputs);        h = T(rms_g(x) * w_next)
//   streams_norm         x_t <- sum_s mix[s][t] x_s + out[t] * y;        h = T(rms_g(sum_t in[t] x_t) * w_next)
//
// with rms(v) = v / sqrt(mean(v^2) + eps), and rms_g the same over each of `groups` equal consecutive parts of the vector.
// embed_norm and residual_norm also exist with layer norms, (v - mean) / sqrt(variance + eps), in the place of rms, and both can
// add a vector to the residual in front of the last norm; residual_norm also the scaled embedding, which makes it the seam
// between two passes of a range of layers that runs several times.
// residual_norm is the whole seam between two sublayers of a layer with a norm before and after each sublayer: y is the
// sublayer's output projection, w_out the product of the output norm's weight and the layer scale, w_next the weight of the
// norm that feeds the next projection.  residual_add_norm is the seam between two layers whose mixer and feed-forward run
// in parallel from one norm: y holds the sum of their output projections, and the outputs of a mixture of experts are
// gathered from the experts' token lists on the way.  streams_norm is the seam of hyper-connections: the residual is a small
// number of streams that a sublayer reads through one set of weights and writes through another.
//
// Rows are padded: `ld` columns (a multiple of 64) of which the first `width` are real; padding columns of every operand
// are zero, so only the mean knows the difference.
//
//   few_linear      z[t, f] = x[t, :] . w[f, :] + b[f] in fp32 for a handful of features (gate pre-activations that
//                   enter a recurrence), where a GEMM with a 16-bit output would round them
//   gemm_f32        plain fp32 matrix product for the 32-bit mode
//   rotary_table    cosines and sines of the rotary positions of a step
#include "common.cuh"

namespace tahb {

template <typename T> struct Vec4;
template <> struct Vec4<float> {
  static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Vec4<__nv_bfloat16> {
  static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
    uint2 u;
    *reinterpret_cast<__nv_bfloat162*>(&u.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&u.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = u;
  }
};

constexpr int RN_THREADS = 128;

__device__ __forceinline__ float block_sum_128(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();                       // red may still be read from the previous use
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  return red[0] + red[1] + red[2] + red[3];
}

__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// Inverse root mean squares of the `groups` parts of a row whose vectors c = threadIdx.x + i * RN_THREADS sit in v[i]; r[i]
// receives the factor of each element of vector i (0 in the padding).  Parts of whole 128-element warp blocks (real model
// sizes, one group included) are summed by warp shuffles, any other size through the row in shared memory.
// sm: 64 + groups floats, and ld more when the part size is not a multiple of 128.
template <int VPT>
__device__ __forceinline__ void group_inv_rms(const float4* v, int width, int groups, int ld, float eps, float* sm, float4* r) {
  const int gs = width / groups, nvec = ld / 4, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* inv = sm + 64;
  if (gs % 128 == 0) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const float s = warp_sum(threadIdx.x + i * RN_THREADS < nvec ? sq4(v[i]) : 0.f);
      if (lane == 0) sm[i * 4 + warp] = s;                  // elements 128 (4 i + warp) ..
    }
    __syncthreads();
    const int per = gs / 128;
    for (int g = threadIdx.x; g < groups; g += RN_THREADS) {
      float s = 0.f;
      for (int k = 0; k < per; ++k) s += sm[g * per + k];
      inv[g] = 1.0f / sqrtf(s / (float)gs + eps);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int g = (i * 4 + warp) / per;
      const float f = g < groups ? inv[g] : 0.f;
      r[i] = make_float4(f, f, f, f);
    }
    return;
  }
  float* row = inv + groups;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      row[4 * c] = v[i].x; row[4 * c + 1] = v[i].y; row[4 * c + 2] = v[i].z; row[4 * c + 3] = v[i].w;
    }
  }
  __syncthreads();
  for (int g = warp; g < groups; g += RN_THREADS / 32) {
    float s = 0.f;
    for (int k = lane; k < gs; k += 32) s = fmaf(row[g * gs + k], row[g * gs + k], s);
    s = warp_sum(s);
    if (lane == 0) inv[g] = 1.0f / sqrtf(s / (float)gs + eps);
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = 4 * (threadIdx.x + i * RN_THREADS);
    auto at = [&](int e) { return e < width ? inv[e / gs] : 0.f; };
    r[i] = make_float4(at(c), at(c + 1), at(c + 2), at(c + 3));
  }
}

// Mean and inverse standard deviation of a row whose vectors c = threadIdx.x + i * RN_THREADS sit in v[i]; the deviations of its
// `width` real elements are squared after the mean is known.
template <int VPT>
__device__ __forceinline__ float2 row_moments(const float4* v, int width, int nvec, float eps, float* red) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (threadIdx.x + i * RN_THREADS < nvec) s += v[i].x + v[i].y + v[i].z + v[i].w;
  const float mean = block_sum_128(s, red) / (float)width;
  s = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = 4 * (threadIdx.x + i * RN_THREADS);
    if (c < width) s += (v[i].x - mean) * (v[i].x - mean);
    if (c + 1 < width) s += (v[i].y - mean) * (v[i].y - mean);
    if (c + 2 < width) s += (v[i].z - mean) * (v[i].z - mean);
    if (c + 3 < width) s += (v[i].w - mean) * (v[i].w - mean);
  }
  return make_float2(mean, 1.0f / sqrtf(block_sum_128(s, red) / (float)width + eps));
}

// (mean or 0, factor) of one of the two norms
template <int VPT, bool CENTER>
__device__ __forceinline__ float2 row_norm(const float4* v, int width, int nvec, float eps, float* red) {
  if constexpr (CENTER) return row_moments<VPT>(v, width, nvec, eps, red);
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i)
    if (threadIdx.x + i * RN_THREADS < nvec) s += sq4(v[i]);
  return make_float2(0.f, 1.0f / sqrtf(block_sum_128(s, red) / (float)width + eps));
}

static size_t group_rms_smem(int width, int groups, int ld) {
  return (64 + (size_t)groups + ((width / groups) % 128 ? ld : 0)) * 4;
}

// Sine and cosine of p * f for the pair of entries (2 i, 2 i + 1); f = hi + lo, and the rounding error e of the angle (4e-3 at
// position 70,000) goes into the result by the Taylor terms up to e^2.
__device__ __forceinline__ float2 sin_cos_pair(float p, float hi, float lo) {
  const float a = p * hi, e = fmaf(p, lo, fmaf(p, hi, -a));
  float s, c;
  sincosf(a, &s, &c);
  return make_float2(fmaf(e, fmaf(-0.5f * e, s, c), s), fmaf(-e, fmaf(0.5f * e, c, s), c));
}

// pos / freq: position of every token and [2, (width + 1) / 2] frequencies (high parts, then low parts), or null.
// streams copies of the embedding go to x [M, streams, ld]; w_in [streams]: weights of their sum, which is what the norm
// sees (null: one stream as it is).  add [ld]: vector added to the scaled embedding (zero in the padding), or null.  CENTER: layer
// norm (groups is 1).
template <typename T, int VPT, bool CENTER>
__global__ void __launch_bounds__(RN_THREADS) embed_norm_kernel(const T* __restrict__ E, const int* __restrict__ tok,
                                                                float scale, const int* __restrict__ pos,
                                                                const float* __restrict__ freq, int streams, const float* __restrict__ w_in,
                                                                const float* __restrict__ add, float* __restrict__ x, const float* __restrict__ w,
                                                                T* __restrict__ h, int vocab, int width, int groups, int ld,
                                                                float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float gsm[];
  const size_t row = blockIdx.x;
  const int id = min(max(tok[row], 0), vocab - 1);
  const int nvec = ld / 4;
  float sum_in = 1.0f;
  if (w_in != nullptr) {
    sum_in = 0.f;
    for (int s = 0; s < streams; ++s) sum_in += w_in[s];
  }
  float4 v[VPT], r[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      v[i] = Vec4<T>::load(E + (size_t)id * ld + c * 4);
      v[i].x *= scale; v[i].y *= scale; v[i].z *= scale; v[i].w *= scale;
      if (freq != nullptr) {
        const float p = (float)pos[row];
        const float* lo = freq + (width + 1) / 2;
        if (4 * c < width) {
          const float2 a = sin_cos_pair(p, freq[2 * c], lo[2 * c]);
          v[i].x += a.x;
          if (4 * c + 1 < width) v[i].y += a.y;
        }
        if (4 * c + 2 < width) {
          const float2 a = sin_cos_pair(p, freq[2 * c + 1], lo[2 * c + 1]);
          v[i].z += a.x;
          if (4 * c + 3 < width) v[i].w += a.y;
        }
      }
      if (add != nullptr) {
        const float4 a = Vec4<float>::load(add + c * 4);
        v[i].x += a.x; v[i].y += a.y; v[i].z += a.z; v[i].w += a.w;
      }
      for (int s = 0; s < streams; ++s) Vec4<float>::store(x + (row * streams + s) * ld + c * 4, v[i]);
      v[i].x *= sum_in; v[i].y *= sum_in; v[i].z *= sum_in; v[i].w *= sum_in;
    }
  }
  if constexpr (CENTER) {
    const float2 n = row_moments<VPT>(v, width, nvec, eps, gsm);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      v[i].x -= n.x; v[i].y -= n.x; v[i].z -= n.x; v[i].w -= n.x;
      r[i] = make_float4(n.y, n.y, n.y, n.y);
    }
  } else {
    group_inv_rms<VPT>(v, width, groups, ld, eps, gsm, r);
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      const float4 g = Vec4<float>::load(w + c * 4);
      Vec4<T>::store(h + row * ld + c * 4,
                     make_float4(v[i].x * r[i].x * g.x, v[i].y * r[i].y * g.y, v[i].z * r[i].z * g.z, v[i].w * r[i].w * g.w));
    }
  }
}

// y_ex / slot: expert outputs [list rows, ld] and the list rows slot[row * top ..] of this token, or null
template <typename T, int VPT>
__global__ void __launch_bounds__(RN_THREADS) residual_add_norm_kernel(const T* __restrict__ y, long long ldy,
                                                                       const T* __restrict__ y_ex,
                                                                       const int* __restrict__ slot, int top, float mult,
                                                                       float* __restrict__ x, const float* __restrict__ w_next,
                                                                       T* __restrict__ h, int width, int groups, int ld,
                                                                       float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float gsm[];
  const size_t row = blockIdx.x;
  const int nvec = ld / 4;
  float4 v[VPT], r[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) r[i] = Vec4<T>::load(y + row * ldy + c * 4);
  }
  if (y_ex != nullptr) {
    for (int j = 0; j < top; ++j) {
      const T* src = y_ex + (size_t)slot[row * top + j] * ld;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * RN_THREADS;
        if (c < nvec) {
          const float4 e = Vec4<T>::load(src + c * 4);
          r[i].x += e.x; r[i].y += e.y; r[i].z += e.z; r[i].w += e.w;
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      v[i] = Vec4<float>::load(x + row * ld + c * 4);
      v[i].x = fmaf(mult, r[i].x, v[i].x); v[i].y = fmaf(mult, r[i].y, v[i].y);
      v[i].z = fmaf(mult, r[i].z, v[i].z); v[i].w = fmaf(mult, r[i].w, v[i].w);
      Vec4<float>::store(x + row * ld + c * 4, v[i]);
    }
  }
  group_inv_rms<VPT>(v, width, groups, ld, eps, gsm, r);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      const float4 g = Vec4<float>::load(w_next + c * 4);
      Vec4<T>::store(h + row * ld + c * 4,
                     make_float4(v[i].x * r[i].x * g.x, v[i].y * r[i].y * g.y, v[i].z * r[i].z * g.z, v[i].w * r[i].w * g.w));
    }
  }
}

// Hyper-connections.  hc: mix [S][S] (from, to), out [S], then the next reader's in [S].  y_bias [ld] (zero in the padding)
// or null; y_ex / slot / y_weight: expert outputs [list rows, ld], list rows and weights [M, top], or null.  Every element of
// the streams is read and written once.
struct StreamsParams {
  const void* y;
  long long ldy;
  const float* y_bias;
  const void* y_ex;
  const int* slot;
  const float* y_weight;
  int top;
  float* x;                   // [M, S, ld]
  const float* hc;
  const float* w_next;
  void* h;
  int width, groups, ld;
  float eps;
};

template <typename T, int VPT, int S>
__global__ void __launch_bounds__(RN_THREADS) streams_norm_kernel(const StreamsParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float gsm[];
  const size_t row = blockIdx.x;
  const int nvec = p.ld / 4;
  const T* y = reinterpret_cast<const T*>(p.y) + row * p.ldy;
  float4 v[VPT], r[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    r[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < nvec && p.y != nullptr) r[i] = Vec4<T>::load(y + c * 4);
    if (c < nvec && p.y_bias != nullptr) {
      const float4 b = Vec4<float>::load(p.y_bias + c * 4);
      r[i].x += b.x; r[i].y += b.y; r[i].z += b.z; r[i].w += b.w;
    }
  }
  if (p.y_ex != nullptr) {
    for (int j = 0; j < p.top; ++j) {
      const T* src = reinterpret_cast<const T*>(p.y_ex) + (size_t)p.slot[row * p.top + j] * p.ld;
      const float w = p.y_weight != nullptr ? p.y_weight[row * p.top + j] : 1.0f;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * RN_THREADS;
        if (c < nvec) {
          const float4 e = Vec4<T>::load(src + c * 4);
          r[i].x = fmaf(w, e.x, r[i].x); r[i].y = fmaf(w, e.y, r[i].y);
          r[i].z = fmaf(w, e.z, r[i].z); r[i].w = fmaf(w, e.w, r[i].w);
        }
      }
    }
  }
  float mix[S][S], out[S], in[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = __ldg(p.hc + s * S + t);
    out[s] = __ldg(p.hc + S * S + s);
    in[s] = __ldg(p.hc + S * S + S + s);
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < nvec) {
      float* x = p.x + row * S * p.ld + c * 4;
      float4 old[S];
#pragma unroll
      for (int s = 0; s < S; ++s) old[s] = Vec4<float>::load(x + (size_t)s * p.ld);
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float4 n = make_float4(out[t] * r[i].x, out[t] * r[i].y, out[t] * r[i].z, out[t] * r[i].w);
#pragma unroll
        for (int s = 0; s < S; ++s) {
          n.x = fmaf(mix[s][t], old[s].x, n.x); n.y = fmaf(mix[s][t], old[s].y, n.y);
          n.z = fmaf(mix[s][t], old[s].z, n.z); n.w = fmaf(mix[s][t], old[s].w, n.w);
        }
        Vec4<float>::store(x + (size_t)t * p.ld, n);
        v[i].x = fmaf(in[t], n.x, v[i].x); v[i].y = fmaf(in[t], n.y, v[i].y);
        v[i].z = fmaf(in[t], n.z, v[i].z); v[i].w = fmaf(in[t], n.w, v[i].w);
      }
    }
  }
  group_inv_rms<VPT>(v, p.width, p.groups, p.ld, p.eps, gsm, r);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      const float4 g = Vec4<float>::load(p.w_next + c * 4);
      Vec4<T>::store(reinterpret_cast<T*>(p.h) + row * p.ld + c * 4,
                     make_float4(v[i].x * r[i].x * g.x, v[i].y * r[i].y * g.y, v[i].z * r[i].z * g.z, v[i].w * r[i].w * g.w));
    }
  }
}

// out[t][i] = mscale * (cos, sin) of pos[t] * f_i; freq: [2, half] high parts, then low parts
__global__ void rotary_table_kernel(const int* __restrict__ pos, const float* __restrict__ freq, float mscale,
                                    float2* __restrict__ out, int M, int half) {
  pdl_launch_dependents();
  pdl_wait();
  const int n = M * half;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
    const float2 a = sin_cos_pair((float)pos[i / half], freq[i % half], freq[half + i % half]);
    out[i] = make_float2(mscale * a.y, mscale * a.x);
  }
}

struct ResidualNormParams {
  const void* y;              // [M, ldy]
  long long ldy;
  float* x;                   // [M, ld]
  const float* w_out;
  const float* w_next;
  void* h;                    // [M, ld]
  int width, ld;
  float eps;
  const float* add;           // [ld] added to the residual behind the sublayer's sum, or null
  const void* E;              // embedding table [vocab, ld] whose rows, times scale, are added too, or null
  const int* tok;             // [M], with E
  int vocab;
  float scale;
  float* before;              // [M, ld] receives the residual as it is before these two, or null
};

// CENTER: layer norms; ENTER: add / E / before may be given
template <typename T, int VPT, bool CENTER, bool ENTER>
__global__ void __launch_bounds__(RN_THREADS) residual_norm_kernel(const ResidualNormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[4];
  const size_t row = blockIdx.x;
  const int nvec = p.ld / 4;
  const T* y = reinterpret_cast<const T*>(p.y) + row * p.ldy;
  float* x = p.x + row * p.ld;
  float4 u[VPT], v[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      u[i] = Vec4<T>::load(y + c * 4);
      v[i] = Vec4<float>::load(x + c * 4);
    }
  }
  const float2 ny = row_norm<VPT, CENTER>(u, p.width, nvec, p.eps, red);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      const float4 g = Vec4<float>::load(p.w_out + c * 4);
      if constexpr (CENTER) { u[i].x -= ny.x; u[i].y -= ny.x; u[i].z -= ny.x; u[i].w -= ny.x; }
      v[i].x += u[i].x * ny.y * g.x; v[i].y += u[i].y * ny.y * g.y; v[i].z += u[i].z * ny.y * g.z; v[i].w += u[i].w * ny.y * g.w;
      if constexpr (ENTER) {
        if (p.before != nullptr) Vec4<float>::store(p.before + row * p.ld + c * 4, v[i]);
        if (p.E != nullptr) {
          const int id = min(max(p.tok[row], 0), p.vocab - 1);
          const float4 e = Vec4<T>::load(reinterpret_cast<const T*>(p.E) + (size_t)id * p.ld + c * 4);
          v[i].x = fmaf(p.scale, e.x, v[i].x); v[i].y = fmaf(p.scale, e.y, v[i].y);
          v[i].z = fmaf(p.scale, e.z, v[i].z); v[i].w = fmaf(p.scale, e.w, v[i].w);
        }
        if (p.add != nullptr) {
          const float4 a = Vec4<float>::load(p.add + c * 4);
          v[i].x += a.x; v[i].y += a.y; v[i].z += a.z; v[i].w += a.w;
        }
      }
      Vec4<float>::store(x + c * 4, v[i]);
    }
  }
  const float2 nx = row_norm<VPT, CENTER>(v, p.width, nvec, p.eps, red);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c < nvec) {
      const float4 g = Vec4<float>::load(p.w_next + c * 4);
      if constexpr (CENTER) { v[i].x -= nx.x; v[i].y -= nx.x; v[i].z -= nx.x; v[i].w -= nx.x; }
      Vec4<T>::store(reinterpret_cast<T*>(p.h) + row * p.ld + c * 4,
                     make_float4(v[i].x * nx.y * g.x, v[i].y * nx.y * g.y, v[i].z * nx.y * g.z, v[i].w * nx.y * g.w));
    }
  }
}

// ---------------------------------------------------------------------------------------------
// few_linear: grid (ceil(M / FL_TOK)); the rows of FL_TOK tokens sit in shared memory as fp32, one warp per feature and
// step.  A weight row is read once per FL_TOK tokens.
// ---------------------------------------------------------------------------------------------
constexpr int FL_THREADS = 256;

template <typename T, int TOK>
__global__ void __launch_bounds__(FL_THREADS) few_linear_kernel(const T* __restrict__ x, long long ldx,
                                                                const T* __restrict__ w, const float* __restrict__ b,
                                                                float* __restrict__ out, int M, int K, int F) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float xs[];              // [TOK][K]
  const int t0 = blockIdx.x * TOK, n = min(TOK, M - t0);
  const int nvec = K / 4;
  for (int i = threadIdx.x; i < TOK * nvec; i += FL_THREADS) {
    const int r = i / nvec, c = i % nvec;
    Vec4<float>::store(xs + r * K + c * 4,
                       r < n ? Vec4<T>::load(x + (size_t)(t0 + r) * ldx + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f));
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int f = blockIdx.y * (FL_THREADS / 32) + warp; f < F; f += gridDim.y * (FL_THREADS / 32)) {
    float acc[TOK];
#pragma unroll
    for (int r = 0; r < TOK; ++r) acc[r] = 0.f;
    for (int c = lane; c < nvec; c += 32) {
      const float4 wv = Vec4<T>::load(w + (size_t)f * K + c * 4);
#pragma unroll
      for (int r = 0; r < TOK; ++r) {
        const float4 xv = Vec4<float>::load(xs + r * K + c * 4);
        acc[r] += xv.x * wv.x + xv.y * wv.y + xv.z * wv.z + xv.w * wv.w;
      }
    }
#pragma unroll
    for (int r = 0; r < TOK; ++r) {
      const float s = warp_sum(acc[r]);
      if (lane == 0 && r < n) out[(size_t)(t0 + r) * F + f] = s + (b != nullptr ? b[f] : 0.f);
    }
  }
}

// bf16 operands: far too few features for a tcgen05 tile, so warp-level m16n8k16 products with fp32 sums.  A CTA owns 16
// tokens and up to 32 features; its 8 warps split K.  A lane fetches 8 consecutive k of its rows with one 16-byte load:
// which k sit in which register slot does not matter as long as x and w agree.
constexpr int FLM_NT = 4;                  // feature tiles of 8 per CTA
__global__ void __launch_bounds__(FL_THREADS) few_linear_mma_kernel(const __nv_bfloat16* __restrict__ x, long long ldx,
                                                                    const __nv_bfloat16* __restrict__ w,
                                                                    const float* __restrict__ b, float* __restrict__ out,
                                                                    int M, int K, int F) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float part[FL_THREADS / 32][16][FLM_NT * 8 + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int t0 = blockIdx.x * 16, f0 = blockIdx.y * FLM_NT * 8;
  const int nt = min(FLM_NT, (F - f0 + 7) / 8);
  const __nv_bfloat16* x0 = x + (size_t)min(t0 + g, M - 1) * ldx + q * 8;
  const __nv_bfloat16* x1 = x + (size_t)min(t0 + g + 8, M - 1) * ldx + q * 8;
  const __nv_bfloat16* wr[FLM_NT];
  float acc[FLM_NT][4];
#pragma unroll
  for (int j = 0; j < FLM_NT; ++j) {
    wr[j] = w + (size_t)min(f0 + j * 8 + g, F - 1) * K + q * 8;
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  }
#pragma unroll 4
  for (int k = warp * 32; k < K; k += FL_THREADS) {
    const uint4 a = *reinterpret_cast<const uint4*>(x0 + k), c = *reinterpret_cast<const uint4*>(x1 + k);
#pragma unroll
    for (int j = 0; j < FLM_NT; ++j) {
      if (j < nt) {
        const uint4 v = *reinterpret_cast<const uint4*>(wr[j] + k);
        asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                     : "+f"(acc[j][0]), "+f"(acc[j][1]), "+f"(acc[j][2]), "+f"(acc[j][3])
                     : "r"(a.x), "r"(c.x), "r"(a.y), "r"(c.y), "r"(v.x), "r"(v.y));
        asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                     : "+f"(acc[j][0]), "+f"(acc[j][1]), "+f"(acc[j][2]), "+f"(acc[j][3])
                     : "r"(a.z), "r"(c.z), "r"(a.w), "r"(c.w), "r"(v.z), "r"(v.w));
      }
    }
  }
#pragma unroll
  for (int j = 0; j < FLM_NT; ++j) {
    part[warp][g][j * 8 + q * 2] = acc[j][0];
    part[warp][g][j * 8 + q * 2 + 1] = acc[j][1];
    part[warp][g + 8][j * 8 + q * 2] = acc[j][2];
    part[warp][g + 8][j * 8 + q * 2 + 1] = acc[j][3];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < 16 * nt * 8; i += FL_THREADS) {
    const int r = i / (nt * 8), f = i % (nt * 8);
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < FL_THREADS / 32; ++k) s += part[k][r][f];
    if (t0 + r < M && f0 + f < F) out[(size_t)(t0 + r) * F + f0 + f] = s + (b != nullptr ? b[f0 + f] : 0.f);
  }
}

// ---------------------------------------------------------------------------------------------
// out[M, F] = x[M, K] w[F, K]^T in fp32 (FMA units, no reduced-precision matrix mode): 64 x 64 tiles, 4 x 4 per thread.
// ---------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ x, long long ldx,
                                                       const float* __restrict__ w, long long ldw, float* __restrict__ out,
                                                       long long ldo, int M, int F, int K) {
  constexpr int BK = 16;
  __shared__ float xs[BK][64 + 4], ws[BK][64 + 4];
  const int t0 = blockIdx.y * 64, f0 = blockIdx.x * 64;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int lr = tid >> 2, lc = (tid & 3) * 4;              // tile row, first of 4 columns this thread loads
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += BK) {
    const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 xv = t0 + lr < M ? Vec4<float>::load(x + (size_t)(t0 + lr) * ldx + k0 + lc) : z;
    const float4 wv = f0 + lr < F ? Vec4<float>::load(w + (size_t)(f0 + lr) * ldw + k0 + lc) : z;
    __syncthreads();
    xs[lc][lr] = xv.x; xs[lc + 1][lr] = xv.y; xs[lc + 2][lr] = xv.z; xs[lc + 3][lr] = xv.w;
    ws[lc][lr] = wv.x; ws[lc + 1][lr] = wv.y; ws[lc + 2][lr] = wv.z; ws[lc + 3][lr] = wv.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, f = f0 + tx * 4 + j;
      if (t < M && f < F) out[(size_t)t * ldo + f] = acc[i][j];
    }
}

__global__ void swiglu_f32_kernel(const float* __restrict__ gu, float* __restrict__ out, int M, int I, long long ld_in,
                                  long long ld_out) {
  const long long n = (long long)M * I;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / I, c = i % I;
    const float g = gu[r * ld_in + c], u = gu[r * ld_in + I + c];
    out[r * ld_out + c] = g / (1.0f + expf(-g)) * u;
  }
}

// In place: up z^2 + z / 2 above zero, low (exp(z) - 1 - z) + z / 2 below
__global__ void xielu_f32_kernel(float* __restrict__ x, float up, float low, int M, int I, long long ld) {
  const long long n = (long long)M * I;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    float* q = x + i / I * ld + i % I;
    const float z = *q;
    *q = (z > 0.f ? up * z * z : low * (expm1f(z) - z)) + 0.5f * z;
  }
}

template <typename T, bool CENTER>
static int embed_norm_launch(const void* E, const int* tok, float scale, const int* pos, const float* freq, int streams,
                             const float* w_in, const float* add, float* x, const float* w, void* h, int M, int vocab, int width,
                             int groups, int ld, float eps, cudaStream_t stream) {
  const size_t smem = group_rms_smem(width, groups, ld);
  const int need = (ld / 4 + RN_THREADS - 1) / RN_THREADS;
  auto e = reinterpret_cast<const T*>(E);
  auto o = reinterpret_cast<T*>(h);
  cudaError_t rc;
#define TAHB_EN(V_) rc = launch_chain(embed_norm_kernel<T, V_, CENTER>, dim3(M), dim3(RN_THREADS), smem, stream, e, tok, scale, pos, freq, streams, w_in, add, x, w, o, vocab, width, groups, ld, eps)
  if (need <= 1) TAHB_EN(1);
  else if (need <= 2) TAHB_EN(2);
  else if (need <= 4) TAHB_EN(4);
  else if (need <= 8) TAHB_EN(8);
  else if (need <= 16) TAHB_EN(16);
  else return -2;
#undef TAHB_EN
  return rc == cudaSuccess ? 0 : -3;
}

template <typename T, int S>
static int streams_norm_launch(const StreamsParams& p, int M, cudaStream_t stream) {
  const int need = (p.ld / 4 + RN_THREADS - 1) / RN_THREADS;
  const size_t smem = group_rms_smem(p.width, p.groups, p.ld);
  cudaError_t rc;
#define TAHB_SN(V_) rc = launch_chain(streams_norm_kernel<T, V_, S>, dim3(M), dim3(RN_THREADS), smem, stream, p)
  if (need <= 1) TAHB_SN(1);
  else if (need <= 2) TAHB_SN(2);
  else if (need <= 4) TAHB_SN(4);
  else if (need <= 8) TAHB_SN(8);
  else if (need <= 16) TAHB_SN(16);
  else return -2;
#undef TAHB_SN
  return rc == cudaSuccess ? 0 : -3;
}

template <typename T, bool CENTER, bool ENTER>
static int residual_norm_launch(const ResidualNormParams& p, int M, cudaStream_t stream) {
  const int need = (p.ld / 4 + RN_THREADS - 1) / RN_THREADS;
  cudaError_t rc;
#define TAHB_RN(V_) rc = launch_chain(residual_norm_kernel<T, V_, CENTER, ENTER>, dim3(M), dim3(RN_THREADS), 0, stream, p)
  if (need <= 1) TAHB_RN(1);
  else if (need <= 2) TAHB_RN(2);
  else if (need <= 4) TAHB_RN(4);
  else if (need <= 8) TAHB_RN(8);
  else if (need <= 16) TAHB_RN(16);
  else return -2;
#undef TAHB_RN
  return rc == cudaSuccess ? 0 : -3;
}

template <typename T>
static int residual_add_norm_launch(const void* y, long long ldy, const void* y_ex, const int* slot, int top, float mult,
                                    float* x, const float* w_next, void* h, int M, int width, int groups, int ld, float eps,
                                    cudaStream_t stream) {
  const int need = (ld / 4 + RN_THREADS - 1) / RN_THREADS;
  const size_t smem = group_rms_smem(width, groups, ld);
  auto yy = reinterpret_cast<const T*>(y);
  auto ye = reinterpret_cast<const T*>(y_ex);
  auto o = reinterpret_cast<T*>(h);
  cudaError_t rc;
#define TAHB_RA(V_) rc = launch_chain(residual_add_norm_kernel<T, V_>, dim3(M), dim3(RN_THREADS), smem, stream, yy, ldy, ye, slot, top, mult, x, w_next, o, width, groups, ld, eps)
  if (need <= 1) TAHB_RA(1);
  else if (need <= 2) TAHB_RA(2);
  else if (need <= 4) TAHB_RA(4);
  else if (need <= 8) TAHB_RA(8);
  else if (need <= 16) TAHB_RA(16);
  else return -2;
#undef TAHB_RA
  return rc == cudaSuccess ? 0 : -3;
}

template <typename T, int TOK>
static int few_linear_launch(const void* x, long long ldx, const void* w, const float* b, float* out, int M, int K, int F,
                             cudaStream_t stream) {
  const size_t smem = (size_t)TOK * K * 4;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(few_linear_kernel<T, TOK>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return -10;
    configured = true;
  }
  if (smem > 200 * 1024) return -2;
  const dim3 grid((M + TOK - 1) / TOK, TOK == 1 ? (F + 7) / 8 : 1);
  cudaError_t rc = launch_chain(few_linear_kernel<T, TOK>, grid, dim3(FL_THREADS), smem, stream,
                                reinterpret_cast<const T*>(x), ldx, reinterpret_cast<const T*>(w), b, out, M, K, F);
  return rc == cudaSuccess ? 0 : -3;
}

}  // namespace tahb

using namespace tahb;

// pos / freq: sinusoidal positions; streams / w_in: copies in x and the weights of their sum; add: vector added to x (see
// embed_norm_kernel).  groups must divide width; centered: layer norm, groups = 1.
extern "C" int tahb_embed_norm(const void* E, const int* tok, float scale, const int* pos, const float* freq, int streams,
                               const float* w_in, const float* add, float* x, const float* w, void* h, int M, int vocab, int width,
                               int groups, int ld, float eps, int centered, int f32, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (ld % 4 || width > ld || groups < 1 || width % groups || (freq != nullptr && pos == nullptr) || streams < 1 ||
      (centered && groups != 1))
    return -1;
#define TAHB_EL(T_, C_) return embed_norm_launch<T_, C_>(E, tok, scale, pos, freq, streams, w_in, add, x, w, h, M, vocab, width, groups, ld, eps, stream)
  if (centered) {
    if (f32) TAHB_EL(float, true);
    TAHB_EL(__nv_bfloat16, true);
  }
  if (f32) TAHB_EL(float, false);
  TAHB_EL(__nv_bfloat16, false);
#undef TAHB_EL
}

// Seam of hyper-connections over `streams` (1..8) residual streams (see streams_norm_kernel).
extern "C" int tahb_streams_norm(const StreamsParams* p, int M, int streams, int f32, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (p->ld % 4 || p->ldy % 4 || p->width > p->ld || p->groups < 1 || p->width % p->groups ||
      (p->y_ex != nullptr && (p->slot == nullptr || p->top < 1)))
    return -1;
#define TAHB_SS(S_) if (streams == S_) return f32 ? streams_norm_launch<float, S_>(*p, M, stream) : streams_norm_launch<__nv_bfloat16, S_>(*p, M, stream);
  TAHB_SS(1) TAHB_SS(2) TAHB_SS(3) TAHB_SS(4) TAHB_SS(5) TAHB_SS(6) TAHB_SS(7) TAHB_SS(8)
#undef TAHB_SS
  return -2;
}

extern "C" int tahb_rotary_table(const int* pos, const float* freq, float mscale, float* out, int M, int half,
                                 cudaStream_t stream) {
  if (M <= 0 || half <= 0) return 0;
  if ((long long)M * half > 0x3fffffffll) return -2;
  int blocks = (M * half + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  const cudaError_t e = launch_chain(rotary_table_kernel, dim3(blocks), dim3(256), 0, stream, pos, freq, mscale,
                                     reinterpret_cast<float2*>(out), M, half);
  return e == cudaSuccess ? 0 : -3;
}

// x += mult * (y + sum_j y_ex[slot[., j]]); h = rms_g(x) * w_next.  y_ex / slot null: no expert outputs.
extern "C" int tahb_residual_add_norm(const void* y, long long ldy, const void* y_ex, const int* slot, int top, float mult,
                                      float* x, const float* w_next, void* h, int M, int width, int groups, int ld, float eps,
                                      int f32, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (ld % 4 || ldy % 4 || width > ld || groups < 1 || width % groups || (y_ex != nullptr && slot == nullptr)) return -1;
  return f32 ? residual_add_norm_launch<float>(y, ldy, y_ex, slot, top, mult, x, w_next, h, M, width, groups, ld, eps, stream)
             : residual_add_norm_launch<__nv_bfloat16>(y, ldy, y_ex, slot, top, mult, x, w_next, h, M, width, groups, ld, eps,
                                                       stream);
}

// centered: layer norms in the place of the RMS norms (see residual_norm_kernel)
extern "C" int tahb_residual_norm(const ResidualNormParams* p, int M, int centered, int f32, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (p->ld % 4 || p->ldy % 4 || p->width > p->ld || (p->E != nullptr && p->tok == nullptr)) return -1;
  const bool enter = p->add != nullptr || p->E != nullptr || p->before != nullptr;
#define TAHB_RL(T_) \
  return centered ? (enter ? residual_norm_launch<T_, true, true>(*p, M, stream) : residual_norm_launch<T_, true, false>(*p, M, stream)) \
                  : (enter ? residual_norm_launch<T_, false, true>(*p, M, stream) : residual_norm_launch<T_, false, false>(*p, M, stream))
  if (f32) TAHB_RL(float);
  TAHB_RL(__nv_bfloat16);
#undef TAHB_RL
}

extern "C" int tahb_few_linear(const void* x, long long ldx, const void* w, const float* b, float* out, int M, int K, int F,
                               int f32, cudaStream_t stream) {
  if (M <= 0 || F <= 0) return 0;
  if (K % 4 || ldx % 4) return -1;
  const bool one = M <= 148 || (size_t)4 * K * 4 > 200 * 1024;
  if (f32)
    return one ? few_linear_launch<float, 1>(x, ldx, w, b, out, M, K, F, stream)
               : few_linear_launch<float, 4>(x, ldx, w, b, out, M, K, F, stream);
  if (K % 32 || ldx % 8) return -1;
  const dim3 grid((M + 15) / 16, (F + FLM_NT * 8 - 1) / (FLM_NT * 8));
  cudaError_t rc = launch_chain(few_linear_mma_kernel, grid, dim3(FL_THREADS), 0, stream, reinterpret_cast<const __nv_bfloat16*>(x),
                                ldx, reinterpret_cast<const __nv_bfloat16*>(w), b, out, M, K, F);
  return rc == cudaSuccess ? 0 : -3;
}

extern "C" int tahb_gemm_f32(const float* x, long long ldx, const float* w, long long ldw, float* out, long long ldo, int M,
                             int F, int K, cudaStream_t stream) {
  if (M <= 0 || F <= 0) return 0;
  if (K % 16 || ldx % 4 || ldw % 4) return -1;
  gemm_f32_kernel<<<dim3((F + 63) / 64, (M + 63) / 64), 256, 0, stream>>>(x, ldx, w, ldw, out, ldo, M, F, K);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int tahb_swiglu_f32(const float* gu, float* out, int M, int I, long long ld_in, long long ld_out,
                               cudaStream_t stream) {
  if (M <= 0) return 0;
  long long blocks = ((long long)M * I + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  swiglu_f32_kernel<<<(int)blocks, 256, 0, stream>>>(gu, out, M, I, ld_in, ld_out);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int tahb_xielu_f32(float* x, float up, float low, int M, int I, long long ld, cudaStream_t stream) {
  if (M <= 0) return 0;
  long long blocks = ((long long)M * I + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  xielu_f32_kernel<<<(int)blocks, 256, 0, stream>>>(x, up, low, M, I, ld);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
