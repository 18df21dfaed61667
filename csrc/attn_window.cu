// Paged attention with a sliding window, kept first tokens, a per-distance bias, a softmax sink and a per-head output gate.
//
// Query at position i of a sequence sees key j when  j <= i  and  (i - j < window  or  j < keep_first).
// score = (q . k) * scale + bias[h][min(i - j, D)]; softmax over the visible keys with exp(sink_h) added to the
// denominator; out_h *= sigmoid(gate_h).  Every constant is a launch parameter: window = INT_MAX is plain causal
// attention, keep_first = 0 a plain window, and the bias table, the sink and the gate may each be absent.
//
// Keys and values are read from the paged cache only (the tokens of the running step are written there first), so
// portions of a prompt, single decoded tokens and layers that read another layer's cache are the same case:
//   page of one layer:  [K: kv_heads][page_size][dk]  then  [V: kv_heads][page_size][dv]
// dk and dv are padded to multiples of 8; padding dims hold zeros.
#include "common.cuh"

namespace tahb {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// 8 consecutive elements as floats (16-byte loads)
__device__ __forceinline__ void load8(const float* p, float* o) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* o) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = __bfloat1622float2(h[j]);
    o[2 * j] = f.x;
    o[2 * j + 1] = f.y;
  }
}

// ---------------------------------------------------------------------------------------------
// Append the tokens of a step to the paged cache.  entry e: `count[e]` further tokens of row `row[e]`, whose packed
// places start at `start[e]`.  Takes pages from the free stack, fills the page table, advances the length and writes for
// every packed token its position, row and slot (page * page_size + offset).  One CTA.  When the pool or the row's table
// is too small nothing is taken: the status word is set and the tokens get slot -1 and position 0.
// ---------------------------------------------------------------------------------------------
constexpr int APPEND_MAX = 1024;
__global__ void __launch_bounds__(256) kv_append_kernel(const int* __restrict__ row, const int* __restrict__ count,
                                                        const int* __restrict__ start, int n_entries, int* len,
                                                        int* page_table, int* free_stack, int* free_count, int rows,
                                                        int max_pages, int page_size, int* __restrict__ pos_out,
                                                        int* __restrict__ row_out, int* __restrict__ slot_out, int* status) {
  __shared__ int s_len[APPEND_MAX], s_off[APPEND_MAX];
  __shared__ int s_ok, s_free;
  if (threadIdx.x == 0) {
    int off = 0;
    bool ok = true;
    for (int e = 0; e < n_entries; ++e) {
      const int L = len[row[e]], c = count[e];
      const int need = (L + c + page_size - 1) / page_size - (L + page_size - 1) / page_size;
      s_len[e] = L;
      s_off[e] = off;
      off += need;
      ok = ok && (L + c + page_size - 1) / page_size <= max_pages;
    }
    const int have = free_count[0];
    ok = ok && off <= have;
    s_ok = ok;
    s_free = have;
    if (ok) {
      free_count[0] = have - off;
      for (int e = 0; e < n_entries; ++e) len[row[e]] = s_len[e] + count[e];
    } else {
      atomicCAS(status, 0, STATUS_BAD_INDEX);
    }
  }
  __syncthreads();
  const bool ok = s_ok != 0;
  if (ok) {
    for (int e = 0; e < n_entries; ++e) {
      const int have = (s_len[e] + page_size - 1) / page_size;
      const int need = (s_len[e] + count[e] + page_size - 1) / page_size - have;
      for (int i = threadIdx.x; i < need; i += blockDim.x)
        page_table[(size_t)row[e] * max_pages + have + i] = free_stack[s_free - 1 - s_off[e] - i];
    }
  }
  __syncthreads();
  for (int e = 0; e < n_entries; ++e) {
    const int r = row[e];
    for (int t = threadIdx.x; t < count[e]; t += blockDim.x) {
      const int p = ok ? s_len[e] + t : 0;
      pos_out[start[e] + t] = p;
      row_out[start[e] + t] = r;
      slot_out[start[e] + t] = ok ? page_table[(size_t)r * max_pages + p / page_size] * page_size + p % page_size : -1;
    }
  }
}

// ---------------------------------------------------------------------------------------------
// After the fused projection [q | k | v | ...]: bias, per-head RMS norm of q and k, q to its own matrix, k and v to the
// paged cache.  One warp per (token, head); a lane owns dim pairs 2 * lane, 2 * lane + 64, ...
// ---------------------------------------------------------------------------------------------
struct QkvPostParams {
  const void* qkv;            // [M, ld]: nq heads of dk, then nkv heads of dk, then nkv heads of dv
  const float* bias;          // same columns, or null
  const float* q_w;           // [dk] (padding dims zero), null = no norm
  const float* k_w;
  void* q_out;                // [M, nq * dk]
  void* cache;                // paged cache of the layer (nkv > 0)
  const int* slot;            // [M], negative = no cache write
  int M, nq, nkv, dk, dv, dim, page_size;     // dim = real (unpadded) size of a q / k head
  long long ld;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(128) qkv_post_kernel(const QkvPostParams p) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int MAXP = 4;                       // dk, dv <= 256
  const int heads = p.nq + 2 * p.nkv;
  const long long wg = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (wg >= (long long)p.M * heads) return;
  const int t = (int)(wg / heads), h = (int)(wg % heads);
  const bool is_q = h < p.nq, is_k = !is_q && h < p.nq + p.nkv;
  const int d = is_q || is_k ? p.dk : p.dv;
  const int col = is_q || is_k ? h * p.dk : (p.nq + p.nkv) * p.dk + (h - p.nq - p.nkv) * p.dv;
  const T* src = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.ld + col;
  float x[2 * MAXP];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < MAXP; ++i) {
    const int c = 2 * lane + 64 * i;
    x[2 * i] = x[2 * i + 1] = 0.f;
    if (c < d) {
      x[2 * i] = to_f<T>(src[c]);
      x[2 * i + 1] = to_f<T>(src[c + 1]);
      if (p.bias != nullptr) {
        x[2 * i] += p.bias[col + c];
        x[2 * i + 1] += p.bias[col + c + 1];
      }
      ss += x[2 * i] * x[2 * i] + x[2 * i + 1] * x[2 * i + 1];
    }
  }
  const float* w = is_q ? p.q_w : is_k ? p.k_w : nullptr;
  if (w != nullptr) {
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
#pragma unroll
    for (int i = 0; i < MAXP; ++i) {
      const int c = 2 * lane + 64 * i;
      if (c < d) {
        x[2 * i] *= r * w[c];
        x[2 * i + 1] *= r * w[c + 1];
      }
    }
  }
  T* dst;
  if (is_q) {
    dst = reinterpret_cast<T*>(p.q_out) + ((size_t)t * p.nq + h) * p.dk;
  } else {
    const int sl = p.slot[t];
    if (sl < 0) return;
    const int page = sl / p.page_size, off = sl % p.page_size;
    const size_t page_elems = (size_t)p.nkv * p.page_size * (p.dk + p.dv);
    dst = reinterpret_cast<T*>(p.cache) + (size_t)page * page_elems;
    if (is_k) dst += ((size_t)(h - p.nq) * p.page_size + off) * p.dk;
    else dst += (size_t)p.nkv * p.page_size * p.dk + ((size_t)(h - p.nq - p.nkv) * p.page_size + off) * p.dv;
  }
#pragma unroll
  for (int i = 0; i < MAXP; ++i) {
    const int c = 2 * lane + 64 * i;
    if (c < d) {
      dst[c] = from_f<T>(x[2 * i]);
      dst[c + 1] = from_f<T>(x[2 * i + 1]);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// What every attention kernel of this file gets.
// ---------------------------------------------------------------------------------------------
struct WindowAttnParams {
  const void* q;              // [n, nq * dk]
  void* out;                  // [n, ld_out], head h at column h * dv
  const void* cache;          // paged cache of the layer that owns the keys
  const int* page_table;      // [rows, max_pages]
  const int* pos;             // [n] position of each query
  const int* row;             // [n] cache row of each query
  const float* bias;          // [nq, far + 1] bias by distance (the last entry serves every larger distance), or null
  const float* sink;          // [nq] or null
  const void* gate;           // pre-activation of head h of query t at gate[t * ld_gate + h], or null
  int n, nq, nkv, dk, dv, page_size, max_pages, window, keep_first, far;
  long long ld_out, ld_gate;
  float scale;
  float* ws;                  // split partial results (decode kernel, n_split > 1)
  int n_split;
  int* status;
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

// First key of the window part, and the end of the kept part in front of it: visible keys are [0, keep_end) and [lo, i].
__device__ __forceinline__ void visible_range(int i, int window, int keep_first, int& keep_end, int& lo) {
  lo = i - window + 1;
  if (window > i) lo = 0;
  keep_end = min(keep_first, lo);
}

// ---------------------------------------------------------------------------------------------
// Plain kernel: any head sizes up to 256, bf16 or fp32 cache.  One warp per (query, head); 32 keys at a time, one key
// per lane for the scores, one dim pair per lane for the weighted values.  Used by the 32-bit mode and for head sizes
// that the tensor-core and pipelined kernels do not cover.
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) window_attn_plain_kernel(const WindowAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int MAXP = 4;
  __shared__ float s_q[4][256];
  __shared__ float s_w[4][32];
  __shared__ int s_page[4][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long wg = (long long)blockIdx.x * 4 + warp;
  if (wg >= (long long)p.n * p.nq) return;
  const int t = (int)(wg / p.nq), h = (int)(wg % p.nq), kvh = h / (p.nq / p.nkv);
  const int i = p.pos[t];
  const int* pt = p.page_table + (size_t)p.row[t] * p.max_pages;
  const T* q = reinterpret_cast<const T*>(p.q) + ((size_t)t * p.nq + h) * p.dk;
  for (int d = lane; d < p.dk; d += 32) s_q[warp][d] = to_f<T>(q[d]);
  __syncwarp();
  const size_t page_elems = (size_t)p.nkv * p.page_size * (p.dk + p.dv);
  const T* kc = reinterpret_cast<const T*>(p.cache) + (size_t)kvh * p.page_size * p.dk;
  const T* vc = reinterpret_cast<const T*>(p.cache) + (size_t)p.nkv * p.page_size * p.dk + (size_t)kvh * p.page_size * p.dv;
  float m = -INFINITY, l = 0.f, acc[2 * MAXP];
#pragma unroll
  for (int c = 0; c < 2 * MAXP; ++c) acc[c] = 0.f;
  int keep_end, lo;
  visible_range(i, p.window, p.keep_first, keep_end, lo);
  for (int part = 0; part < 2; ++part) {
    const int a = part == 0 ? 0 : lo, b = part == 0 ? keep_end : i + 1;
    for (int j0 = a; j0 < b; j0 += 32) {
      const int j = j0 + lane;
      float s = -INFINITY;
      int page = 0;
      if (j < b) {
        page = pt[j / p.page_size];
        const T* k = kc + (size_t)page * page_elems + (size_t)(j % p.page_size) * p.dk;
        float dot = 0.f;
        for (int d = 0; d < p.dk; d += 8) {
          float kv[8];
          load8(k + d, kv);
#pragma unroll
          for (int u = 0; u < 8; ++u) dot = fmaf(s_q[warp][d + u], kv[u], dot);
        }
        s = dot * p.scale;
        if (p.bias != nullptr) s += p.bias[(size_t)h * (p.far + 1) + min(i - j, p.far)];
      }
      const float mx = fmaxf(m, warp_max(s));
      const float corr = m == -INFINITY ? 0.f : expf(m - mx);
      const float w = j < b ? expf(s - mx) : 0.f;
      l = l * corr + warp_sum(w);
      m = mx;
      __syncwarp();
      s_w[warp][lane] = w;
      s_page[warp][lane] = page;
      __syncwarp();
#pragma unroll
      for (int c = 0; c < 2 * MAXP; ++c) acc[c] *= corr;
      const int n_here = min(32, b - j0);
      for (int u = 0; u < n_here; ++u) {
        const T* v = vc + (size_t)s_page[warp][u] * page_elems + (size_t)((j0 + u) % p.page_size) * p.dv;
        const float wu = s_w[warp][u];
#pragma unroll
        for (int c = 0; c < MAXP; ++c) {
          const int d = 2 * lane + 64 * c;
          if (d < p.dv) {
            acc[2 * c] = fmaf(wu, to_f<T>(v[d]), acc[2 * c]);
            acc[2 * c + 1] = fmaf(wu, to_f<T>(v[d + 1]), acc[2 * c + 1]);
          }
        }
      }
    }
  }
  float f = 1.0f;
  if (p.sink != nullptr) {
    const float top = fmaxf(m, p.sink[h]);
    f = expf(m - top);
    l = l * f + expf(p.sink[h] - top);
  }
  f = f / l;
  if (p.gate != nullptr) f *= sigmoid_f(to_f<T>(reinterpret_cast<const T*>(p.gate)[(size_t)t * p.ld_gate + h]));
  T* o = reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + (size_t)h * p.dv;
#pragma unroll
  for (int c = 0; c < MAXP; ++c) {
    const int d = 2 * lane + 64 * c;
    if (d < p.dv) {
      o[d] = from_f<T>(acc[2 * c] * f);
      o[d + 1] = from_f<T>(acc[2 * c + 1] * f);
    }
  }
}

}  // namespace tahb

using namespace tahb;

extern "C" int tahb_kv_append(const int* row, const int* count, const int* start, int n_entries, int* len, int* page_table,
                              int* free_stack, int* free_count, int rows, int max_pages, int page_size, int* pos_out,
                              int* row_out, int* slot_out, int* status, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (n_entries > APPEND_MAX) return -1;
  kv_append_kernel<<<1, 256, 0, stream>>>(row, count, start, n_entries, len, page_table, free_stack, free_count, rows,
                                          max_pages, page_size, pos_out, row_out, slot_out, status);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int tahb_qkv_post(const void* qkv, long long ld, const float* bias, const float* q_w, const float* k_w,
                             void* q_out, void* cache, const int* slot, int M, int nq, int nkv, int dk, int dv, int dim,
                             int page_size, float eps, int f32, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (dk > 256 || dv > 256 || dk % 8 || dv % 8 || dim > dk) return -2;
  QkvPostParams p;
  p.qkv = qkv; p.bias = bias; p.q_w = q_w; p.k_w = k_w; p.q_out = q_out; p.cache = cache; p.slot = slot;
  p.M = M; p.nq = nq; p.nkv = nkv; p.dk = dk; p.dv = dv; p.dim = dim; p.page_size = page_size; p.ld = ld; p.eps = eps;
  const long long warps = (long long)M * (nq + 2 * nkv);
  const dim3 grid((unsigned)((warps + 3) / 4));
  cudaError_t e = f32 ? launch_chain(qkv_post_kernel<float>, grid, dim3(128), 0, stream, p)
                      : launch_chain(qkv_post_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p);
  return e == cudaSuccess ? 0 : -3;
}

// Host-side description of one attention launch (same fields as WindowAttnParams).
extern "C" int tahb_window_attn_plain(const WindowAttnParams* p, int f32, cudaStream_t stream) {
  if (p->n <= 0) return 0;
  if (p->nkv <= 0 || p->nq % p->nkv || p->dk > 256 || p->dv > 256 || p->dk % 8 || p->dv % 8 || p->window < 1 || p->far < 0)
    return -2;
  const long long warps = (long long)p->n * p->nq;
  const dim3 grid((unsigned)((warps + 3) / 4));
  cudaError_t e = f32 ? launch_chain(window_attn_plain_kernel<float>, grid, dim3(128), 0, stream, *p)
                      : launch_chain(window_attn_plain_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}
