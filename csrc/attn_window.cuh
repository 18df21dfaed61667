// What the kernels over paged keys share (attn_window.cu, attn_tied.cu): launch parameters, visibility rule, finish of a head,
// tensor maps of pages.
#pragma once
#include <cuda.h>

#include "attn_common.cuh"
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
// What every attention kernel gets.
// ---------------------------------------------------------------------------------------------
struct WindowAttnParams {
  const void* q;              // [n, ld_q], head h at column h * dk
  void* out;                  // [n, ld_out], head h at column h * dv
  const void* cache;          // paged cache of the layer that owns the keys
  const int* page_table;      // [rows, max_pages]
  const int* pos;             // [n] position of each query
  const int* row;             // [n] cache row of each query
  const float* bias;          // [nq, far + 1] bias by distance (the last entry serves every larger distance), or null
  const float* sink;          // [nq] or null
  const void* gate;           // pre-activation of head h of query t at gate[t * ld_gate + h], or null
  const void* wide_gate;      // pre-activation of every output element, gate[t * ld_gate + h * dv + d], or null
  int n, nq, nkv, dk, dv, page_size, max_pages, window, keep_first, far;
  long long ld_q, ld_out, ld_gate;
  float scale;
  float softcap;              // 0 = no cap
  float temp_coef;            // 0 = no query temperature
  double temp_every;
  float* ws;                  // split partial results (decode kernel, n_split > 1)
  int n_split;
  int* status;
  const float* slope;         // [nq] taken off the scores per token of distance, or null
  const float* factor;        // [pages][page_size] factor of every key's scores (tied layers), or null
  const void* pooled;         // pooled blocks of a tied layer (plain and decode kernels: their pool; portion kernel: a matrix), or null
  int tied;                   // the values are the keys
  int n_pages;                // pages of the pool (tied decode kernel)
  int pool, pool_rows;        // tokens of a pooled block, pooled rows of a page
  float out_scale;            // factor of the output
};

// scale of the scores of a query at position i
__device__ __forceinline__ float query_scale(const WindowAttnParams& p, int i) {
  if (p.temp_coef == 0.f) return p.scale;
  return p.scale * (1.0f + p.temp_coef * logf((float)floor((double)(i + 1) / p.temp_every) + 1.0f));
}

// tanh on the special-function unit, 1 - 2 / (1 + exp(2 x)): absolute error ~2^-22, saturates to +-1
__device__ __forceinline__ float tanh_sfu(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + ex2_approx(x * (2.0f * 1.4426950408889634f))));
  return fmaf(-2.0f, r, 1.0f);
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

// First key of the window part, and the end of the kept part in front of it: visible keys are [0, keep_end) and [lo, i].
__device__ __forceinline__ void visible_range(int i, int window, int keep_first, int& keep_end, int& lo) {
  lo = i - window + 1;
  if (window > i) lo = 0;
  keep_end = min(keep_first, lo);
}

// pooled blocks that a query at position i sees
__device__ __forceinline__ int visible_blocks(int i, int window, int pool) { return max(0, i - window + 1) / pool; }

// 8 elements as they lie in memory
template <typename T> struct Row8;
template <> struct Row8<float> { using type = struct { float4 a, b; }; };
template <> struct Row8<__nv_bfloat16> { using type = uint4; };

constexpr int WD_PAGE = 16;
constexpr float LOG2E = 1.4426950408889634f;

// o = sum / (mass + exp2(sink - m)), times the head's gate; m, mass, sink in log2 units
__device__ __forceinline__ float finish_scale(const WindowAttnParams& p, int t, int h, float m, float mass) {
  float f = 1.0f;
  if (p.sink != nullptr) {
    const float top = fmaxf(m, p.sink[h]);
    f = exp2f(m - top);
    mass = mass * f + exp2f(p.sink[h] - top);
  }
  f = mass > 0.f ? f / mass * p.out_scale : 0.f;
  if (p.gate != nullptr)
    f *= sigmoid_f(__bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.gate)[(size_t)t * p.ld_gate + h]));
  return f;
}

// factor of output element d of head h from its own gate
__device__ __forceinline__ float element_gate(const WindowAttnParams& p, int t, int h, int d) {
  if (p.wide_gate == nullptr) return 1.0f;
  const float z = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.wide_gate)[(size_t)t * p.ld_gate + (size_t)h * p.dv + d]);
  return __fdividef(1.0f, 1.0f + __expf(-z));
}

__device__ __forceinline__ void tma_load_4d(void* smem_dst, const void* tmap, int c0, int c1, int c2, int c3, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(tmap)), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3)
      : "memory");
}

// Keys (or values) of a paged cache as a 4-D tensor [pages][kv heads][tokens of a page][dims], read in boxes of one page's tokens x
// 64 dims; tok / head / page: strides in elements
static inline int make_page_map(CUtensorMap* m, const void* base, int d, int nkv, int n_pages, size_t tok, size_t head, size_t page,
                                int tokens = WD_PAGE, bool swizzle = true) {
  PfEncodeFn fn = pf_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || d % 8 || tok % 8 || head % 8 || page % 8) return -2;
  cuuint64_t dims[4] = {(cuuint64_t)d, (cuuint64_t)tokens, (cuuint64_t)nkv, (cuuint64_t)n_pages};
  cuuint64_t strides[3] = {(cuuint64_t)tok * 2, (cuuint64_t)head * 2, (cuuint64_t)page * 2};
  cuuint32_t box[4] = {64u, (cuuint32_t)tokens, 1u, 1u}, estr[4] = {1u, 1u, 1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, swizzle ? CU_TENSOR_MAP_SWIZZLE_128B : CU_TENSOR_MAP_SWIZZLE_NONE,
                  CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}

int check_window_attn(const WindowAttnParams* p);                                  // attn_window.cu
cudaError_t launch_window_merge(const WindowAttnParams& p, cudaStream_t stream);   // attn_window.cu: merge of the decode kernels' key splits
int launch_tied_decode(const WindowAttnParams& p, cudaStream_t stream);            // attn_tied.cu

}  // namespace tahb
