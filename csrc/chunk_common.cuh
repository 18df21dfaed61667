// Pieces shared by the chunkwise matrix-memory kernels (mlstm.cu, gla.cu): chunk geometry, 3-D tensor-map copies, the split of
// an fp32 operand into a bf16 pair, and the tensor maps of head matrices and states.
#pragma once
#include <cuda.h>

#include "attn_common.cuh"
#include "common.cuh"

namespace tahb {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float4 ldf4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ldf4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

constexpr int MC_TOK = 128;
constexpr int MC_KCH = MC_TOK * 128;          // bytes of one 64-column chunk of a 128-token tile

__device__ __forceinline__ void tma_load_3d(void* smem_dst, const void* tmap, int c0, int c1, int c2, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(tmap)), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2)
      : "memory");
}
__device__ __forceinline__ void tma_store_3d(const void* tmap, const void* smem_src, int c0, int c1, int c2) {
  asm volatile("cp.async.bulk.tensor.3d.global.shared::cta.bulk_group [%0, {%2, %3, %4}], [%1];"
               ::"l"(reinterpret_cast<uint64_t>(tmap)), "r"(smem_u32(smem_src)), "r"(c0), "r"(c1), "r"(c2)
               : "memory");
}
constexpr float MC_LOG2E = 1.4426950408889634f;
// A MN-major (transposed), B MN-major
__host__ __device__ constexpr uint32_t umma_idesc_bf16_amn_bmn(int m, int n) { return umma_idesc_bf16(m, n) | (1u << 15) | (1u << 16); }

__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// [n tokens][heads of d dims] inside a row-major matrix of pitch ld: boxes of 128 tokens x 64 dims of one head
static int make_head_map(CUtensorMap* m, const __nv_bfloat16* base, int d, int heads, long long n, long long ld) {
  PfEncodeFn fn = pf_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || d % 8 || ld % 8) return -2;
  cuuint64_t dims[3] = {(cuuint64_t)d, (cuuint64_t)heads, (cuuint64_t)n};
  cuuint64_t strides[2] = {(cuuint64_t)d * 2, (cuuint64_t)ld * 2};
  cuuint32_t box[3] = {64u, 1u, (cuuint32_t)MC_TOK}, estr[3] = {1u, 1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<__nv_bfloat16*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}
static int make_state_map(CUtensorMap* m, const __nv_bfloat16* base, int dk, int dv, long long n) {
  PfEncodeFn fn = pf_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || dv % 8) return -2;
  cuuint64_t dims[3] = {(cuuint64_t)dv, (cuuint64_t)dk, (cuuint64_t)n};
  cuuint64_t strides[2] = {(cuuint64_t)dv * 2, (cuuint64_t)dk * dv * 2};
  cuuint32_t box[3] = {64u, 64u, 1u}, estr[3] = {1u, 1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<__nv_bfloat16*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}

// [n][dk][dv] fp32, boxes of 128 rows x 32 columns (rows past dk are not written)
static int make_dS_map(CUtensorMap* m, float* base, int dk, int dv, long long n) {
  PfEncodeFn fn = pf_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || dv % 4) return -2;
  cuuint64_t dims[3] = {(cuuint64_t)dv, (cuuint64_t)dk, (cuuint64_t)n};
  cuuint64_t strides[2] = {(cuuint64_t)dv * 4, (cuuint64_t)dk * dv * 4};
  cuuint32_t box[3] = {32u, 128u, 1u}, estr[3] = {1u, 1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_FLOAT32, 3, base, dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}

}  // namespace tahb
