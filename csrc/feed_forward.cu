// Feed-forward mechanisms of decoders with an fp32 residual stream (activations T = bf16, or fp32 in the 32-bit mode).
//
//   poly_norm       act(z) = a N(z) + b N(z^2) + c N(z^3) + e with powers element by element and N(v) = v / sqrt(mean(v^2) +
//                   eps) over the token's vector
//   clamped_glu     y = g sigmoid(slope g) (u + offset), g = min(gate, limit), u = clamp(up, -limit, limit), of interleaved
//                   gate / up columns, optionally with a factor per row in front (a routed token's weight) or behind (a
//                   shared expert's gate).  SwiGLU is slope 1, offset 0, limit infinity
//   moe_route       sigmoid or softmax scores, the `top` largest per token, and the experts' token lists in blocks of `bn` rows
//   moe_gather      the tokens' rows copied into the lists
//   moe_gemm        grouped product over the lists, one weight matrix per expert (tcgen05, persistent CTAs, two accumulators
//                   in tensor memory so that the epilogue of a tile runs under the main loop of the next); plain, or with
//                   the clamped_glu epilogue
//   moe_gemm_f32    the same product in fp32 on the FMA units
//
// Expert lists.  Expert e owns blocks of bn consecutive list rows; blocks of all experts follow one another, so block b
// covers rows [b * bn, (b + 1) * bn) and belongs to expert blk_expert[b].  Rows behind an expert's last token hold nothing
// of use: their products stay in rows that nobody reads.  Where a token sits in a list does not enter its arithmetic.
#include <cuda.h>

#include "attn_common.cuh"
#include "common.cuh"

namespace tahb {

// 8 consecutive elements: as they lie in memory (Raw, 16-byte units) and as floats
template <typename T> struct Vec8;
template <> struct Vec8<float> {
  struct Raw { float4 a, b; };
  static __device__ __forceinline__ void renew(Raw&) {}
  static __device__ __forceinline__ Raw raw(const float* p) {
    return {reinterpret_cast<const float4*>(p)[0], reinterpret_cast<const float4*>(p)[1]};
  }
  static __device__ __forceinline__ void unpack(const Raw& r, float* o) {
    o[0] = r.a.x; o[1] = r.a.y; o[2] = r.a.z; o[3] = r.a.w; o[4] = r.b.x; o[5] = r.b.y; o[6] = r.b.z; o[7] = r.b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* v) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
  }
};
template <> struct Vec8<__nv_bfloat16> {
  typedef uint4 Raw;
  // keeps the compiler from holding the unpacked floats (twice the registers) across the use in between
  static __device__ __forceinline__ void renew(Raw& r) { asm volatile("" : "+r"(r.x), "+r"(r.y), "+r"(r.z), "+r"(r.w)); }
  static __device__ __forceinline__ Raw raw(const __nv_bfloat16* p) { return *reinterpret_cast<const uint4*>(p); }
  static __device__ __forceinline__ void unpack(const Raw& r, float* o) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = __bfloat1622float2(h[j]);
      o[2 * j] = f.x;
      o[2 * j + 1] = f.y;
    }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
    uint4 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
    *reinterpret_cast<uint4*>(p) = u;
  }
};

// ---------------------------------------------------------------------------------------------
// poly_norm: one CTA per token.  The normalised powers share z, so with k1 = a / rms(z), k2 = b / rms(z^2), k3 = c /
// rms(z^3) the activation is z (k1 + z (k2 + z k3)) + e.  Columns [n, np) are padding (z = 0 there; they get e, and meet
// zero columns of the next weight).
// ---------------------------------------------------------------------------------------------
constexpr int PN_THREADS = 256;

template <typename T, int VPT>
__global__ void __launch_bounds__(PN_THREADS) poly_norm_kernel(const T* __restrict__ z, long long ldz,
                                                               const float* __restrict__ act, T* __restrict__ out,
                                                               long long ldo, int n, int np, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[3][PN_THREADS / 32];
  const size_t row = blockIdx.x;
  const int nvec = np / 8;
  typename Vec8<T>::Raw raw[VPT];
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * PN_THREADS;
    if (c < nvec) raw[i] = Vec8<T>::raw(z + row * ldz + c * 8);
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * PN_THREADS;
    if (c < nvec) {
      float v[8];
      Vec8<T>::unpack(raw[i], v);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float q = v[e] * v[e], q2 = q * q;
        s2 += q;
        s4 += q2;
        s6 = fmaf(q2, q, s6);
      }
    }
  }
  s2 = warp_sum(s2); s4 = warp_sum(s4); s6 = warp_sum(s6);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = s2; red[1][threadIdx.x >> 5] = s4; red[2][threadIdx.x >> 5] = s6;
  }
  __syncthreads();
  float k[3];
#pragma unroll
  for (int j = 0; j < 3; ++j) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < PN_THREADS / 32; ++w) s += red[j][w];
    k[j] = act[j] / sqrtf(s / (float)n + eps);
  }
  const float e0 = act[3];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * PN_THREADS;
    if (c < nvec) {
      float v[8];
      Vec8<T>::renew(raw[i]);
      Vec8<T>::unpack(raw[i], v);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = fmaf(v[e], fmaf(v[e], fmaf(v[e], k[2], k[1]), k[0]), e0);
      Vec8<T>::store(out + row * ldo + c * 8, v);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// clamped_glu as a kernel of its own: 8 outputs (16 interleaved inputs) per thread and step.
// ---------------------------------------------------------------------------------------------
struct GluShape {
  float limit, slope, offset;
};

struct GluParams {
  const void* in;             // [rows, ld_in] gate_0, up_0, gate_1, up_1, ...
  void* out;                  // [rows, ld_out]
  long long ld_in, ld_out;
  int rows, width;            // width = outputs per row (a multiple of 8)
  GluShape a;
  const float* in_scale;      // [rows] factor of gate and up, or null
  const float* gate;          // row r of the result times sigmoid(gate[r * ld_gate]), or null
  long long ld_gate;
  const int* n_blocks;        // rows of expert lists: only the first *n_blocks * bn are live, or null
  int bn;
};

template <typename T>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const GluParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const unsigned rows = p.n_blocks != nullptr ? min((long long)p.rows, (long long)*p.n_blocks * p.bn) : p.rows;
  const unsigned nv = p.width / 8, n = rows * nv;              // the host checks that rows * nv fits
  for (unsigned i = blockIdx.x * 256u + threadIdx.x; i < n; i += gridDim.x * 256u) {
    const size_t r = i / nv;
    const int c = (int)(i % nv) * 8;
    float v[16], o[8];
    const T* src = reinterpret_cast<const T*>(p.in) + r * p.ld_in + 2 * c;
    const typename Vec8<T>::Raw lo = Vec8<T>::raw(src), hi = Vec8<T>::raw(src + 8);
    Vec8<T>::unpack(lo, v);
    Vec8<T>::unpack(hi, v + 8);
    const float w = p.in_scale != nullptr ? p.in_scale[r] : 1.0f;
    const float f = p.gate != nullptr ? 1.0f / (1.0f + expf(-p.gate[r * p.ld_gate])) : 1.0f;
    constexpr bool fast = sizeof(T) == 2;       // the result is rounded to 16 bits: approximate exponential and division do
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float g = fminf(w * v[2 * e], p.a.limit), u = fminf(fmaxf(w * v[2 * e + 1], -p.a.limit), p.a.limit);
      o[e] = (fast ? __fdividef(g, 1.0f + __expf(-p.a.slope * g)) : g / (1.0f + expf(-p.a.slope * g))) * (u + p.a.offset) * f;
    }
    Vec8<T>::store(reinterpret_cast<T*>(p.out) + r * p.ld_out + c, o);
  }
}

// ---------------------------------------------------------------------------------------------
// moe_route: one warp per token picks the `top` largest scores (lower index on a tie; softmax scores are over all experts
// and stay as they are); ranks inside an expert's list come
// from counters (shared per CTA, one global addition per CTA and expert).  The CTA that finishes last turns the counts
// into list starts and the block table and clears the counters for the next launch.
// ---------------------------------------------------------------------------------------------
struct RouteParams {
  const float* z;             // [M, ldz] router logits, experts in columns 0 .. E - 1
  long long ldz;
  int M, E, top, bn, tok;     // tok = tokens per CTA
  int softmax;
  int* expert;                // [M * top]
  int* rank;                  // [M * top] place in the expert's list
  float* weight;              // [M * top] score
  int* count;                 // [E + 1]: counters and a ticket, zero between launches
  int* seg;                   // [E] first list row of the expert
  int* blk_expert;            // [max_blocks]
  int* n_blocks;              // [1]
  int max_blocks;
  int* status;
};
constexpr int ROUTE_THREADS = 256;
constexpr int ROUTE_MAX_EXPERTS = 1024;

template <int NV>             // experts per lane
__global__ void __launch_bounds__(ROUTE_THREADS) moe_route_kernel(const RouteParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ int rsm[];
  int* cnt = rsm;                              // [E]
  int* base = cnt + p.E;                       // [E]
  int* my_e = base + p.E;                      // [tok * top]
  int* my_r = my_e + p.tok * p.top;            // [tok * top]
  __shared__ int s_last, s_part[ROUTE_THREADS / 32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * p.tok, nt = min(p.tok, p.M - t0);
  for (int e = threadIdx.x; e < p.E; e += ROUTE_THREADS) cnt[e] = 0;
  __syncthreads();
  for (int t = warp; t < nt; t += ROUTE_THREADS / 32) {
    float s[NV];
    if (p.softmax) {
      float mx = -INFINITY, sum = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int e = lane + 32 * i;
        s[i] = e < p.E ? p.z[(size_t)(t0 + t) * p.ldz + e] : -INFINITY;
        mx = fmaxf(mx, s[i]);
      }
      mx = warp_max(mx);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        s[i] = lane + 32 * i < p.E ? expf(s[i] - mx) : 0.f;
        sum += s[i];
      }
      sum = warp_sum(sum);
#pragma unroll
      for (int i = 0; i < NV; ++i) s[i] = lane + 32 * i < p.E ? s[i] / sum : -1.0f;
    } else {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int e = lane + 32 * i;
        s[i] = e < p.E ? 1.0f / (1.0f + expf(-p.z[(size_t)(t0 + t) * p.ldz + e])) : -1.0f;
      }
    }
    for (int j = 0; j < p.top; ++j) {
      float bv = -1.0f;
      int be = p.E;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (s[i] > bv) { bv = s[i]; be = lane + 32 * i; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const int oe = __shfl_xor_sync(0xffffffffu, be, o);
        if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; }
      }
      be = min(be, p.E - 1);                   // scores that are not numbers: any expert, but one that exists
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (be == lane + 32 * i) s[i] = -1.0f;
      if (lane == 0) {
        my_e[t * p.top + j] = be;
        my_r[t * p.top + j] = atomicAdd(&cnt[be], 1);
        p.weight[(size_t)(t0 + t) * p.top + j] = bv;
      }
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < p.E; e += ROUTE_THREADS)
    if (cnt[e] > 0) base[e] = atomicAdd(&p.count[e], cnt[e]);
  __syncthreads();
  for (int i = threadIdx.x; i < nt * p.top; i += ROUTE_THREADS) {
    p.expert[(size_t)t0 * p.top + i] = my_e[i];
    p.rank[(size_t)t0 * p.top + i] = base[my_e[i]] + my_r[i];
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(&p.count[p.E], 1) == (int)gridDim.x - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  // counts -> first block of every expert (each thread takes a run of consecutive experts)
  const int per = (p.E + ROUTE_THREADS - 1) / ROUTE_THREADS;
  const int e0 = threadIdx.x * per, e1 = min(p.E, e0 + per);
  int mine = 0;
  for (int e = e0; e < e1; ++e) mine += (__ldcg(&p.count[e]) + p.bn - 1) / p.bn;
  int pre = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, pre, o);
    if (lane >= o) pre += v;
  }
  if (lane == 31) s_part[warp] = pre;
  __syncthreads();
  int at = pre - mine;
  for (int w = 0; w < warp; ++w) at += s_part[w];
  for (int e = e0; e < e1; ++e) {
    const int nb = (__ldcg(&p.count[e]) + p.bn - 1) / p.bn;
    p.seg[e] = at * p.bn;
    for (int b = 0; b < nb && at + b < p.max_blocks; ++b) p.blk_expert[at + b] = e;
    at += nb;
    p.count[e] = 0;
  }
  if (threadIdx.x == ROUTE_THREADS - 1) {
    if (at > p.max_blocks) atomicCAS(p.status, 0, STATUS_BAD_INDEX);
    *p.n_blocks = min(at, p.max_blocks);
    p.count[p.E] = 0;
  }
}

// One CTA per token: its row (16-byte units) goes to a list row of each of its experts; list_weight and slot on the way.
__global__ void __launch_bounds__(128) moe_gather_kernel(const uint4* __restrict__ h, int units, long long ld_units, int top,
                                                         const int* __restrict__ expert, const int* __restrict__ rank,
                                                         const float* __restrict__ weight, const int* __restrict__ seg,
                                                         uint4* __restrict__ list, float* __restrict__ list_weight,
                                                         int* __restrict__ slot, int list_rows, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int s_slot[64];
  const size_t t = blockIdx.x;
  for (int j = threadIdx.x; j < top; j += 128) {
    const size_t a = t * top + j;
    int s = seg[expert[a]] + rank[a];
    if (s >= list_rows) {                       // cannot happen with the capacity the host computes
      atomicCAS(status, 0, STATUS_BAD_INDEX);
      s = 0;
    }
    s_slot[j] = s;
    slot[a] = s;
    list_weight[s] = weight[a];
  }
  __syncthreads();
  for (int c = threadIdx.x; c < units; c += 128) {
    const uint4 v = h[t * ld_units + c];
    for (int j = 0; j < top; ++j) list[(size_t)s_slot[j] * units + c] = v;
  }
}

// ---------------------------------------------------------------------------------------------
// moe_gemm: out[r, f] = list[r, :] . W[expert of r's block][f, :], features on the 128 lanes and the bn rows of a block on
// the columns of the accumulator, as in the dense GEMM.  Persistent CTAs walk the tiles (block, 128 features), features
// fastest, so that the CTAs at work share the rows of a block and the weights of an expert in L2.  Tensor memory holds two
// accumulators; the epilogue warps drain one while the tensor core fills the other.
// Warp roles (192 threads): warp 0 TMA, warp 1 tensor memory + MMA, warps 2..5 epilogue.
// ---------------------------------------------------------------------------------------------
struct MoeGemmParams {
  const int* blk_expert;
  const int* n_blocks;
  const float* row_weight;    // GLU: factor of gate and up of every list row, or null
  int f_rows;                 // weight rows of an expert
  int f_tiles;                // 128-row tiles of them
  int kb;                     // K / 64
  GluShape a;
  int* status;
};

template <int BN, bool GLU>
struct MoeCfg {
  static constexpr int W_BYTES = 128 * 64 * 2, X_BYTES = BN * 64 * 2, STAGE_BYTES = W_BYTES + X_BYTES;
  static constexpr int OUT_COLS = GLU ? 64 : 128;
  static constexpr int OUT_BYTES = BN * OUT_COLS * 2;
  static constexpr int NS_RAW = (227 * 1024 - 1024 - 512 - OUT_BYTES) / STAGE_BYTES;
  static constexpr int NS = NS_RAW > 10 ? 10 : NS_RAW;
  static constexpr int TMEM_COLS = 2 * BN < 32 ? 32 : 2 * BN;
  static constexpr int CHUNK = BN >= 32 ? 32 : 16;
  static constexpr int SMEM_BYTES = NS * STAGE_BYTES + OUT_BYTES + 1024 + 512;
};

template <int BN, bool GLU>
__global__ void __launch_bounds__(192, 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x,
                const __grid_constant__ CUtensorMap tm_out, const MoeGemmParams p) {
  using C = MoeCfg<BN, GLU>;
  pdl_launch_dependents();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* stg_raw = smem + C::NS * C::STAGE_BYTES;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(stg_raw + C::OUT_BYTES);
  uint64_t* empty_bar = full_bar + C::NS;
  uint64_t* acc_full = empty_bar + C::NS;
  uint64_t* acc_empty = acc_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < C::NS; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(&acc_full[a], 1);
      mbar_init(&acc_empty[a], 128);
    }
    *abort_flag = 0;
    mbar_fence_init();
    prefetch_tensormap(&tm_w);
    prefetch_tensormap(&tm_x);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, C::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_wait();
  const uint32_t tmem_base = *tmem_slot;
  const int n_tiles = *p.n_blocks * p.f_tiles;

  if (warp == 0) {
    if (lane == 0) {
      int g = 0;
      for (int tile = blockIdx.x; tile < n_tiles && !*abort_flag; tile += gridDim.x) {
        const int b = tile / p.f_tiles, w_row = p.blk_expert[b] * p.f_rows + (tile % p.f_tiles) * 128;
        for (int k = 0; k < p.kb; ++k, ++g) {
          const int s = g % C::NS;
          mbar_wait(&empty_bar[s], ((g / C::NS) & 1) ^ 1, abort_flag, p.status, STATUS_TIMEOUT_STAGE_EMPTY);
          if (*abort_flag) break;
          mbar_expect_tx(&full_bar[s], C::STAGE_BYTES);
          uint8_t* st = smem + s * C::STAGE_BYTES;
          tma_load_2d(st, &tm_w, k * 64, w_row, &full_bar[s]);
          tma_load_2d(st + C::W_BYTES, &tm_x, k * 64, b * BN, &full_bar[s]);
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc_bf16(128, BN);
      int g = 0, it = 0;
      for (int tile = blockIdx.x; tile < n_tiles && !*abort_flag; tile += gridDim.x, ++it) {
        const int a = it & 1;
        mbar_wait(&acc_empty[a], ((it >> 1) & 1) ^ 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
        tc_fence_after();
        for (int k = 0; k < p.kb; ++k, ++g) {
          const int s = g % C::NS;
          mbar_wait(&full_bar[s], (g / C::NS) & 1, abort_flag, p.status, STATUS_TIMEOUT_TMA_FULL);
          tc_fence_after();
          const uint32_t w_addr = smem_u32(smem + s * C::STAGE_BYTES);
          const uint64_t dw = umma_desc_sw128(w_addr), dx = umma_desc_sw128(w_addr + C::W_BYTES);
#pragma unroll
          for (int j = 0; j < 4; ++j)
            umma_bf16(tmem_base + a * BN, dw + 2 * j, dx + 2 * j, idesc, (k > 0 || j > 0) ? 1u : 0u);
          umma_commit(&empty_bar[s]);
        }
        umma_commit(&acc_full[a]);
      }
    }
    __syncwarp();
  } else {
    const int q = warp & 3, row = q * 32 + lane;
    const bool odd = row & 1;
    __nv_bfloat16* stg = reinterpret_cast<__nv_bfloat16*>(stg_raw);          // [BN rows][OUT_COLS]
    int it = 0;
    // no early exit here: the named barriers need all 128 threads in every round, and after an abort the waits return at once
    for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++it) {
      const int a = it & 1, b = tile / p.f_tiles, f0 = (tile % p.f_tiles) * 128;
      const uint32_t trow = tmem_base + a * BN + (static_cast<uint32_t>(q * 32) << 16);
      if (threadIdx.x == 64) tma_store_wait_read();                            // the previous tile has left the staging area
      named_bar_sync(1, 128);
      mbar_wait(&acc_full[a], (it >> 1) & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
      tc_fence_after();
#pragma unroll 1
      for (int c0 = 0; c0 < BN; c0 += C::CHUNK) {
        float v[C::CHUNK];
        if constexpr (C::CHUNK == 32) tmem_ld32(trow + c0, v);
        else tmem_ld16(trow + c0, v);
        float wl = 1.0f;
        if constexpr (GLU) {
          if (lane < C::CHUNK && p.row_weight != nullptr) wl = p.row_weight[b * BN + c0 + lane];
        }
        tmem_ld_wait();
        if constexpr (GLU) {
          // lanes 2 i / 2 i + 1 hold gate_i / up_i: the even lane finishes token j, the odd one token j + 1
#pragma unroll
          for (int j = 0; j < C::CHUNK; j += 2) {
            const float recv = __shfl_xor_sync(0xffffffffu, odd ? v[j] : v[j + 1], 1);
            const float w = __shfl_sync(0xffffffffu, wl, j + (odd ? 1 : 0));
            const float g = fminf(w * (odd ? recv : v[j]), p.a.limit);
            const float u = fminf(fmaxf(w * (odd ? v[j + 1] : recv), -p.a.limit), p.a.limit);
            stg[(c0 + j + (odd ? 1 : 0)) * 64 + (row >> 1)] =
                __float2bfloat16_rn(__fdividef(g, 1.0f + __expf(-p.a.slope * g)) * (u + p.a.offset));
          }
        } else {
#pragma unroll
          for (int j = 0; j < C::CHUNK; ++j) stg[(c0 + j) * 128 + row] = __float2bfloat16_rn(v[j]);
        }
      }
      tc_fence_before();
      mbar_arrive(&acc_empty[a]);
      fence_proxy_async_smem();
      named_bar_sync(1, 128);
      if (threadIdx.x == 64) {
        tma_store_2d(&tm_out, stg, GLU ? f0 / 2 : f0, b * BN);
        tma_store_commit();
      }
    }
    if (threadIdx.x == 64) tma_store_wait_read();
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, C::TMEM_COLS);
  }
}

// fp32: blocks of 64 rows, 64 x 64 tiles, 4 x 4 per thread
__global__ void __launch_bounds__(256) moe_gemm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                           float* __restrict__ out, const int* __restrict__ blk_expert,
                                                           const int* __restrict__ n_blocks, int F, int K) {
  if ((int)blockIdx.y >= *n_blocks) return;
  constexpr int BK = 16;
  __shared__ float xs[BK][64 + 4], ws[BK][64 + 4];
  const size_t r0 = (size_t)blockIdx.y * 64;
  const int f0 = blockIdx.x * 64;
  const float* we = w + (size_t)blk_expert[blockIdx.y] * F * K;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int lr = tid >> 2, lc = (tid & 3) * 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += BK) {
    const float4 xv = *reinterpret_cast<const float4*>(x + (r0 + lr) * K + k0 + lc);
    const float4 wv = f0 + lr < F ? *reinterpret_cast<const float4*>(we + (size_t)(f0 + lr) * K + k0 + lc)
                                  : make_float4(0.f, 0.f, 0.f, 0.f);
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
    for (int j = 0; j < 4; ++j)
      if (f0 + tx * 4 + j < F) out[(r0 + ty * 4 + i) * F + f0 + tx * 4 + j] = acc[i][j];
}

// bf16 [rows, cols] row-major, boxes of box_rows x box_cols; operands with the 128-byte swizzle
static int matrix_map(CUtensorMap* m, const void* base, long long rows, long long cols, unsigned box_rows, unsigned box_cols,
                      bool operand) {
  PfEncodeFn fn = pf_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || cols % 8) return -2;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
  cuuint32_t box[2] = {box_cols, box_rows}, estr[2] = {1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, operand ? CU_TENSOR_MAP_SWIZZLE_128B : CU_TENSOR_MAP_SWIZZLE_NONE,
                  operand ? CU_TENSOR_MAP_L2_PROMOTION_L2_256B : CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}

template <int BN, bool GLU>
static int launch_moe_gemm(const void* w, const void* x, void* out, long long w_rows, int K, int list_rows, int f_out,
                           const MoeGemmParams& p, cudaStream_t stream) {
  using C = MoeCfg<BN, GLU>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(moe_gemm_kernel<BN, GLU>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES) != cudaSuccess)
      return -10;
    configured = true;
  }
  CUtensorMap mw, mx, mo;
  int rc;
  if ((rc = matrix_map(&mw, w, w_rows, K, 128, 64, true))) return rc;
  if ((rc = matrix_map(&mx, x, list_rows, K, BN, 64, true))) return rc;
  if ((rc = matrix_map(&mo, out, list_rows, f_out, BN, C::OUT_COLS, false))) return rc;
  const long long tiles = (long long)(list_rows / BN) * p.f_tiles;
  const cudaError_t e = launch_chain(moe_gemm_kernel<BN, GLU>, dim3((unsigned)(tiles < 148 ? tiles : 148)), dim3(192),
                                     C::SMEM_BYTES, stream, mw, mx, mo, p);
  return e == cudaSuccess ? 0 : -12;
}

template <typename T>
static int poly_norm_launch(const void* z, long long ldz, const float* act, void* out, long long ldo, int M, int n, int np,
                            float eps, cudaStream_t stream) {
  const int need = (np / 8 + PN_THREADS - 1) / PN_THREADS;
  auto zz = reinterpret_cast<const T*>(z);
  auto oo = reinterpret_cast<T*>(out);
  cudaError_t rc;
#define TAHB_PN(V_) rc = launch_chain(poly_norm_kernel<T, V_>, dim3(M), dim3(PN_THREADS), 0, stream, zz, ldz, act, oo, ldo, n, np, eps)
  if (need <= 1) TAHB_PN(1);
  else if (need <= 2) TAHB_PN(2);
  else if (need <= 4) TAHB_PN(4);
  else if (need <= 6) TAHB_PN(6);
  else if (need <= 10) TAHB_PN(10);
  else return -2;
#undef TAHB_PN
  return rc == cudaSuccess ? 0 : -3;
}

}  // namespace tahb

using namespace tahb;

extern "C" int tahb_poly_norm(const void* z, long long ldz, const float* act, void* out, long long ldo, int M, int n, int np,
                              float eps, int f32, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (n > np || np % 8 || ldz % 8 || ldo % 8 || ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15)) return -1;
  return f32 ? poly_norm_launch<float>(z, ldz, act, out, ldo, M, n, np, eps, stream)
             : poly_norm_launch<__nv_bfloat16>(z, ldz, act, out, ldo, M, n, np, eps, stream);
}

extern "C" int tahb_clamped_glu(const void* in, long long ld_in, void* out, long long ld_out, int rows, int width, float limit,
                                float slope, float offset, const float* in_scale, const float* gate, long long ld_gate, const int* n_blocks, int bn,
                                int f32, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width % 8 || ld_in % 8 || ld_out % 8 || ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out)) & 15)) return -1;
  if ((long long)rows * (width / 8) > 0x7fffffffll) return -2;
  GluParams p{in, out, ld_in, ld_out, rows, width, {limit, slope, offset}, in_scale, gate, ld_gate, n_blocks, bn};
  long long blocks = ((long long)rows * (width / 8) + 255) / 256;
  if (blocks > 148 * 32) blocks = 148 * 32;
  const cudaError_t e = f32 ? launch_chain(clamped_glu_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, p)
                            : launch_chain(clamped_glu_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, p);
  return e == cudaSuccess ? 0 : -3;
}

// Router and expert lists (see moe_route_kernel); count: E + 1 ints that are zero before the first launch.
extern "C" int tahb_moe_route(const float* z, long long ldz, int M, int E, int top, int bn, int softmax, int* expert, int* rank,
                              float* weight, int* count, int* seg, int* blk_expert, int* n_blocks, int max_blocks,
                              int* status, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (E < 1 || E > ROUTE_MAX_EXPERTS || top < 1 || top > E || top > 64 || bn < 1 || ldz < E) return -2;
  RouteParams p{z, ldz, M, E, top, bn, M >= 4096 ? 32 : 8, softmax, expert, rank, weight, count, seg, blk_expert, n_blocks, max_blocks, status};
  const dim3 grid((M + p.tok - 1) / p.tok);
  const size_t smem = (size_t)(2 * E + 2 * p.tok * top) * 4;
  const int nv = (E + 31) / 32;
  cudaError_t e;
  if (nv <= 1) e = launch_chain(moe_route_kernel<1>, grid, dim3(ROUTE_THREADS), smem, stream, p);
  else if (nv <= 2) e = launch_chain(moe_route_kernel<2>, grid, dim3(ROUTE_THREADS), smem, stream, p);
  else if (nv <= 4) e = launch_chain(moe_route_kernel<4>, grid, dim3(ROUTE_THREADS), smem, stream, p);
  else if (nv <= 8) e = launch_chain(moe_route_kernel<8>, grid, dim3(ROUTE_THREADS), smem, stream, p);
  else e = launch_chain(moe_route_kernel<32>, grid, dim3(ROUTE_THREADS), smem, stream, p);
  return e == cudaSuccess ? 0 : -3;
}

// h: M rows of row_bytes (pitch ld_bytes), both multiples of 16
extern "C" int tahb_moe_gather(const void* h, int row_bytes, long long ld_bytes, int M, int top, const int* expert,
                               const int* rank, const float* weight, const int* seg, void* list, float* list_weight, int* slot,
                               int list_rows, int* status, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (row_bytes % 16 || ld_bytes % 16 || top > 64) return -2;
  const cudaError_t e = launch_chain(moe_gather_kernel, dim3(M), dim3(128), 0, stream, reinterpret_cast<const uint4*>(h),
                                     row_bytes / 16, ld_bytes / 16, top, expert, rank, weight, seg,
                                     reinterpret_cast<uint4*>(list), list_weight, slot, list_rows, status);
  return e == cudaSuccess ? 0 : -3;
}

// W: [E * f_rows, K]; x: [list_rows, K]; out: [list_rows, f_rows] or, with glu (interleaved gate / up rows), [.., f_rows / 2].
// list_rows is a multiple of bn.
extern "C" int tahb_moe_gemm(const void* w, const void* x, void* out, int E, int f_rows, int K, int list_rows, int bn,
                             const int* blk_expert, const int* n_blocks, int glu, const float* row_weight, float limit,
                             float slope, float offset, int* status, cudaStream_t stream) {
  if (list_rows <= 0) return 0;
  if (K % 64 || K <= 0 || f_rows % 64 || list_rows % bn || (glu && f_rows % 128)) return -2;
  if ((long long)E * f_rows > 0x7fffffffll) return -2;
  MoeGemmParams p{blk_expert, n_blocks, row_weight, f_rows, (f_rows + 127) / 128, K / 64, {limit, slope, offset}, status};
  const long long w_rows = (long long)E * f_rows;
#define TAHB_MG(B_)                                                                                           \
  if (bn == B_) return glu ? launch_moe_gemm<B_, true>(w, x, out, w_rows, K, list_rows, f_rows / 2, p, stream) \
                           : launch_moe_gemm<B_, false>(w, x, out, w_rows, K, list_rows, f_rows, p, stream);
  TAHB_MG(16) TAHB_MG(32) TAHB_MG(64) TAHB_MG(128) TAHB_MG(256)
#undef TAHB_MG
  return -2;
}

extern "C" int tahb_moe_gemm_f32(const float* w, const float* x, float* out, int f_rows, int K, int list_rows,
                                 const int* blk_expert, const int* n_blocks, cudaStream_t stream) {
  if (list_rows <= 0) return 0;
  if (K % 16 || list_rows % 64 || list_rows / 64 > 65535) return -2;
  moe_gemm_f32_kernel<<<dim3((f_rows + 63) / 64, list_rows / 64), 256, 0, stream>>>(x, w, out, blk_expert, n_blocks, f_rows, K);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
