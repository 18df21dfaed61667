// Latent attention: keys and values of all heads are linear in one cached vector per token.
//
//   cached row of a token:  [c: kv_rank, padded to Rp][r: rot dims, padded to rw], both multiples of 64
//     c = rms(low part) * w,  r = rotated shared key part
//   head h:  key = [Wk_h c, r], value = Wv_h c;  score = (q . key) * scale over the last `window` tokens;  softmax with exp(sink_h)
//   in the denominator (optional);  out_h *= sigmoid(gate), element by element (optional)
//
// Single tokens run in the absorbed form: q' = [Wk_h^T q_unrotated, q_rotated] against the cached rows themselves (one key
// and one value, c, for all heads), then Wv_h on the weighted sum of c.  Prompt portions expand the row's cached latents to
// keys and values with one matrix product and run the portion kernel of attn_window.cu on them.
//
// Head lists.  Activations of the absorbed form are ordered head by head: row h * npad + t for token t, so that the per-head
// products are the grouped products of feed_forward.cu with heads in the place of experts.
#include <cuda.h>

#include "chunk_common.cuh"

namespace tahb {

template <typename T> __device__ __forceinline__ void ld8(const T* p, float* o);
template <> __device__ __forceinline__ void ld8<float>(const float* p, float* o) {
  const float4 a = ldf4(p), b = ldf4(p + 4);
  o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
}
template <> __device__ __forceinline__ void ld8<__nv_bfloat16>(const __nv_bfloat16* p, float* o) {
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
// latent_post, after the projection [query latent | c | r | gate]: RMS norm of the query latent to a matrix of its own; RMS
// norm of c and rotation of r (pairs (2 i, 2 i + 1)) to the paged cache.  One CTA per token.
// ---------------------------------------------------------------------------------------------
struct LatentPostParams {
  const void* proj;           // [M, ld]
  const float* q_w;           // [Qp] zero in the padding
  const float* c_w;           // [Rp]
  const float2* rope;         // [M, rot / 2] (cos, sin)
  void* cq;                   // [M, Qp]
  void* cache;                // [pages][page_size][Rp + rw]
  const int* slot;            // [M], negative = no cache write
  int M, q_rank, Qp, q_col, kv_rank, Rp, c_col, rot, rw, r_col;
  long long ld;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_post_kernel(const LatentPostParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[2][4];
  const size_t t = blockIdx.x;
  const T* x = reinterpret_cast<const T*>(p.proj) + t * p.ld;
  float sq = 0.f, sc = 0.f;
  for (int i = threadIdx.x * 4; i < p.Qp; i += 512) {
    const float4 v = ldf4(x + p.q_col + i);
    sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  for (int i = threadIdx.x * 4; i < p.Rp; i += 512) {
    const float4 v = ldf4(x + p.c_col + i);
    sc += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = sq;
    red[1][threadIdx.x >> 5] = sc;
  }
  __syncthreads();
  const float rq = 1.0f / sqrtf((red[0][0] + red[0][1] + red[0][2] + red[0][3]) / (float)p.q_rank + p.eps);
  const float rc = 1.0f / sqrtf((red[1][0] + red[1][1] + red[1][2] + red[1][3]) / (float)p.kv_rank + p.eps);
  T* cq = reinterpret_cast<T*>(p.cq) + t * p.Qp;
  for (int i = threadIdx.x * 4; i < p.Qp; i += 512) {
    const float4 v = ldf4(x + p.q_col + i), w = ldf4(p.q_w + i);
    stf(cq + i, v.x * rq * w.x); stf(cq + i + 1, v.y * rq * w.y); stf(cq + i + 2, v.z * rq * w.z); stf(cq + i + 3, v.w * rq * w.w);
  }
  const int sl = p.slot[t];
  if (sl < 0) return;
  T* row = reinterpret_cast<T*>(p.cache) + (size_t)sl * (p.Rp + p.rw);
  for (int i = threadIdx.x * 4; i < p.Rp; i += 512) {
    const float4 v = ldf4(x + p.c_col + i), w = ldf4(p.c_w + i);
    stf(row + i, v.x * rc * w.x); stf(row + i + 1, v.y * rc * w.y); stf(row + i + 2, v.z * rc * w.z); stf(row + i + 3, v.w * rc * w.w);
  }
  for (int i = threadIdx.x; i < p.rw / 2; i += 128) {
    float a = 0.f, b = 0.f;
    if (2 * i < p.rot) {
      const float2 f = p.rope[t * (p.rot / 2) + i];
      const float u = ldf(x + p.r_col + 2 * i), v = ldf(x + p.r_col + 2 * i + 1);
      a = u * f.x - v * f.y;
      b = v * f.x + u * f.y;
    }
    stf(row + p.Rp + 2 * i, a);
    stf(row + p.Rp + 2 * i + 1, b);
  }
}

// ---------------------------------------------------------------------------------------------
// latent_query: the projected queries [n, heads * dk], head = [dim | rot], get their last rot dims rotated.  Tokens below
// n_list go to head lists [heads * npad, dq] (zero behind dim + rot), the others stay where they are.  Grid (n, head blocks).
// ---------------------------------------------------------------------------------------------
struct LatentQueryParams {
  void* q;
  const float2* rope;
  void* list;
  int n, n_list, npad, heads, dk, dq, dim, rot;
  long long ld;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_query_kernel(const LatentQueryParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, half = p.rot / 2, per = (p.heads + gridDim.y - 1) / gridDim.y;
  const int h0 = blockIdx.y * per, nh = min(per, p.heads - h0);
  const bool listed = t < p.n_list;
  T* src = reinterpret_cast<T*>(p.q) + (size_t)t * p.ld;
  T* list = reinterpret_cast<T*>(p.list) + (size_t)t * p.dq;             // head h at h * npad * dq
  const size_t head = listed ? (size_t)p.npad * p.dq : p.dk;
  T* dst = listed ? list : src;
  for (int i = threadIdx.x; i < nh * half; i += 256) {
    const int h = h0 + i / half, k = i % half;
    const float2 f = p.rope[(size_t)t * half + k];
    const T* q = src + (size_t)h * p.dk + p.dim + 2 * k;
    const float u = ldf(q), v = ldf(q + 1);
    T* o = dst + h * head + p.dim + 2 * k;
    stf(o, u * f.x - v * f.y);
    stf(o + 1, v * f.x + u * f.y);
  }
  if (listed) {
    const int rest = p.dq - p.rot;                                        // unrotated dims, then the zeros behind the head
    for (int i = threadIdx.x; i < nh * rest; i += 256) {
      const int h = h0 + i / rest, d = i % rest;
      if (d < p.dim) list[h * head + d] = src[(size_t)h * p.dk + d];
      else stf(list + h * head + d + p.rot, 0.f);
    }
  }
}

// Pages of the cache one after another as rows of pitch lp (16-byte units; zero behind the cached row).
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint4* __restrict__ cache, const int* __restrict__ src, int n_pool,
                                                            int page_size, int units, int lp_units, uint4* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int page = src[blockIdx.x];
  for (int i = threadIdx.x; i < page_size * lp_units; i += 128) {
    const int r = i / lp_units, c = i % lp_units;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (c < units && page >= 0 && page < n_pool) v = cache[((size_t)page * page_size + r) * units + c];
    out[((size_t)blockIdx.x * page_size + r) * lp_units + c] = v;
  }
}

// out[t, h * dv + d] = list[h * npad + t, d] * sigmoid(gate[t, h * dv + d]) (gate null: no factor), 8 elements per thread
template <typename T>
__global__ void __launch_bounds__(256) latent_gate_kernel(const T* __restrict__ list, int npad, int ld_list, const T* __restrict__ gate,
                                                          long long ld_gate, T* __restrict__ out, long long ld_out, int n, int heads,
                                                          int dv) {
  pdl_launch_dependents();
  pdl_wait();
  const int nv = dv / 8;
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= (long long)n * heads * nv) return;
  const int c = (int)(i % nv) * 8, h = (int)(i / nv % heads), t = (int)(i / nv / heads);
  float v[8], z[8];
  ld8(list + ((size_t)h * npad + t) * ld_list + c, v);
  if (gate == nullptr) {
#pragma unroll
    for (int e = 0; e < 8; ++e) stf(out + (size_t)t * ld_out + (size_t)h * dv + c + e, v[e]);
    return;
  }
  ld8(gate + (size_t)t * ld_gate + (size_t)h * dv + c, z);
#pragma unroll
  for (int e = 0; e < 8; ++e) stf(out + (size_t)t * ld_out + (size_t)h * dv + c + e, v[e] / (1.0f + expf(-z[e])));
}

// ---------------------------------------------------------------------------------------------
// What the absorbed attention kernels get.
// ---------------------------------------------------------------------------------------------
struct LatentAttnParams {
  const void* q;              // head lists [heads * npad, lq]: Rp + rw real columns
  void* out;                  // head lists [heads * npad, Rp]
  const void* cache;
  const int* page_table;      // [rows, max_pages]
  const int* pos;             // [n]
  const int* row;             // [n]
  const float* sink;          // [heads] or null
  int n, npad, heads, Rp, rw, lq, page_size, max_pages;
  float scale;
  float* ws;                  // split partial results (n_split > 1)
  int n_split;
  int n_pages;                // pages of the pool
  int* status;
  int window;                 // tokens that a query sees, itself the last of them
};

// Plain kernel: any sizes, bf16 or fp32.  One CTA per (head, token); 128 keys at a time, one key per thread for the scores,
// the columns of c dealt out to the threads for the weighted sum.  sink in natural units.
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_plain_kernel(const LatentAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float lsm[];
  const int len = p.Rp + p.rw;
  float* s_q = lsm;                    // [len]
  float* s_acc = s_q + len;            // [Rp]
  float* s_w = s_acc + p.Rp;           // [128]
  float* s_red = s_w + 128;            // [8]
  int* s_page = reinterpret_cast<int*>(s_red + 8);   // [128]
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int i = p.pos[t];
  const int* pt = p.page_table + (size_t)p.row[t] * p.max_pages;
  const size_t lrow = (size_t)h * p.npad + t;
  const T* q = reinterpret_cast<const T*>(p.q) + lrow * p.lq;
  for (int d = tid; d < len; d += 128) s_q[d] = ldf(q + d);
  for (int d = tid; d < p.Rp; d += 128) s_acc[d] = 0.f;
  __syncthreads();
  float m = -INFINITY, l = 0.f;
  for (int j0 = p.window > i ? 0 : i - p.window + 1; j0 <= i; j0 += 128) {
    const int j = j0 + tid;
    float s = -INFINITY;
    int at = 0;
    if (j <= i) {
      at = pt[j / p.page_size] * p.page_size + j % p.page_size;
      const T* k = reinterpret_cast<const T*>(p.cache) + (size_t)at * len;
      float dot = 0.f;
      for (int d = 0; d < len; d += 8) {
        float kv[8];
        ld8(k + d, kv);
#pragma unroll
        for (int e = 0; e < 8; ++e) dot = fmaf(s_q[d + e], kv[e], dot);
      }
      s = dot * p.scale;
    }
    float mx = warp_max(s);
    if (lane == 0) s_red[warp] = mx;
    __syncthreads();
    mx = fmaxf(m, fmaxf(fmaxf(s_red[0], s_red[1]), fmaxf(s_red[2], s_red[3])));
    const float corr = m == -INFINITY ? 0.f : expf(m - mx);
    const float w = j <= i ? expf(s - mx) : 0.f;
    s_w[tid] = w;
    s_page[tid] = at;
    const float sum = warp_sum(w);
    if (lane == 0) s_red[4 + warp] = sum;
    m = mx;
    __syncthreads();
    l = l * corr + s_red[4] + s_red[5] + s_red[6] + s_red[7];
    const int nh = min(128, i + 1 - j0);
    for (int d = tid; d < p.Rp; d += 128) {
      float a = s_acc[d] * corr;
      for (int u = 0; u < nh; ++u) a = fmaf(s_w[u], ldf(reinterpret_cast<const T*>(p.cache) + (size_t)s_page[u] * len + d), a);
      s_acc[d] = a;
    }
    __syncthreads();
  }
  float f = 1.0f;
  if (p.sink != nullptr) {
    const float top = fmaxf(m, p.sink[h]);
    f = expf(m - top);
    l = l * f + expf(p.sink[h] - top);
  }
  f /= l;
  T* o = reinterpret_cast<T*>(p.out) + lrow * p.Rp;
  for (int d = tid; d < p.Rp; d += 128) stf(o + d, s_acc[d] * f);
}

// ---------------------------------------------------------------------------------------------
// Decode kernel (bf16, pages of 16) on the tensor cores: one CTA = N query heads of one token over a run of 48-key tiles.
// Keys lie on the lanes of the score accumulator and heads on its columns, S[key][head] = row . q', so that a few heads fill
// a product whose M side is the keys; the weighted sum is O[latent][head] += c^T P with the same shared-memory tile read
// transposed.  Every cached row crosses HBM once per CTA for all of its heads.
//   A stage is 48 cached rows as groups of 8 keys, [group][64-column chunk][8 keys][64], one copy per group for the whole
//   row.  The score product has M = 64 rows, 16 on the lanes of each warp; its last 16 are whatever follows the stage and
//   are not read.  Three stages of a 512 + 64 row fit, two of them on their way while one is at work; scores and weights
//   exist twice, so that the score product of a tile runs beside the softmax of the one before.
//   The products are short (few heads), so their issue rate matters: the whole MMA warp walks the loop, which keeps the
//   descriptors in uniform registers, and one elected lane issues (42 instead of 57 cycles a product).
// Every thread keeps the heads' reference maxima in registers; a tile whose scores stay below 2^8 times them (one vote) needs
// no reduction, any other goes through a reduction over its keys and a pass over O.
// Warp roles (192 threads): warp 0 TMA, warp 1 tensor memory + MMA, warps 2..5 softmax, 16 lanes of each a key, and epilogue,
// one thread per latent.  sink in log2 units.
// ---------------------------------------------------------------------------------------------
constexpr int LD_PAGE = 16, LD_TILE = 48, LD_GROUPS = LD_TILE / 8, LD_THREADS = 192, LD_MAX_STAGES = 8;
constexpr float LD_LOG2E = 1.4426950408889634f;

// Reduce N values per lane over the 32 lanes of a warp: lane x returns the result of column x / (32 / N).
template <int N, bool MAX>
__device__ __forceinline__ float warp_columns(const float* v, int lane) {
  float a[N];
#pragma unroll
  for (int c = 0; c < N; ++c) a[c] = v[c];
  int n = N;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = lane & o;
#pragma unroll
      for (int c = 0; c < N / 2; ++c) {
        if (c < n) {
          const float mine = up ? a[c + n] : a[c], give = up ? a[c] : a[c + n];
          const float got = __shfl_xor_sync(0xffffffffu, give, o);
          a[c] = MAX ? fmaxf(mine, got) : mine + got;
        }
      }
    } else {
      const float got = __shfl_xor_sync(0xffffffffu, a[0], o);
      a[0] = MAX ? fmaxf(a[0], got) : a[0] + got;
    }
  }
  return a[0];
}

// barrier of `nthreads` threads that also tells every one of them whether `pred` holds in any
__device__ __forceinline__ bool named_bar_any(int id, int nthreads, bool pred) {
  int r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %3, 0;\n\t"
      "barrier.cta.red.or.pred q, %1, %2, p;\n\t"
      "selp.b32 %0, 1, 0, q;\n\t}"
      : "=r"(r)
      : "r"(id), "r"(nthreads), "r"((int)pred)
      : "memory");
  return r != 0;
}

struct LatentDecodeShape {
  int nc, chunks, pairs, stages;      // 64-column chunks of c, of the whole row; ceil(nc / 2); ring stages
  int tmem_cols;
};

template <int N>
__device__ __forceinline__ void tmem_ld_heads(uint32_t addr, float* v) {
  if constexpr (N == 32) tmem_ld32(addr, v);
  else tmem_ld16(addr, v);
}

// Descriptors of a stage whose 8-key groups are `group` bytes apart: keys x columns (K-major), and the same rows read as
// columns x keys (MN-major, 64-column chunks 1024 bytes apart).  Adding n to a descriptor moves its start by 16 n bytes.
__device__ __forceinline__ uint64_t desc_rows(uint32_t addr, uint32_t group) {
  return (umma_desc_sw128(addr) & ~(static_cast<uint64_t>(0x3FFF) << 32)) | (static_cast<uint64_t>(group >> 4) << 32);
}
__device__ __forceinline__ uint64_t desc_columns(uint32_t addr, uint32_t group) {
  return (umma_desc_mn_sw128(addr, 1024) & ~(static_cast<uint64_t>(0x3FFF) << 32)) | (static_cast<uint64_t>(group >> 4) << 32);
}

// As umma_bf16, by a whole warp in step: one elected lane issues.
__device__ __forceinline__ void umma_bf16_elect(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "@e tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}

template <int N>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_c, const LatentAttnParams p,
                     const LatentDecodeShape sh) {
  extern __shared__ __align__(1024) uint8_t smem[];
  constexpr int QCH = N * 128;                               // bytes of one 64-column chunk of q', or of the weights of a tile
  const uint32_t group = sh.chunks * 1024, stage_bytes = LD_GROUPS * group;
  uint8_t* ring = smem;
  uint8_t* q_s = ring + sh.stages * stage_bytes;
  uint8_t* p_s = q_s + sh.chunks * QCH;                      // [2]
  float* s_max = reinterpret_cast<float*>(p_s + 2 * QCH);    // [4][32]
  float* s_sum = s_max + 128;                                // [4][32]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_sum + 128);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;                               // [2]
  uint64_t* p_ready = bars + 3;                              // [2]
  uint64_t* pv_done = bars + 5;                              // [2]
  uint64_t* full = bars + 7;                                 // [stages]
  uint64_t* empty = full + LD_MAX_STAGES;                    // [stages]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(empty + LD_MAX_STAGES);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  if ((smem_u32(smem) & 1023u) != 0) {                       // the swizzled tiles need a 1024-byte aligned base
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) atomicCAS(p.status, 0, STATUS_BAD_INDEX);
    return;
  }
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int g = 0; g < 2; ++g) { mbar_init(&s_full[g], 1); mbar_init(&p_ready[g], 128); mbar_init(&pv_done[g], 1); }
    for (int s = 0; s < sh.stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    *abort_flag = 0;
    mbar_fence_init();
    prefetch_tensormap(&tm_q);
    prefetch_tensormap(&tm_c);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, sh.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();            // only now: a successor must not take the tensor memory first
  pdl_wait();
  const uint32_t tmem_s = __shfl_sync(0xffffffffu, *tmem_slot, 0), tmem_o = tmem_s + 2 * N;
  const int h0 = blockIdx.x * N, t = blockIdx.y, split = blockIdx.z;
  const int i = __shfl_sync(0xffffffffu, p.pos[t], 0);
  const int lo = p.window > i ? 0 : i - p.window + 1;        // first visible key
  const int tile0 = lo / LD_TILE, tiles = i / LD_TILE + 1, per = (tiles - tile0 + p.n_split - 1) / p.n_split;
  const int tb = tile0 + split * per, te = min(tiles, tb + per), n_tiles = max(0, te - tb);

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0 && n_tiles > 0) {
      mbar_expect_tx(q_full, sh.chunks * QCH);
      for (int k = 0; k < sh.chunks; ++k) tma_load_3d(q_s + k * QCH, &tm_q, k * 64, t, h0, q_full);
      const int* pt = p.page_table + (size_t)p.row[t] * p.max_pages;
      const int last_page = i / LD_PAGE;
      int st = 0, ph = 1;
      for (int n = 0; n < n_tiles; ++n) {
        int page[LD_TILE / LD_PAGE];
#pragma unroll
        for (int u = 0; u < LD_TILE / LD_PAGE; ++u) {
          const int a = (tb + n) * (LD_TILE / LD_PAGE) + u;
          page[u] = a <= last_page ? pt[a] : p.n_pages;      // rows past the pool read as zeros
        }
        mbar_wait(&empty[st], ph, abort_flag, p.status, STATUS_TIMEOUT_STAGE_EMPTY);
        if (*abort_flag) break;
        mbar_expect_tx(&full[st], stage_bytes);
#pragma unroll
        for (int u = 0; u < LD_GROUPS; ++u)
          tma_load_3d(ring + st * stage_bytes + u * group, &tm_c, 0, page[u / 2] * LD_PAGE + (u & 1) * 8, 0, &full[st]);
        if (++st == sh.stages) { st = 0; ph ^= 1; }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issuer (whole warp): scores of tile n, then the weighted sum of tile n - 1 ----------------
    if (n_tiles > 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(64, N);
      constexpr uint32_t idesc_o = umma_idesc_bf16(128, N) | (1u << 15);     // A (c) read transposed
      const uint64_t rows0 = desc_rows(smem_u32(ring), group), cols0 = desc_columns(smem_u32(ring), group);
      const uint64_t q0 = umma_desc_sw128(smem_u32(q_s)), w0 = umma_desc_sw128(smem_u32(p_s));
      const uint32_t stage16 = stage_bytes >> 4, group16 = group >> 4;
      mbar_wait(q_full, 0, abort_flag, p.status, STATUS_TIMEOUT_TMA_FULL);
      __syncwarp();
      int st = 0, ph = 0, prev = 0;
      for (int n = 0; n <= n_tiles; ++n) {                   // after an abort every wait returns at once
        if (n < n_tiles) {
          mbar_wait(&full[st], ph, abort_flag, p.status, STATUS_TIMEOUT_TMA_FULL);
          __syncwarp();
          tc_fence_after();
          uint64_t a = rows0 + st * stage16, b = q0;
          const uint32_t d = tmem_s + (n & 1) * N;
          uint32_t acc = 0u;
#pragma unroll 3
          for (int k = 0; k < sh.chunks; ++k, a += 64, b += QCH / 16) {
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
              umma_bf16_elect(d, a + 2 * ks, b + 2 * ks, idesc_s, acc);
              acc = 1u;
            }
          }
          if (elect_one()) umma_commit(&s_full[n & 1]);
          __syncwarp();
        }
        if (n > 0) {
          const int m = n - 1;
          mbar_wait(&p_ready[m & 1], (m >> 1) & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
          __syncwarp();
          tc_fence_after();
          uint64_t a = cols0 + prev * stage16;
          const uint64_t w = w0 + (m & 1) * (QCH / 16);
          // an odd last pair takes in the chunk behind c as well: its sums lie on lanes that nobody reads
#pragma unroll 2
          for (int q = 0; q < sh.pairs; ++q, a += 128) {
#pragma unroll
            for (int ks = 0; ks < LD_TILE / 16; ++ks)
              umma_bf16_elect(tmem_o + q * N, a + ks * 2 * group16, w + 2 * ks, idesc_o, (m > 0 || ks > 0) ? 1u : 0u);
          }
          if (elect_one()) {
            umma_commit(&empty[prev]);
            umma_commit(&pv_done[m & 1]);
          }
          __syncwarp();
        }
        prev = st;
        if (++st == sh.stages) { st = 0; ph ^= 1; }
      }
    }
  } else {
    // ---------------- softmax / epilogue ----------------
    const int qd = warp & 3, key = qd * 16 + lane;           // lanes 0..15 of the first three quadrants hold the tile's keys
    const bool mine = lane < 16 && key < LD_TILE;
    const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
    const float sc = p.scale * LD_LOG2E;
    float m[N], sum[N];                                      // reference maxima, the same in every thread; weights of its keys
#pragma unroll
    for (int c = 0; c < N; ++c) { m[c] = -INFINITY; sum[c] = 0.f; }
    for (int n = 0; n < n_tiles; ++n) {
      const int g = n & 1;
      const int j = (tb + n) * LD_TILE + key;
      const bool seen = mine && j <= i && j >= lo;
      float v[N];
      bool over = false;
      mbar_wait(&s_full[g], (n >> 1) & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
      __syncwarp();
      tc_fence_after();
      tmem_ld_heads<N>(tmem_s + g * N + lane_off, v);
      tmem_ld_wait();
      tc_fence_before();
#pragma unroll
      for (int c = 0; c < N; ++c) {
        v[c] = seen ? v[c] * sc : -INFINITY;
        over = over || v[c] > m[c] + 8.0f;
      }
      if (named_bar_any(1, 128, over)) {                     // some head's maximum grows: reduce, and rescale what is there
        s_max[qd * 32 + lane] = warp_columns<N, true>(v, lane);
        named_bar_sync(1, 128);
        float f[N];
        bool any = false;
#pragma unroll
        for (int c = 0; c < N; ++c) {
          const float* x = s_max + c * (32 / N);
          const float mx = fmaxf(fmaxf(x[0], x[32]), fmaxf(x[64], x[96]));
          const bool grow = mx > m[c] + 8.0f;
          f[c] = grow && m[c] != -INFINITY ? exp2f(m[c] - mx) : 1.0f;
          any = any || f[c] != 1.0f;
          if (grow) m[c] = mx;
          sum[c] *= f[c];
        }
        if (n > 0 && any) {                                  // the same in all threads
          mbar_wait(&pv_done[g ^ 1], ((n - 1) >> 1) & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
          __syncwarp();
          tc_fence_after();
          for (int q = 0; q < sh.pairs; ++q) {
            float o[N];
            tmem_ld_heads<N>(tmem_o + lane_off + q * N, o);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < N; ++c) tmem_st1(tmem_o + lane_off + q * N + c, o[c] * f[c]);
          }
          tmem_st_wait();
          tc_fence_before();
        }
        named_bar_sync(1, 128);                              // s_max is read
      }
      if (n > 1) mbar_wait(&pv_done[g], ((n - 2) >> 1) & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);     // its weights are read
      if (mine) {
        uint8_t* pd = p_s + g * QCH + (key & 7) * 2;
#pragma unroll
        for (int c = 0; c < N; ++c) {
          const float w = ex2_approx(v[c] - m[c]);           // 0 for a key that is not seen
          sum[c] += w;
          *reinterpret_cast<__nv_bfloat16*>(pd + c * 128 + (((key >> 3) ^ (c & 7)) << 4)) = __float2bfloat16_rn(w);
        }
        fence_proxy_async_smem();
      }
      mbar_arrive(&p_ready[g]);
    }
    // denominators: over the keys of every warp
    s_sum[qd * 32 + lane] = warp_columns<N, false>(sum, lane);
    named_bar_sync(1, 128);
    float den[N];
#pragma unroll
    for (int c = 0; c < N; ++c) {
      const float* x = s_sum + c * (32 / N);
      den[c] = x[0] + x[32] + x[64] + x[96];
    }
    if (n_tiles > 0) mbar_wait(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
    __syncwarp();
    tc_fence_after();
    const int stride = p.Rp + 2;
    if (p.n_split > 1) {
      if (threadIdx.x == 64) {
#pragma unroll
        for (int c = 0; c < N; ++c) {
          if (h0 + c < p.heads) {
            float* w = p.ws + (((size_t)t * p.heads + h0 + c) * p.n_split + split) * stride + p.Rp;
            w[0] = m[c];
            w[1] = den[c];
          }
        }
      }
    } else {
#pragma unroll
      for (int c = 0; c < N; ++c) {
        float f = 1.0f / den[c];
        if (p.sink != nullptr && h0 + c < p.heads) {
          const float sk = p.sink[h0 + c], top = fmaxf(m[c], sk), e = exp2f(m[c] - top);
          f = e / (den[c] * e + exp2f(sk - top));
        }
        den[c] = f;
      }
    }
    for (int q = 0; q < sh.pairs; ++q) {
      float o[N];
      if (n_tiles > 0) {
        tmem_ld_heads<N>(tmem_o + lane_off + q * N, o);
        tmem_ld_wait();
      } else {
#pragma unroll
        for (int c = 0; c < N; ++c) o[c] = 0.f;
      }
      const int d = q * 128 + qd * 32 + lane;
      if (d >= p.Rp) continue;                               // Rp is a multiple of 64: whole warps
#pragma unroll
      for (int c = 0; c < N; ++c) {
        if (h0 + c < p.heads) {
          if (p.n_split == 1)
            reinterpret_cast<__nv_bfloat16*>(p.out)[((size_t)(h0 + c) * p.npad + t) * p.Rp + d] = __float2bfloat16_rn(o[c] * den[c]);
          else
            p.ws[(((size_t)t * p.heads + h0 + c) * p.n_split + split) * stride + d] = o[c];
        }
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_s, sh.tmem_cols);
  }
}

// o = sum over the splits, each against the common maximum: grid (token x head, ceil(Rp / 128)), one latent per thread
__global__ void __launch_bounds__(128) latent_decode_merge_kernel(const LatentAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float s_w[64];
  const int h = blockIdx.x % p.heads, t = blockIdx.x / p.heads, stride = p.Rp + 2;
  const float* w = p.ws + (size_t)blockIdx.x * p.n_split * stride;
  if (threadIdx.x < 32) {                        // up to 64 splits, two per lane
    const int lane = threadIdx.x;
    float m[2], l[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int s = lane + 32 * u;
      m[u] = s < p.n_split ? w[s * stride + p.Rp] : -INFINITY;
      l[u] = s < p.n_split ? w[s * stride + p.Rp + 1] : 0.f;
    }
    float mx = warp_max(fmaxf(m[0], m[1]));
    if (p.sink != nullptr) mx = fmaxf(mx, p.sink[h]);
    float e[2], den = 0.f;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      e[u] = m[u] != -INFINITY ? exp2f(m[u] - mx) : 0.f;
      den += e[u] * l[u];
    }
    den = warp_sum(den);
    if (p.sink != nullptr) den += exp2f(p.sink[h] - mx);
    const float f = den > 0.f ? 1.0f / den : 0.f;
    s_w[lane] = e[0] * f;
    s_w[lane + 32] = e[1] * f;
  }
  __syncthreads();
  const int d = blockIdx.y * 128 + threadIdx.x;
  if (d >= p.Rp) return;
  float num = 0.f;
#pragma unroll 8
  for (int s = 0; s < p.n_split; ++s) num = fmaf(s_w[s], w[s * stride + d], num);      // an empty split holds zeros
  reinterpret_cast<__nv_bfloat16*>(p.out)[((size_t)h * p.npad + t) * p.Rp + d] = __float2bfloat16_rn(num);
}

// bf16 3-D tensor, 64-element inner boxes with the 128-byte swizzle
static int map_3d(CUtensorMap* m, const void* base, cuuint64_t d0, cuuint64_t d1, cuuint64_t d2, cuuint64_t s1, cuuint64_t s2,
                  unsigned b1, unsigned b2) {
  PfEncodeFn fn = pf_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || s1 % 8 || s2 % 8) return -2;
  cuuint64_t dims[3] = {d0, d1, d2}, strides[2] = {s1 * 2, s2 * 2};
  cuuint32_t box[3] = {64u, b1, b2}, estr[3] = {1u, 1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}

// Ring geometry for N heads per CTA; false when two stages do not fit.  The score product reads two groups of 8 rows past its
// stage: behind the last one lie q' and the weights, which are at least as large.
template <int N>
static bool latent_decode_shape(int Rp, int rw, LatentDecodeShape* sh, size_t* smem) {
  sh->nc = Rp / 64;
  sh->chunks = (Rp + rw) / 64;
  sh->pairs = (sh->nc + 1) / 2;
  const size_t stage = (size_t)LD_GROUPS * sh->chunks * 1024, fixed = (size_t)(sh->chunks + 2) * N * 128 + 2048, cap = 227 * 1024;
  if (rw % 64 || fixed + 2 * stage > cap) return false;
  sh->stages = (int)((cap - fixed) / stage);
  if (sh->stages > LD_MAX_STAGES) sh->stages = LD_MAX_STAGES;
  int cols = 32;
  while (cols < (2 + sh->pairs) * N) cols *= 2;
  sh->tmem_cols = cols;
  *smem = fixed + (size_t)sh->stages * stage;
  return cols <= 512;
}

template <int N>
static int launch_latent_decode(const LatentAttnParams& p, cudaStream_t stream) {
  LatentDecodeShape sh;
  size_t smem;
  if (!latent_decode_shape<N>(p.Rp, p.rw, &sh, &smem)) return -2;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(latent_decode_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -10;
    configured = true;
  }
  const int len = p.Rp + p.rw;
  CUtensorMap mq, mc;
  int rc;
  if ((rc = map_3d(&mq, p.q, p.lq, p.npad, p.heads, p.lq, (cuuint64_t)p.npad * p.lq, 1, N))) return rc;
  // the pool as [tokens][chunks of 64 columns], in boxes of 8 tokens x the whole row that land chunk by chunk
  if ((rc = map_3d(&mc, p.cache, 64, (cuuint64_t)LD_PAGE * p.n_pages, sh.chunks, len, 64, 8, sh.chunks))) return rc;
  cudaError_t e = launch_chain(latent_decode_kernel<N>, dim3((p.heads + N - 1) / N, p.n, p.n_split), dim3(LD_THREADS), smem, stream, mq, mc, p, sh);
  if (e == cudaSuccess && p.n_split > 1) e = launch_chain(latent_decode_merge_kernel, dim3(p.n * p.heads, (p.Rp + 127) / 128), dim3(128), 0, stream, p);
  return e == cudaSuccess ? 0 : -3;
}

}  // namespace tahb

using namespace tahb;

extern "C" int tahb_latent_post(const LatentPostParams* p, int f32, cudaStream_t stream) {
  if (p->M <= 0) return 0;
  if (p->Qp % 4 || p->Rp % 64 || p->rw % 8 || p->rot % 2 || p->rot > p->rw || p->q_col % 4 || p->c_col % 4 || p->ld % 4) return -2;
  cudaError_t e = f32 ? launch_chain(latent_post_kernel<float>, dim3(p->M), dim3(128), 0, stream, *p)
                      : launch_chain(latent_post_kernel<__nv_bfloat16>, dim3(p->M), dim3(128), 0, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}

extern "C" int tahb_latent_query(const LatentQueryParams* p, int f32, cudaStream_t stream) {
  if (p->n <= 0) return 0;
  if (p->rot % 2 || p->dim + p->rot > p->dk || p->dk > p->dq || p->n_list > p->npad) return -2;
  const dim3 grid(p->n, p->n <= 1024 ? (p->heads + 1) / 2 : 1);           // few tokens: spread their heads over the SMs
  cudaError_t e = f32 ? launch_chain(latent_query_kernel<float>, grid, dim3(256), 0, stream, *p)
                      : launch_chain(latent_query_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}

// row_bytes: cached row; lp_bytes: output row pitch (both multiples of 16)
extern "C" int tahb_latent_gather(const void* cache, const int* src, int n, int n_pool, int page_size, int row_bytes, int lp_bytes,
                                  void* out, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (row_bytes % 16 || lp_bytes % 16 || lp_bytes < row_bytes) return -2;
  cudaError_t e = launch_chain(latent_gather_kernel, dim3(n), dim3(128), 0, stream, reinterpret_cast<const uint4*>(cache), src, n_pool,
                               page_size, row_bytes / 16, lp_bytes / 16, reinterpret_cast<uint4*>(out));
  return e == cudaSuccess ? 0 : -3;
}

extern "C" int tahb_latent_gate(const void* list, int npad, int ld_list, const void* gate, long long ld_gate, void* out,
                                long long ld_out, int n, int heads, int dv, int f32, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (dv % 8 || ld_list % 8 || ld_gate % 8 || ((reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(list)) & 15)) return -2;
  const long long work = (long long)n * heads * (dv / 8);
  const dim3 grid((unsigned)((work + 255) / 256));
  cudaError_t e = f32 ? launch_chain(latent_gate_kernel<float>, grid, dim3(256), 0, stream, reinterpret_cast<const float*>(list), npad,
                                     ld_list, reinterpret_cast<const float*>(gate), ld_gate, reinterpret_cast<float*>(out), ld_out, n, heads, dv)
                      : launch_chain(latent_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, reinterpret_cast<const __nv_bfloat16*>(list),
                                     npad, ld_list, reinterpret_cast<const __nv_bfloat16*>(gate), ld_gate,
                                     reinterpret_cast<__nv_bfloat16*>(out), ld_out, n, heads, dv);
  return e == cudaSuccess ? 0 : -3;
}

static int check_latent(const LatentAttnParams* p) {
  return p->Rp % 64 || p->Rp < 64 || p->rw % 8 || p->rw < 8 || p->lq < p->Rp + p->rw || p->lq % 8 || p->n > p->npad ||
         p->heads < 1 || p->heads > 65535 || p->window < 1 ? -2 : 0;
}

extern "C" int tahb_latent_attn_plain(const LatentAttnParams* p, int f32, cudaStream_t stream) {
  if (p->n <= 0) return 0;
  if (check_latent(p)) return -2;
  const size_t smem = ((size_t)2 * p->Rp + p->rw + 128 + 8 + 128) * 4;
  if (smem > 48 * 1024) return -2;
  const dim3 grid(p->n, p->heads);
  cudaError_t e = f32 ? launch_chain(latent_attn_plain_kernel<float>, grid, dim3(128), smem, stream, *p)
                      : launch_chain(latent_attn_plain_kernel<__nv_bfloat16>, grid, dim3(128), smem, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}

// 1 when the decode kernel covers these sizes
extern "C" int tahb_latent_decode_fits(int heads, int Rp, int rw) {
  LatentDecodeShape sh;
  size_t smem;
  return (heads <= 16 ? latent_decode_shape<16>(Rp, rw, &sh, &smem) : latent_decode_shape<32>(Rp, rw, &sh, &smem)) ? 1 : 0;
}

// One query token per entry; ws: n * heads * n_split * (Rp + 2) floats when n_split > 1.
extern "C" int tahb_latent_attn_decode(const LatentAttnParams* p, cudaStream_t stream) {
  if (p->n <= 0) return 0;
  if (check_latent(p) || p->n > 65535 || p->n_split < 1 || p->n_split > 64) return -2;
  if (p->page_size != LD_PAGE) return -5;
  if (p->n_split > 1 && p->ws == nullptr) return -4;
  return p->heads <= 16 ? launch_latent_decode<16>(*p, stream) : launch_latent_decode<32>(*p, stream);
}
