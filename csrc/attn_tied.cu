// Tied attention layers, whose values are their keys as projected (the cache holds K only; see attn_window.cu for the rule and the
// layout): keys, block means and norms on their way to the cache, and the attention of single tokens.
#include "attn_window.cuh"

namespace tahb {

// ---------------------------------------------------------------------------------------------
// Keys of tied layers without norm, bias and rotation, [M, nkv * dk] of pitch ld: to the paged cache, and when a token is the
// last of a block of P, the mean of the block to the pooled rows.  One warp per (token, head), 8 dims per lane.  The block's other
// keys come from the projection when they are tokens of the same step (their cache writes may not have happened yet), from the
// cache otherwise, oldest first: the sum does not depend on how a prompt was cut.
// ---------------------------------------------------------------------------------------------
struct TiedKeysParams {
  const void* k;              // [M, ld]
  void* cache;                // [pages][nkv][page_size][dk]
  void* pooled;               // [pages][nkv][pool_rows][dk], or null
  const int* slot;            // [M], negative = nothing to do
  const int* pos;
  const int* row;
  const int* page_table;      // [rows, max_pages]
  int M, nkv, dk, page_size, max_pages, pool, pool_rows;
  long long ld;
};

template <typename T>
__global__ void __launch_bounds__(128) tied_keys_kernel(const TiedKeysParams p) {
  pdl_launch_dependents();
  pdl_wait();
  using R = typename Row8<T>::type;
  const long long wg = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31, c = lane * 8;
  if (wg >= (long long)p.M * p.nkv) return;
  const int t = (int)(wg / p.nkv), g = (int)(wg % p.nkv), sl = p.slot[t];
  if (sl < 0) return;
  const T* src0 = reinterpret_cast<const T*>(p.k) + (size_t)t * p.ld + (size_t)g * p.dk;
  T* cache = reinterpret_cast<T*>(p.cache);
  auto at = [&](int page, int off) { return (((size_t)page * p.nkv + g) * p.page_size + off) * p.dk; };
  if (c < p.dk) *reinterpret_cast<R*>(cache + at(sl / p.page_size, sl % p.page_size) + c) = *reinterpret_cast<const R*>(src0 + c);
  if (p.pooled == nullptr) return;
  const int i = p.pos[t], r = p.row[t], P = p.pool;
  if ((i + 1) % P) return;
  const int* pt = p.page_table + (size_t)r * p.max_pages;
  float sum[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) sum[e] = 0.f;
  for (int k0 = P - 1; k0 >= 0; k0 -= 32) {                      // every lane finds one of the next 32 keys
    const int k = k0 - lane, u = t - max(k, 0);
    const T* q = src0;
    if (k >= 0) {
      const bool here = u >= 0 && p.row[max(u, 0)] == r && p.pos[max(u, 0)] == i - k;
      q = here ? src0 - (size_t)k * p.ld : cache + at(pt[(i - k) / p.page_size], (i - k) % p.page_size);
    }
    const int n = min(32, k0 + 1);
#pragma unroll 8
    for (int j = 0; j < n; ++j) {
      const T* f = reinterpret_cast<const T*>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(q), j)) + min(c, p.dk - 8);
      float v[8];
      load8(f, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) sum[e] += v[e];
    }
  }
  if (c >= p.dk) return;
  const int b = i / P;
  T* dst = reinterpret_cast<T*>(p.pooled) + (((size_t)pt[b / p.pool_rows] * p.nkv + g) * p.pool_rows + b % p.pool_rows) * p.dk + c;
#pragma unroll
  for (int e = 0; e < 8; ++e) dst[e] = from_f<T>(sum[e] / (float)P);
}

// Pooled rows one after another for the portion kernel: out[r][g * dk + d] = pooled row src[r] (page * pool_rows + row), zeros
// where src[r] is negative.  16-byte units.
__global__ void __launch_bounds__(128) pool_gather_kernel(const uint4* __restrict__ pooled, const int* __restrict__ src, int nkv, int units,
                                                          int pool_rows, int n_pages, uint4* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int s = src[blockIdx.x], page = s < 0 ? -1 : s / pool_rows;
  for (int i = threadIdx.x; i < nkv * units; i += 128) {
    const int g = i / units, c = i % units;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (page >= 0 && page < n_pages) v = pooled[(((size_t)page * nkv + g) * pool_rows + s % pool_rows) * units + c];
    out[(size_t)blockIdx.x * nkv * units + i] = v;
  }
}

// ---------------------------------------------------------------------------------------------
// RMS norms of q and k over all heads of a token, for tied layers: q times its factor and the weights of both norms to q_out, the
// projected k to the paged cache, k's factor to the factors beside it.  One CTA per token.
// ---------------------------------------------------------------------------------------------
struct NormAllParams {
  const void* q;              // [M, ld]: nq heads of dk
  const void* k;              // the same rows: nkv heads of dk
  const float* w;             // [nq * dk]: weight of q's norm times that of the key head it meets (padding dims zero)
  void* q_out;                // [M, nq * dk]
  void* cache;                // [pages][nkv][page_size][dk]
  float* factor;              // [pages][page_size]
  const int* slot;            // [M], negative = no cache write
  int M, nq, nkv, dk, dim, page_size;
  long long ld;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(256) norm_all_kernel(const NormAllParams p) {
  pdl_launch_dependents();
  pdl_wait();
  using R = typename Row8<T>::type;
  __shared__ float red[2][8];
  const size_t t = blockIdx.x;
  const T* q = reinterpret_cast<const T*>(p.q) + t * p.ld;
  const T* k = reinterpret_cast<const T*>(p.k) + t * p.ld;
  const int sl = p.slot[t], cq = p.nq * p.dk, ck = p.nkv * p.dk;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * 8; c < cq; c += 2048) {
    float v[8];
    load8(q + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) sq = fmaf(v[e], v[e], sq);
  }
  for (int c = threadIdx.x * 8; c < ck; c += 2048) {
    float v[8];
    load8(k + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) sk = fmaf(v[e], v[e], sk);
    if (sl >= 0) {
      const int g = c / p.dk;
      T* dst = reinterpret_cast<T*>(p.cache) + (((size_t)(sl / p.page_size) * p.nkv + g) * p.page_size + sl % p.page_size) * p.dk + c % p.dk;
      *reinterpret_cast<R*>(dst) = *reinterpret_cast<const R*>(k + c);
    }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = sq;
    red[1][threadIdx.x >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) {
    sq += red[0][w];
    sk += red[1][w];
  }
  if (threadIdx.x == 0 && sl >= 0) p.factor[sl] = 1.0f / sqrtf(sk / (float)(p.nkv * p.dim) + p.eps);
  const float r = 1.0f / sqrtf(sq / (float)(p.nq * p.dim) + p.eps);
  for (int c = threadIdx.x * 8; c < cq; c += 2048) {
    float v[8], w[8];
    load8(q + c, v);
    load8(p.w + c, w);
    T o[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = from_f<T>(v[e] * r * w[e]);
    *reinterpret_cast<R*>(reinterpret_cast<T*>(p.q_out) + t * cq + c) = *reinterpret_cast<const R*>(o);
  }
}

// ---------------------------------------------------------------------------------------------
// Decode kernel (bf16, pages of 16): up to 8 query heads of one key head and token per CTA, grid (nkv * groups, n, n_split).
// Warp 4 streams pages of the window into a ring, one stage each: 64-column chunks [16 keys][128 bytes], swizzled.  16 pooled
// blocks, which are scattered rows, count as a page in front of those; the warp that works on one gathers it itself.  Warps 0..3
// take a page in turn.
// Keys are bound by HBM only while little work is done per key, so both products are warp-level m16n8k16 (a tile of eight heads
// is a fraction of a tcgen05 one, and keys read once feed both without leaving shared memory):
//   scores  [heads x 16 keys]: A = queries, rows 8..15 zero, B = keys;
//   output  [heads x dims]:    A = weights as a bf16 pair, high parts in rows 0..7 and low parts in rows 8..15, B = keys transposed.
// So the weights keep 2^-17 of relative accuracy at no cost.  A head's reference maximum moves only when a score is 2^8 times above
// it, hence rarely.  slope and sink in log2 units.
// ---------------------------------------------------------------------------------------------
constexpr int TD_HEADS = 8, TD_THREADS = 160;

template <int HK>
struct TdCfg {
  static constexpr int PAGE_BYTES = HK * 2048, NSTAGE = HK == 1 ? 16 : 8;
  static constexpr int Q_PITCH = HK * 128 + 16;              // bytes of a query in shared memory (rows fall into different banks)
  static constexpr int RING_BYTES = NSTAGE * (PAGE_BYTES + 64) + TD_HEADS * Q_PITCH + NSTAGE * 16 + 64;
  static constexpr int MEANS_AT = (RING_BYTES + 1023) / 1024 * 1024;                     // the warps' own pages: pooled layers only
  static constexpr int SMEM_BYTES = MEANS_AT + 8 * PAGE_BYTES;
  static constexpr int MIN_CTAS = HK <= 2 ? 3 : 1;
};

__device__ __forceinline__ void tma_load_5d(void* smem_dst, const void* tmap, int c0, int c1, int c2, int c3, int c4, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.5d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6, %7}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(tmap)), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(c4)
      : "memory");
}
// 16 bytes to shared memory, zeros unless `live`
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_16816(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// (a, b) as a pair of bf16 numbers and what is missing
__device__ __forceinline__ void pair_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <int HK>
__global__ void __launch_bounds__(TD_THREADS, TdCfg<HK>::MIN_CTAS)
tied_decode_kernel(const __grid_constant__ CUtensorMap tm_k, const WindowAttnParams p, const int whole) {
  using C = TdCfg<HK>;
  extern __shared__ __align__(1024) uint8_t smem[];
  float* factor_s = reinterpret_cast<float*>(smem + C::NSTAGE * C::PAGE_BYTES);          // [NSTAGE][16]
  uint8_t* q_s = reinterpret_cast<uint8_t*>(factor_s + C::NSTAGE * WD_PAGE);             // [8 heads][HK * 64], zeros behind the real ones
  uint64_t* full = reinterpret_cast<uint64_t*>(q_s + TD_HEADS * C::Q_PITCH);
  uint64_t* empty = full + C::NSTAGE;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty + C::NSTAGE);
  uint8_t* means_s = smem + C::MEANS_AT;         // [4 warps][2]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid == 0) {
    for (int s = 0; s < C::NSTAGE; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    prefetch_tensormap(&tm_k);
  }
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();
  if ((smem_u32(smem) & 1023u) != 0) {          // the swizzled tiles need a 1024-byte aligned base
    if (tid == 0) atomicCAS(p.status, 0, STATUS_BAD_INDEX);
    return;
  }
  const int G = p.nq / p.nkv, groups = (G + TD_HEADS - 1) / TD_HEADS;
  const int kvh = blockIdx.x / groups, grp0 = (blockIdx.x % groups) * TD_HEADS;          // first query head of the group inside kvh
  const int nh = min(TD_HEADS, G - grp0), h0 = kvh * G + grp0;
  const int t = blockIdx.y, split = blockIdx.z, i = p.pos[t];
  const int* pt = p.page_table + (size_t)p.row[t] * p.max_pages;
  const int lo = p.window > i ? 0 : i - p.window + 1;
  const bool pooled = p.pooled != nullptr;
  const int blocks = pooled ? visible_blocks(i, p.window, p.pool) : 0;                    // in the first kp pages
  const int keep_end = min(p.keep_first, lo);
  const int kp = ((pooled ? blocks : keep_end) + WD_PAGE - 1) / WD_PAGE;
  const int w0 = pooled ? lo / WD_PAGE : max(lo / WD_PAGE, kp);
  const int total = kp + max(0, i / WD_PAGE - w0 + 1), per = (total + p.n_split - 1) / p.n_split;
  const int pb = split * per, n_pages = max(0, min(total, pb + per) - pb);

  for (int x = tid; x < TD_HEADS * HK * 8; x += TD_THREADS) {
    const int g = x / (HK * 8), c = x % (HK * 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (g < nh && c * 8 < p.dk)
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.q) + (size_t)t * p.ld_q + (size_t)(h0 + g) * p.dk + c * 8);
    *reinterpret_cast<uint4*>(q_s + g * C::Q_PITCH + c * 16) = v;
  }
  __syncthreads();

  float m = -INFINITY, l = 0.f;                  // of head lane / 4; weights of this lane's keys
  float acc[HK * 8][4];
#pragma unroll
  for (int x = 0; x < HK * 8; ++x)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[x][e] = 0.f;

  if (warp == 4) {
    // window pages (the pooled ones in front of them are the consumers' own business)
    if (lane == 0) {
      const int k0 = pooled ? max(0, min(n_pages, kp - pb)) : 0;
      int next = k0 < n_pages ? pt[pb + k0 < kp ? pb + k0 : w0 + pb + k0 - kp] : 0;
      for (int k = k0, s = 0, ph = 1; k < n_pages; ++k) {
        const int page = next, idx = pb + k + 1;
        if (k + 1 < n_pages) next = pt[idx < kp ? idx : w0 + idx - kp];
        mbar_wait(&empty[s], ph, abort_flag, p.status, STATUS_TIMEOUT_STAGE_EMPTY);
        mbar_expect_tx(&full[s], C::PAGE_BYTES + (p.factor != nullptr ? 64 : 0));
        uint8_t* dst = smem + s * C::PAGE_BYTES;
        if (whole) {
          tma_load_5d(dst, &tm_k, 0, 0, 0, kvh, page, &full[s]);
        } else {
#pragma unroll
          for (int h = 0; h < HK; ++h) tma_load_4d(dst + h * 2048, &tm_k, h * 64, 0, kvh, page, &full[s]);
        }
        if (p.factor != nullptr) bulk_load(factor_s + s * WD_PAGE, p.factor + (size_t)page * WD_PAGE, 64, &full[s]);
        if (++s == C::NSTAGE) { s = 0; ph ^= 1; }
      }
    }
    __syncwarp();
  } else {
    const int g = lane >> 2, q = lane & 3;
    const float scale = query_scale(p, i) * LOG2E, slope = p.slope != nullptr && g < nh ? p.slope[h0 + g] : 0.f;
    const int key_s = (lane & 7) + ((lane >> 4) << 3), ch_s = (lane >> 3) & 1;            // row and chunk this lane addresses: scores,
    const int key_o = lane & 15, ch_o = lane >> 4;                                        // output
    const uint32_t q_addr = smem_u32(q_s) + (lane & 7) * C::Q_PITCH + (lane >> 3) * 16;
    const int n_means = pooled ? max(0, min(n_pages, kp - pb)) : 0;                       // pooled pages of this split, the first ones
    uint8_t* own = means_s + warp * 2 * C::PAGE_BYTES;                                    // two pages that this warp fills itself
    auto fetch = [&](int k) {                    // pooled blocks of page k, a 16-byte chunk per lane and step; zeros where there are none
      const int S = p.pool_rows, cpr = HK * 8, b0 = (pb + k) * WD_PAGE;
#pragma unroll
      for (int x = lane; x < WD_PAGE * HK * 8; x += 32) {
        const int r = x / cpr, c = x % cpr, b = b0 + r;
        const bool live = b < blocks && c * 8 < p.dk;
        const size_t at = live ? (((size_t)pt[b / S] * p.nkv + kvh) * S + b % S) * p.dk + c * 8 : 0;
        cp_async16(smem_u32(own + ((k >> 2) & 1) * C::PAGE_BYTES + (c / 8) * 2048 + r * 128 + ((c % 8) ^ (r & 7)) * 16),
                   reinterpret_cast<const __nv_bfloat16*>(p.pooled) + at, live);
      }
      cp_async_commit();
    };
    if (warp < n_means) fetch(warp);
    int s = (warp - n_means) & 3, ph = 0;        // ring stage of this warp's first window page
    for (int k = warp; k < n_pages; k += 4) {
      const int idx = pb + k;
      const bool means = k < n_means;
      const int j0 = (idx < kp ? idx : w0 + idx - kp) * WD_PAGE;
      uint32_t base;
      if (means) {
        if (k + 4 < n_means) {
          fetch(k + 4);
          cp_async_wait<1>();
        } else {
          cp_async_wait<0>();
        }
        __syncwarp();
        base = smem_u32(own + ((k >> 2) & 1) * C::PAGE_BYTES);
      } else {
        mbar_wait(&full[s], ph, abort_flag, p.status, STATUS_TIMEOUT_TMA_FULL);
        __syncwarp();
        base = smem_u32(smem + s * C::PAGE_BYTES);
      }
      float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};                   // keys 0..7 and 8..15 of the page
#pragma unroll
      for (int x = 0; x < HK * 4; x += 2) {
        uint32_t a[4];                           // queries of 32 dims, rows 0..7 of A
        ldmatrix_x4(q_addr + x * 32, a);
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          uint32_t r[4];
          ldmatrix_x4(base + (x / 4) * 2048 + key_s * 128 + ((((x + y) % 4) * 2 + ch_s) ^ (key_s & 7)) * 16, r);
          mma_16816(c0, a[2 * y], 0u, a[2 * y + 1], 0u, r[0], r[1]);
          mma_16816(c1, a[2 * y], 0u, a[2 * y + 1], 0u, r[2], r[3]);
        }
      }
      float v[4] = {c0[0] * scale, c0[1] * scale, c1[0] * scale, c1[1] * scale};          // keys 2 q, 2 q + 1, 8 + 2 q, 9 + 2 q
      if (p.factor != nullptr && !means) {
        const float2 fa = *reinterpret_cast<const float2*>(factor_s + s * WD_PAGE + 2 * q);
        const float2 fb = *reinterpret_cast<const float2*>(factor_s + s * WD_PAGE + 8 + 2 * q);
        v[0] *= fa.x; v[1] *= fa.y; v[2] *= fb.x; v[3] *= fb.y;
      }
      if (p.bias != nullptr) {
        const float* bias = p.bias + (size_t)(h0 + min(g, nh - 1)) * (p.far + 1);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] += __ldg(bias + min(max(i - j0 - 2 * q - (e & 1) - (e >> 1) * 8, 0), p.far));
      }
      // visible: places first .. first + n - 1, or kept first tokens
      const unsigned first = means ? 0u : lo, n = means ? blocks : i - lo + 1, kept = means ? 0u : min(p.keep_first, i + 1);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const unsigned j = j0 + 2 * q + (e & 1) + (e >> 1) * 8;
        v[e] = j - first < n || j < kept ? fmaf(-slope, (float)(i - (int)j), v[e]) : -INFINITY;
      }
      float top = fmaxf(fmaxf(v[0], v[1]), fmaxf(v[2], v[3]));
      if (__any_sync(0xffffffffu, top > m + 8.0f)) {
        top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1));
        top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 2));
        const bool up = top > m + 8.0f;
        const float corr = !up ? 1.0f : m == -INFINITY ? 0.f : ex2_approx(m - top);
        if (up) m = top;
        l *= corr;
#pragma unroll
        for (int x = 0; x < HK * 8; ++x)
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[x][e] *= corr;
      }
      const float ref = m == -INFINITY ? 0.f : m;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[e] = ex2_approx(v[e] - ref);
        l += v[e];
      }
      uint32_t a0, a1, a2, a3;
      pair_bf16(v[0], v[1], a0, a1);
      pair_bf16(v[2], v[3], a2, a3);
#pragma unroll
      for (int x = 0; x < HK * 4; ++x) {
        uint32_t r[4];
        ldmatrix_x4_trans(base + (x / 4) * 2048 + key_o * 128 + (((x % 4) * 2 + ch_o) ^ (key_o & 7)) * 16, r);
        mma_16816(acc[2 * x], a0, a1, a2, a3, r[0], r[1]);
        mma_16816(acc[2 * x + 1], a0, a1, a2, a3, r[2], r[3]);
      }
      __syncwarp();
      if (!means) {
        if (lane == 0) mbar_arrive(&empty[s]);
        s += 4;
        if (s >= C::NSTAGE) { s -= C::NSTAGE; ph ^= 1; }
      }
    }
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
  }

  // merge the four warps through shared memory (the ring is free now)
  __syncthreads();
  float* sm_m = reinterpret_cast<float*>(smem);              // [4][8]
  float* sm_l = sm_m + 4 * TD_HEADS;                         // [4][8]
  float* sm_o = sm_l + 4 * TD_HEADS;                         // [4][nh][HK * 64]
  if (warp < 4) {
    const int g = lane >> 2, q = lane & 3;
    if (q == 0) {
      sm_m[warp * TD_HEADS + g] = m;
      sm_l[warp * TD_HEADS + g] = l;
    }
    if (g < nh) {
#pragma unroll
      for (int x = 0; x < HK * 8; ++x)
        *reinterpret_cast<float2*>(sm_o + (warp * nh + g) * (HK * 64) + x * 8 + 2 * q) = make_float2(acc[x][0] + acc[x][2], acc[x][1] + acc[x][3]);
    }
  }
  __syncthreads();
  for (int x = tid; x < nh * p.dk; x += TD_THREADS) {
    const int g = x / p.dk, d = x % p.dk, h = h0 + g;
    float mx = -INFINITY, num = 0.f, den = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) mx = fmaxf(mx, sm_m[w * TD_HEADS + g]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = sm_m[w * TD_HEADS + g], f = mw == -INFINITY ? 0.f : ex2_approx(mw - mx);
      num = fmaf(f, sm_o[(w * nh + g) * (HK * 64) + d], num);
      den = fmaf(f, sm_l[w * TD_HEADS + g], den);
    }
    if (p.n_split == 1) {
      reinterpret_cast<__nv_bfloat16*>(p.out)[(size_t)t * p.ld_out + (size_t)h * p.dk + d] =
          __float2bfloat16_rn(num * finish_scale(p, t, h, mx, den) * element_gate(p, t, h, d));
    } else {
      float* w = p.ws + (((size_t)t * p.nq + h) * p.n_split + split) * (p.dk + 2);
      w[d] = num;
      if (d == 0) { w[p.dk] = mx; w[p.dk + 1] = den; }
    }
  }
}

// [pages][kv heads][64-column chunks][16 tokens][64 columns]: a box is a page of one head
static int make_whole_page_map(CUtensorMap* m, const void* base, int d, int nkv, int n_pages) {
  PfEncodeFn fn = pf_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || d % 64) return -2;
  const cuuint64_t row = (cuuint64_t)d * 2, head = row * WD_PAGE;
  cuuint64_t dims[5] = {64, WD_PAGE, (cuuint64_t)d / 64, (cuuint64_t)nkv, (cuuint64_t)n_pages}, strides[4] = {row, 128, head, head * nkv};
  cuuint32_t box[5] = {64u, WD_PAGE, (cuuint32_t)d / 64, 1u, 1u}, estr[5] = {1u, 1u, 1u, 1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 5, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}

template <int HK>
static int launch_tied_decode_as(const WindowAttnParams& p, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(tied_decode_kernel<HK>, cudaFuncAttributeMaxDynamicSharedMemorySize, TdCfg<HK>::SMEM_BYTES) != cudaSuccess) return -10;
    configured = true;
  }
  // a page of one head in one copy when its rows are that many whole chunks, chunk by chunk (zeros behind dk) otherwise
  const int whole = p.dk == HK * 64;
  const size_t page = (size_t)p.nkv * WD_PAGE * p.dk;
  CUtensorMap mk;
  const int rc = whole ? make_whole_page_map(&mk, p.cache, p.dk, p.nkv, p.n_pages)
                       : make_page_map(&mk, p.cache, p.dk, p.nkv, p.n_pages, p.dk, (size_t)WD_PAGE * p.dk, page);
  if (rc) return rc;
  const int groups = (p.nq / p.nkv + TD_HEADS - 1) / TD_HEADS;
  cudaError_t e = launch_chain(tied_decode_kernel<HK>, dim3(p.nkv * groups, p.n, p.n_split), dim3(TD_THREADS),
                               p.pooled != nullptr ? TdCfg<HK>::SMEM_BYTES : TdCfg<HK>::RING_BYTES, stream, mk, p, whole);
  if (e == cudaSuccess && p.n_split > 1) e = launch_window_merge(p, stream);
  return e == cudaSuccess ? 0 : -3;
}

int launch_tied_decode(const WindowAttnParams& p, cudaStream_t stream) {
  if (p.n_pages < 1 || p.ld_q % 8 || (reinterpret_cast<uintptr_t>(p.q) & 15)) return -2;
  return p.dk <= 64 ? launch_tied_decode_as<1>(p, stream) : p.dk <= 128 ? launch_tied_decode_as<2>(p, stream) : launch_tied_decode_as<4>(p, stream);
}

}  // namespace tahb

using namespace tahb;

// Keys (and block means) of a tied layer without norms to the cache.
extern "C" int tahb_tied_keys(const TiedKeysParams* p, int f32, cudaStream_t stream) {
  if (p->M <= 0) return 0;
  if (p->dk > 256 || p->dk % 8 || p->ld % 8 || p->nkv < 1 ||
      (p->pooled != nullptr && (p->pool < 1 || p->pool_rows < 1 || (long long)p->pool_rows * p->pool < p->page_size)))
    return -2;
  const long long warps = (long long)p->M * p->nkv;
  const dim3 grid((unsigned)((warps + 3) / 4));
  cudaError_t e = f32 ? launch_chain(tied_keys_kernel<float>, grid, dim3(128), 0, stream, *p)
                      : launch_chain(tied_keys_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}

// n rows of nkv * row_bytes; src: pooled rows (see pool_gather_kernel)
extern "C" int tahb_pool_gather(const void* pooled, const int* src, int n, int nkv, int row_bytes, int pool_rows, int n_pages, void* out,
                                cudaStream_t stream) {
  if (n <= 0) return 0;
  if (row_bytes % 16 || nkv < 1 || pool_rows < 1) return -2;
  cudaError_t e = launch_chain(pool_gather_kernel, dim3(n), dim3(128), 0, stream, reinterpret_cast<const uint4*>(pooled), src, nkv,
                               row_bytes / 16, pool_rows, n_pages, reinterpret_cast<uint4*>(out));
  return e == cudaSuccess ? 0 : -3;
}

// Norms over all heads, queries out, keys and their factors to the cache.
extern "C" int tahb_norm_all(const NormAllParams* p, int f32, cudaStream_t stream) {
  if (p->M <= 0) return 0;
  if (p->dk % 8 || p->dim > p->dk || p->ld % 8 || p->nq < 1 || p->nkv < 1) return -2;
  cudaError_t e = f32 ? launch_chain(norm_all_kernel<float>, dim3(p->M), dim3(256), 0, stream, *p)
                      : launch_chain(norm_all_kernel<__nv_bfloat16>, dim3(p->M), dim3(256), 0, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}
