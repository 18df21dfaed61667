// Paged attention with a sliding window, kept first tokens or pooled blocks in front of it, a query temperature, a score cap, a
// per-distance bias (a table or a slope), a softmax sink and an output gate per head or per element.
//
// Query at position i of a sequence sees key j when  j <= i  and  (i - j < window  or  j < keep_first).
// score = cap(temp(i) * (q . k) * scale) + bias[h][min(i - j, D)] with cap(s) = softcap * tanh(s / softcap) and
// temp(i) = 1 + temp_coef * ln(floor((i + 1) / temp_every) + 1); softmax over the visible keys with exp(sink_h) added to
// the denominator; out_h *= sigmoid(gate_h).  Every constant is a launch parameter: window = INT_MAX is plain causal
// attention, keep_first = 0 a plain window, softcap = 0 no cap, temp_coef = 0 no temperature, and the bias table, the
// sink and the gate may each be absent.
//
// A slope takes slope_h * (i - j) off a score.  Pooled blocks: block b is the mean of the keys b P .. b P + P - 1 and is seen, as one
// more key and value, when b P + P - 1 <= i - window.
//
// Keys and values are read from the paged cache only (the tokens of the running step are written there first), so
// portions of a prompt, single decoded tokens and layers that read another layer's cache are the same case:
//   page of one layer:  [K: kv_heads][page_size][dk]  then  [V: kv_heads][page_size][dv]
// dk and dv are padded to multiples of 8; padding dims hold zeros.
//   Values that are the keys as projected ("tied"): a page holds K only.  When the keys have a norm over all heads of a token,
//   its weights are folded into the queries and its factor, one number per token, is a page of page_size floats beside the keys:
//   score = factor_j * (q' . k_j), value = k_j.
//   Pooled blocks: a pool of its own under the same page table, with S rows a page ([kv_heads][S][dk], S a power of two >= 16 / P):
//   block b is row b % S of logical page b / S, a page that the row owns by the time the block is complete.
#include "attn_window.cuh"

namespace tahb {

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
// After the fused projection [q | k | v | ...]: bias, per-head RMS norm of q and k, rotation of their first `rot` dims, values
// mixed with those of an earlier layer, q to its own matrix, k and v to the paged cache.  One warp per (token, head); a lane
// owns dim pairs 2 * lane, 2 * lane + 64, ...
//   rotation: entries (a, b) of the pair i become (a cos - b sin, b cos + a sin), pairs (i, i + rot / 2) or (2 i, 2 i + 1)
//   values:   v <- (1 - lambda) v + lambda v_first; without v_first the values are copied to v_keep, for the layers that mix
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
  const float2* rope;         // [M, rot / 2] (cos, sin), or null
  int rot, interleaved;
  const void* v_first;        // [M, nkv * dv] or null
  const float* lambda;        // [1], with v_first
  void* v_keep;               // [M, nkv * dv] or null
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
  float r = 1.0f;
  if (w != nullptr) {
    r = 1.0f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
#pragma unroll
    for (int i = 0; i < MAXP; ++i) {
      const int c = 2 * lane + 64 * i;
      if (c < d) {
        x[2 * i] *= r * w[c];
        x[2 * i + 1] *= r * w[c + 1];
      }
    }
  }
  if (p.rope != nullptr && (is_q || is_k)) {
    const float2* tab = p.rope + (size_t)t * (p.rot / 2);
    const int half = p.rot / 2;
    auto entry = [&](int c) {                   // entry c of the head behind bias and norm (held by another lane)
      float v = to_f<T>(src[c]);
      if (p.bias != nullptr) v += p.bias[col + c];
      return w != nullptr ? v * r * w[c] : v;
    };
#pragma unroll
    for (int i = 0; i < MAXP; ++i) {
      const int c = 2 * lane + 64 * i;
      if (c >= p.rot) continue;
      if (p.interleaved) {                      // rot is even: the pair lies in this lane
        const float2 f = tab[c / 2];
        const float a = x[2 * i], b = x[2 * i + 1];
        x[2 * i] = a * f.x - b * f.y;
        x[2 * i + 1] = b * f.x + a * f.y;
      } else {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int d0 = c + e;                 // d0 < rot, as rot is even
          const bool low = d0 < half;
          const float2 f = tab[low ? d0 : d0 - half];
          const float other = entry(low ? d0 + half : d0 - half);
          x[2 * i + e] = low ? x[2 * i + e] * f.x - other * f.y : x[2 * i + e] * f.x + other * f.y;
        }
      }
    }
  }
  if (!is_q && !is_k && (p.v_first != nullptr || p.v_keep != nullptr)) {
    const size_t at = (size_t)t * p.nkv * p.dv + (size_t)(h - p.nq - p.nkv) * p.dv;
    const float lam = p.v_first != nullptr ? p.lambda[0] : 0.f;
#pragma unroll
    for (int i = 0; i < MAXP; ++i) {
      const int c = 2 * lane + 64 * i;
      if (c < d) {
        if (p.v_first != nullptr) {
          const T* f = reinterpret_cast<const T*>(p.v_first) + at + c;
          x[2 * i] = (1.0f - lam) * x[2 * i] + lam * to_f<T>(f[0]);
          x[2 * i + 1] = (1.0f - lam) * x[2 * i + 1] + lam * to_f<T>(f[1]);
        } else {
          T* f = reinterpret_cast<T*>(p.v_keep) + at + c;
          f[0] = from_f<T>(x[2 * i]);
          f[1] = from_f<T>(x[2 * i + 1]);
        }
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
  const T* q = reinterpret_cast<const T*>(p.q) + (size_t)t * p.ld_q + (size_t)h * p.dk;
  const float scale = query_scale(p, i);
  for (int d = lane; d < p.dk; d += 32) s_q[warp][d] = to_f<T>(q[d]);
  __syncwarp();
  float m = -INFINITY, l = 0.f, acc[2 * MAXP];
#pragma unroll
  for (int c = 0; c < 2 * MAXP; ++c) acc[c] = 0.f;
  int keep_end, lo;
  visible_range(i, p.window, p.keep_first, keep_end, lo);
  if (p.pooled != nullptr) keep_end = visible_blocks(i, p.window, p.pool);
  const float slope = p.slope != nullptr ? p.slope[h] : 0.f;
  for (int part = 0; part < 2; ++part) {
    const int a = part == 0 ? 0 : lo, b = part == 0 ? keep_end : i + 1;
    const bool blocks = part == 0 && p.pooled != nullptr;
    const int ps = blocks ? p.pool_rows : p.page_size;
    const size_t page_elems = (size_t)p.nkv * ps * (p.tied ? p.dk : p.dk + p.dv);
    const T* kc = reinterpret_cast<const T*>(blocks ? p.pooled : p.cache) + (size_t)kvh * ps * p.dk;
    const T* vc = p.tied ? kc : reinterpret_cast<const T*>(p.cache) + (size_t)p.nkv * ps * p.dk + (size_t)kvh * ps * p.dv;
    for (int j0 = a; j0 < b; j0 += 32) {
      const int j = j0 + lane;
      float s = -INFINITY;
      int page = 0;
      if (j < b) {
        page = pt[j / ps];
        const T* k = kc + (size_t)page * page_elems + (size_t)(j % ps) * p.dk;
        float dot = 0.f;
        for (int d = 0; d < p.dk; d += 8) {
          float kv[8];
          load8(k + d, kv);
#pragma unroll
          for (int u = 0; u < 8; ++u) dot = fmaf(s_q[warp][d + u], kv[u], dot);
        }
        s = dot * scale;
        if (p.factor != nullptr) s *= p.factor[(size_t)page * ps + j % ps];
        if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
        if (p.bias != nullptr) s += p.bias[(size_t)h * (p.far + 1) + min(i - j, p.far)];
        s -= slope * (float)(i - j);
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
        const T* v = vc + (size_t)s_page[warp][u] * page_elems + (size_t)((j0 + u) % ps) * p.dv;
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
  f = f / l * p.out_scale;
  if (p.gate != nullptr) f *= sigmoid_f(to_f<T>(reinterpret_cast<const T*>(p.gate)[(size_t)t * p.ld_gate + h]));
  T* o = reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + (size_t)h * p.dv;
  const T* wg_in = p.wide_gate == nullptr ? nullptr : reinterpret_cast<const T*>(p.wide_gate) + (size_t)t * p.ld_gate + (size_t)h * p.dv;
#pragma unroll
  for (int c = 0; c < MAXP; ++c) {
    const int d = 2 * lane + 64 * c;
    if (d < p.dv) {
      if (wg_in != nullptr) {
        acc[2 * c] *= sigmoid_f(to_f<T>(wg_in[d]));
        acc[2 * c + 1] *= sigmoid_f(to_f<T>(wg_in[d + 1]));
      }
      o[d] = from_f<T>(acc[2 * c] * f);
      o[d + 1] = from_f<T>(acc[2 * c + 1] * f);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Decode kernel (bf16, pages of 16): one query per CTA row, all GB query heads of a group share the K / V reads.
// Grid (nkv * groups, n, n_split); warp 4 streams whole K / V page blocks of one KV head with bulk copies through a
// three-stage ring, warps 0..3 are 16 groups of 8 lanes, one token of a page per group.  Only pages that hold a visible
// key are visited: the pages of the kept first tokens, then those of the window.  bias and sink are in log2 units.
// ---------------------------------------------------------------------------------------------
constexpr int WD_STAGE_PAGES = 2;
constexpr int WD_NSTAGE = 3;

// pages of a query at position i: `kp` pages of the kept part, then pages w0 .. i / 16; returns their number
__device__ __forceinline__ int visible_pages(int i, int window, int keep_first, int& kp, int& w0) {
  int keep_end, lo;
  visible_range(i, window, keep_first, keep_end, lo);
  kp = (keep_end + WD_PAGE - 1) / WD_PAGE;
  w0 = max(lo / WD_PAGE, kp);
  return kp + max(0, i / WD_PAGE - w0 + 1);
}

template <int VEC, int GB, bool EXACT, bool CAP>   // EXACT: dk = dv = VEC * 64, known to the compiler; CAP: softcap > 0
__global__ void __launch_bounds__(160, VEC * GB > 4 ? 2 : GB == 4 ? 3 : 4) window_decode_kernel(const WindowAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int DPL = VEC * 8;
  const int dk = EXACT ? VEC * 64 : p.dk, dv = EXACT ? VEC * 64 : p.dv;
  extern __shared__ __align__(128) uint8_t wd_smem[];
  const int kblk = WD_PAGE * dk, vblk = WD_PAGE * dv;              // elements of one K / V block of a page
  const int stage_elems = WD_STAGE_PAGES * (kblk + vblk);
  __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(wd_smem);
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(wd_smem + (size_t)WD_NSTAGE * stage_elems * 2);
  uint64_t* empty_bar = full_bar + WD_NSTAGE;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty_bar + WD_NSTAGE);

  const int G = p.nq / p.nkv, groups = (G + GB - 1) / GB;
  const int kvh = blockIdx.x / groups, grp0 = (blockIdx.x % groups) * GB;   // first query head of the group inside kvh
  const int t = blockIdx.y, split = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int i = p.pos[t];
  const int* pt = p.page_table + (size_t)p.row[t] * p.max_pages;
  int kp, w0;
  const int total = visible_pages(i, p.window, p.keep_first, kp, w0);
  const int lo = p.window > i ? 0 : i - p.window + 1;
  const int ppc = (total + p.n_split - 1) / p.n_split;
  const int pb = split * ppc, pe = min(total, pb + ppc);
  const int n_iter = pe > pb ? (pe - pb + WD_STAGE_PAGES - 1) / WD_STAGE_PAGES : 0;

  if (tid == 0) {
    for (int s = 0; s < WD_NSTAGE; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 4);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  __syncthreads();

  float m[GB], l[GB], acc[GB][DPL];
#pragma unroll
  for (int g = 0; g < GB; ++g) {
    m[g] = -INFINITY;
    l[g] = 0.f;
#pragma unroll
    for (int c = 0; c < DPL; ++c) acc[g][c] = 0.f;
  }
  const int grp = (warp & 3) * 4 + (lane >> 3);
  const int gl = lane & 7;

  if (warp == 4) {
    if (lane == 0) {
      const size_t page_elems = (size_t)p.nkv * (kblk + vblk);
      for (int it = 0; it < n_iter; ++it) {
        const int s = it % WD_NSTAGE;
        mbar_wait(&empty_bar[s], ((it / WD_NSTAGE) & 1) ^ 1, abort_flag, p.status, STATUS_TIMEOUT_STAGE_EMPTY);
        const int first = pb + it * WD_STAGE_PAGES;
        const int n_here = min(WD_STAGE_PAGES, pe - first);
        mbar_expect_tx(&full_bar[s], n_here * (kblk + vblk) * 2);
        for (int u = 0; u < n_here; ++u) {
          const int idx = first + u;
          const int page = pt[idx < kp ? idx : w0 + idx - kp];
          const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.cache) + (size_t)page * page_elems;
          __nv_bfloat16* dst = stages + (size_t)s * stage_elems + (size_t)u * (kblk + vblk);
          bulk_load(dst, base + (size_t)kvh * kblk, kblk * 2, &full_bar[s]);
          bulk_load(dst + kblk, base + (size_t)p.nkv * kblk + (size_t)kvh * vblk, vblk * 2, &full_bar[s]);
        }
      }
    }
    __syncwarp();
  } else {
    float qv[GB][DPL];
    const float* bias[GB];
    float slope[GB];
    const float q_mul = CAP ? query_scale(p, i) / p.softcap : query_scale(p, i) * LOG2E;   // q . k becomes the tanh argument / log2 units
    const float cap = p.softcap * LOG2E;
#pragma unroll
    for (int g = 0; g < GB; ++g) {
      const bool live = grp0 + g < G;
      const int h = kvh * G + (live ? grp0 + g : 0);
      const __nv_bfloat16* qp = reinterpret_cast<const __nv_bfloat16*>(p.q) + (size_t)t * p.ld_q + (size_t)h * dk;
      bias[g] = p.bias == nullptr ? nullptr : p.bias + (size_t)h * (p.far + 1);
      slope[g] = p.slope == nullptr ? 0.f : p.slope[h];
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        const int c = (v * 8 + gl) * 8;
#pragma unroll
        for (int e = 0; e < 8; ++e) qv[g][v * 8 + e] = live && c < dk ? __bfloat162float(qp[c + e]) * q_mul : 0.f;
      }
    }
    for (int it = 0; it < n_iter; ++it) {
      const int s = it % WD_NSTAGE;
      float b[WD_STAGE_PAGES][GB];
      bool ok[WD_STAGE_PAGES];
#pragma unroll
      for (int u = 0; u < WD_STAGE_PAGES; ++u) {          // the biases are fetched while the keys are still on their way
        const int idx = pb + it * WD_STAGE_PAGES + u;
        const int j = (idx < kp ? idx : w0 + idx - kp) * WD_PAGE + grp;
        ok[u] = idx < pe && j <= i && (j >= lo || j < p.keep_first);
        const int dist = max(i - j, 0);
#pragma unroll
        for (int g = 0; g < GB; ++g) b[u][g] = bias[g] != nullptr ? __ldg(bias[g] + min(dist, p.far)) : -slope[g] * (float)dist;
      }
      mbar_wait(&full_bar[s], (it / WD_NSTAGE) & 1, abort_flag, p.status, STATUS_TIMEOUT_TMA_FULL);
      const __nv_bfloat16* st = stages + (size_t)s * stage_elems;
      float sc[WD_STAGE_PAGES][GB];
#pragma unroll
      for (int u = 0; u < WD_STAGE_PAGES; ++u) {
        const __nv_bfloat16* kq = st + (size_t)u * (kblk + vblk) + grp * dk;
        float se[GB], so[GB];
#pragma unroll
        for (int g = 0; g < GB; ++g) { se[g] = 0.f; so[g] = 0.f; }
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          const int c = (v * 8 + gl) * 8;
          if (c < dk) {
            const uint4 kr = *reinterpret_cast<const uint4*>(kq + c);
            const __nv_bfloat162* kh = reinterpret_cast<const __nv_bfloat162*>(&kr);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 kf = __bfloat1622float2(kh[e]);
#pragma unroll
              for (int g = 0; g < GB; ++g) {
                se[g] = fmaf(qv[g][v * 8 + 2 * e], kf.x, se[g]);
                so[g] = fmaf(qv[g][v * 8 + 2 * e + 1], kf.y, so[g]);
              }
            }
          }
        }
#pragma unroll
        for (int g = 0; g < GB; ++g) {
          float d = se[g] + so[g];
          d += __shfl_xor_sync(0xffffffffu, d, 1);
          d += __shfl_xor_sync(0xffffffffu, d, 2);
          d += __shfl_xor_sync(0xffffffffu, d, 4);
          if constexpr (CAP) d = cap * tanh_sfu(d);
          sc[u][g] = ok[u] ? d + b[u][g] : -INFINITY;
        }
      }
#pragma unroll
      for (int g = 0; g < GB; ++g) {
        float mx = m[g];
#pragma unroll
        for (int u = 0; u < WD_STAGE_PAGES; ++u) mx = fmaxf(mx, sc[u][g]);
        const float corr = (m[g] == -INFINITY) ? 0.f : exp2f(m[g] - mx);
        m[g] = mx;
        l[g] *= corr;
#pragma unroll
        for (int c = 0; c < DPL; ++c) acc[g][c] *= corr;
      }
#pragma unroll
      for (int u = 0; u < WD_STAGE_PAGES; ++u) {
        if (!ok[u]) continue;            // never touch stage memory that holds no visible key
        const __nv_bfloat16* vq = st + (size_t)u * (kblk + vblk) + kblk + grp * dv;
        float pw[GB];
#pragma unroll
        for (int g = 0; g < GB; ++g) {
          pw[g] = exp2f(sc[u][g] - m[g]);
          l[g] += pw[g];
        }
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          const int c = (v * 8 + gl) * 8;
          if (c < dv) {
            const uint4 vr = *reinterpret_cast<const uint4*>(vq + c);
            const __nv_bfloat162* vh = reinterpret_cast<const __nv_bfloat162*>(&vr);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 vf = __bfloat1622float2(vh[e]);
#pragma unroll
              for (int g = 0; g < GB; ++g) {
                acc[g][v * 8 + 2 * e] += pw[g] * vf.x;
                acc[g][v * 8 + 2 * e + 1] += pw[g] * vf.y;
              }
            }
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty_bar[s]);
    }
  }

  // merge the 16 token groups through shared memory (the ring is free now)
  __syncthreads();
  float* sm_m = reinterpret_cast<float*>(wd_smem);           // [16][GB]
  float* sm_l = sm_m + 16 * GB;                              // [16][GB]
  float* sm_acc = sm_l + 16 * GB;                            // [16][GB][dv]
  if (warp < 4) {
    if (gl == 0) {
#pragma unroll
      for (int g = 0; g < GB; ++g) { sm_m[grp * GB + g] = m[g]; sm_l[grp * GB + g] = l[g]; }
    }
#pragma unroll
    for (int g = 0; g < GB; ++g)
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        const int c = (v * 8 + gl) * 8;
        if (c < dv) {
#pragma unroll
          for (int e = 0; e < 8; ++e) sm_acc[(grp * GB + g) * dv + c + e] = acc[g][v * 8 + e];
        }
      }
  }
  __syncthreads();
  for (int idx = tid; idx < GB * dv; idx += 160) {
    const int g = idx / dv, d = idx % dv;
    if (grp0 + g >= G) continue;
    float mx = -INFINITY;
#pragma unroll
    for (int k = 0; k < 16; ++k) mx = fmaxf(mx, sm_m[k * GB + g]);
    float num = 0.f, den = 0.f;
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float mk = sm_m[k * GB + g];
      const float w = (mk == -INFINITY) ? 0.f : exp2f(mk - mx);
      num += w * sm_acc[(k * GB + g) * dv + d];
      den += w * sm_l[k * GB + g];
    }
    const int h = kvh * G + grp0 + g;
    if (p.n_split == 1) {
      reinterpret_cast<__nv_bfloat16*>(p.out)[(size_t)t * p.ld_out + (size_t)h * dv + d] =
          __float2bfloat16_rn(num * finish_scale(p, t, h, mx, den) * element_gate(p, t, h, d));
    } else {
      float* w = p.ws + (((size_t)t * p.nq + h) * p.n_split + split) * (dv + 2);
      w[d] = num;
      if (d == 0) { w[dv] = mx; w[dv + 1] = den; }
    }
  }
}

// Key splits (up to 64) of a head together, each against the common maximum: one warp weighs the splits, then a dim per thread.
__global__ void __launch_bounds__(128) window_decode_merge_kernel(const WindowAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float s_w[64];
  const int t = blockIdx.x / p.nq, h = blockIdx.x % p.nq, stride = p.dv + 2;
  const float* w = p.ws + (size_t)blockIdx.x * p.n_split * stride;
  if (threadIdx.x < 32) {                        // two splits per lane
    float m[2], e[2], mx = -INFINITY, den = 0.f;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int s = threadIdx.x + 32 * u;
      m[u] = s < p.n_split ? w[s * stride + p.dv] : -INFINITY;
      e[u] = s < p.n_split ? w[s * stride + p.dv + 1] : 0.f;
      mx = fmaxf(mx, m[u]);
    }
    mx = warp_max(mx);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const float f = m[u] == -INFINITY ? 0.f : exp2f(m[u] - mx);
      den += f * e[u];
      e[u] = f;
    }
    const float f = finish_scale(p, t, h, mx, warp_sum(den));
    s_w[threadIdx.x] = e[0] * f;
    s_w[threadIdx.x + 32] = e[1] * f;
  }
  __syncthreads();
  for (int d = threadIdx.x; d < p.dv; d += blockDim.x) {
    float num = 0.f;
#pragma unroll 8
    for (int s = 0; s < p.n_split; ++s) num = fmaf(s_w[s], w[s * stride + d], num);      // an empty split holds zeros
    reinterpret_cast<__nv_bfloat16*>(p.out)[(size_t)t * p.ld_out + (size_t)h * p.dv + d] = __float2bfloat16_rn(num * element_gate(p, t, h, d));
  }
}

// ---------------------------------------------------------------------------------------------
// Portion kernel on the tensor cores (bf16, pages of 16): one CTA = a tile of up to 128 consecutive queries of one row
// and one query head, walking the blocks of 64 keys that any of its queries sees (kept part, then window).  Same
// structure as prefill_attn_kernel - S = Q K^T and O += P V by tcgen05 with S and O in tensor memory, two softmax
// threads per query, lazily refreshed maximum, two-stage TMA ring - with K / V fetched page by page from the cache
// (four 16-row boxes per 64-key block form one swizzled tile; dims past dk / dv and pages past the last key read as
// zeros) and with the distance bias added to the scores in registers.
// Warp roles (320 threads): warp 0 TMA, warp 1 tensor memory + MMA, warps 2..9 softmax / epilogue.
// ---------------------------------------------------------------------------------------------
struct WindowTiles {
  const int* q0;              // [n_tiles] first packed query
  const int* qn;              // [n_tiles] queries (<= 128)
  int n_pages;                // pages of the pool (an index past it reads zeros)
  long long kv_ld;            // 0: paged cache; else the keys and values are rows [nkv * dk | nkv * dv] of this pitch, one per
                              // token, and a page is 16 consecutive rows
  const int* pool_base;       // [n_tiles] first page (16 rows) of the tile's row in the matrix of pooled blocks
  int n_pool_pages;
};

// TIED: a stage holds keys only (and their factors, 64 floats behind all stages), which the second product reads too
template <int HK, int HV, bool TIED = false>
struct WpCfg {
  static constexpr int BK = 64;
  static constexpr int QTILE = 128 * 64 * 2, KTILE = BK * 64 * 2;
  static constexpr int Q_BYTES = HK * QTILE, K_BYTES = HK * KTILE, V_BYTES = HV * KTILE;
  static constexpr int P_BYTES = 128 * BK * 2;
  static constexpr int STAGE_BYTES = TIED ? K_BYTES : K_BYTES + V_BYTES;
  static constexpr int NSTAGE = TIED ? 3 : 2;
  static constexpr int FACTOR_BYTES = TIED ? NSTAGE * BK * 4 : 0;
  static constexpr int SMEM_BYTES = Q_BYTES + P_BYTES + NSTAGE * STAGE_BYTES + FACTOR_BYTES + 128;
  static constexpr int XCOL = 64;                            // exchange columns between the two halves of a query
  static constexpr int TMEM_COLS = HV <= 2 ? 256 : 512;      // S at 0, O at 128
  static constexpr int MIN_CTAS = HK + HV <= 4 ? 2 : 1;
};
constexpr int WP_THREADS = 320;

// cap * tanh(mul * v) of 32 scores of a thread.  The arguments of trained attention mostly lie well inside (-1, 1), where
// x P(x^2) with a degree-5 minimax P (fitted for the absolute error, 3.3e-7 in fp32) needs no special-function unit, the
// busiest pipe of this kernel; a warp in which some argument is larger takes the exponential form for all of them.
__device__ __forceinline__ uint64_t pack_f32x2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul_f32x2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ void soft_cap32(float* v, float mul, float cap) {
  float big = fabsf(v[0]);
#pragma unroll
  for (int c = 1; c < 32; ++c) big = fmaxf(big, fabsf(v[c]));
  if (__all_sync(0xffffffffu, big * mul <= 1.0f)) {
    constexpr float A[6] = {0.999996854f, -0.333240038f, 0.132535252f, -0.0509728608f, 0.016114178f, -0.00283946425f};
    uint64_t a[6];
#pragma unroll
    for (int k = 0; k < 6; ++k) a[k] = pack_f32x2(A[k] * cap, A[k] * cap);
    const uint64_t m = pack_f32x2(mul, mul);
#pragma unroll
    for (int c = 0; c < 32; c += 2) {
      const uint64_t x = mul_f32x2(pack_f32x2(v[c], v[c + 1]), m), u = mul_f32x2(x, x);
      uint64_t y = a[5];
#pragma unroll
      for (int k = 4; k >= 0; --k) y = fma_f32x2(y, u, a[k]);
      y = mul_f32x2(y, x);
      asm("mov.b64 {%0, %1}, %2;" : "=f"(v[c]), "=f"(v[c + 1]) : "l"(y));
    }
  } else {
#pragma unroll
    for (int c = 0; c < 32; ++c) v[c] = cap * tanh_sfu(v[c] * mul);
  }
}

// TIED: tm_v describes the matrix of pooled blocks (or is unused), whose blocks come first
template <int HK, int HV, bool CAP, bool TIED>
__global__ void __launch_bounds__(WP_THREADS, WpCfg<HK, HV, TIED>::MIN_CTAS)
window_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                      const __grid_constant__ CUtensorMap tm_v, const WindowAttnParams p, const WindowTiles tl) {
  using C = WpCfg<HK, HV, TIED>;
  constexpr int BK = C::BK;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* q_s = smem;
  uint8_t* p_s = q_s + C::Q_BYTES;
  uint8_t* kv_s = p_s + C::P_BYTES;
  float* factor_s = reinterpret_cast<float*>(kv_s + C::NSTAGE * C::STAGE_BYTES);      // [NSTAGE][BK], tied
  uint64_t* bars = reinterpret_cast<uint64_t*>(kv_s + C::NSTAGE * C::STAGE_BYTES + C::FACTOR_BYTES);
  uint64_t* q_full = bars;
  uint64_t* kv_full = bars + 1;
  uint64_t* kv_empty = kv_full + C::NSTAGE;
  uint64_t* s_full = kv_empty + C::NSTAGE;
  uint64_t* p_ready = s_full + 1;
  uint64_t* pv_done = p_ready + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile = blockIdx.x, head = blockIdx.y;
  const int kvh = head / (p.nq / p.nkv);
  if ((smem_u32(smem) & 1023u) != 0) {          // the swizzled tiles need a 1024-byte aligned base
    if (threadIdx.x == 0) atomicCAS(p.status, 0, STATUS_BAD_INDEX);
    return;
  }
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < C::NSTAGE; ++s) { mbar_init(&kv_full[s], 1); mbar_init(&kv_empty[s], 1); }
    mbar_init(s_full, 1);
    mbar_init(p_ready, 256);
    mbar_init(pv_done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, C::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_s = tmem_base, tmem_o = tmem_base + 128;

  const int q0 = tl.q0[tile], qn = tl.qn[tile];
  const int i0 = p.pos[q0], i_last = i0 + qn - 1;             // the tile's positions are consecutive
  int keep_end, lo0;
  visible_range(i0, p.window, p.keep_first, keep_end, lo0);
  const bool pooled = TIED && p.pooled != nullptr;
  const int kb = ((pooled ? visible_blocks(i_last, p.window, p.pool) : keep_end) + BK - 1) / BK;   // blocks of the kept or pooled part
  const int w0 = pooled ? lo0 / BK : max(lo0 / BK, kb);       // first block of the window part
  const int total_blocks = kb + max(0, i_last / BK - w0 + 1);

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      mbar_expect_tx(q_full, C::Q_BYTES);
#pragma unroll
      for (int h = 0; h < HK; ++h) tma_load_2d(q_s + h * C::QTILE, &tm_q, head * p.dk + h * 64, q0, q_full);
      const int* pt = p.page_table + (size_t)p.row[q0] * p.max_pages;
      const int last_page = i_last / WD_PAGE, pool0 = pooled ? tl.pool_base[tile] : 0;
      for (int n = 0; n < total_blocks; ++n) {
        const int st = n % C::NSTAGE;
        const int b = n < kb ? n : w0 + n - kb;
        const bool means = pooled && n < kb;
        int page[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) page[u] = means ? min(pool0 + b * 4 + u, tl.n_pool_pages) : b * 4 + u <= last_page ? pt[b * 4 + u] : tl.n_pages;
        mbar_wait(&kv_empty[st], ((n / C::NSTAGE) & 1) ^ 1, abort_flag, p.status, STATUS_TIMEOUT_STAGE_EMPTY);
        if (*abort_flag) break;
        const bool factors = TIED && p.factor != nullptr && !means;
        mbar_expect_tx(&kv_full[st], C::STAGE_BYTES + (factors ? BK * 4 : 0));
        uint8_t* ks = kv_s + st * C::STAGE_BYTES;
        uint8_t* vs = ks + C::K_BYTES;
        if constexpr (TIED) {
          if (factors) {
#pragma unroll
            for (int u = 0; u < 4; ++u)                       // a page past the last key: any finite numbers
              bulk_load(factor_s + st * BK + u * WD_PAGE, p.factor + (size_t)min(page[u], tl.n_pages - 1) * WD_PAGE, WD_PAGE * 4, &kv_full[st]);
          }
#pragma unroll
          for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int h = 0; h < HK; ++h) tma_load_4d(ks + h * C::KTILE + u * 2048, means ? &tm_v : &tm_k, h * 64, 0, kvh, page[u], &kv_full[st]);
          continue;
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
#pragma unroll
          for (int h = 0; h < HK; ++h) tma_load_4d(ks + h * C::KTILE + u * 2048, &tm_k, h * 64, 0, kvh, page[u], &kv_full[st]);
#pragma unroll
          for (int h = 0; h < HV; ++h) tma_load_4d(vs + h * C::KTILE + u * 2048, &tm_v, h * 64, 0, kvh, page[u], &kv_full[st]);
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(128, BK);
      constexpr uint32_t idesc_o = umma_idesc_bf16_bmn(128, HV * 64);
      mbar_wait(q_full, 0, abort_flag, p.status, STATUS_TIMEOUT_TMA_FULL);
      const uint32_t q_addr = smem_u32(q_s), p_addr = smem_u32(p_s);
      for (int n = 0; n < total_blocks; ++n) {
        const int st = n % C::NSTAGE;
        mbar_wait(&kv_full[st], (n / C::NSTAGE) & 1, abort_flag, p.status, STATUS_TIMEOUT_TMA_FULL);
        tc_fence_after();
        const uint32_t k_addr = smem_u32(kv_s + st * C::STAGE_BYTES);
        const uint32_t v_addr = TIED ? k_addr : k_addr + C::K_BYTES;
#pragma unroll
        for (int ks = 0; ks < HK * 4; ++ks) {
          const uint32_t qo = (ks / 4) * C::QTILE + (ks % 4) * 32;
          const uint32_t ko = (ks / 4) * C::KTILE + (ks % 4) * 32;
          umma_bf16(tmem_s, umma_desc_sw128(q_addr + qo), umma_desc_sw128(k_addr + ko), idesc_s, ks > 0 ? 1u : 0u);
        }
        umma_commit(s_full);
        mbar_wait(p_ready, n & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
        tc_fence_after();
#pragma unroll
        for (int ks = 0; ks < BK / 16; ++ks)
          umma_bf16(tmem_o, umma_desc_sw128(p_addr + ks * 32), umma_desc_mn_sw128(v_addr + ks * 2048, C::KTILE), idesc_o,
                    (n > 0 || ks > 0) ? 1u : 0u);
        umma_commit(&kv_empty[st]);
        umma_commit(pv_done);
      }
    }
    __syncwarp();
  } else {
    // ---------------- softmax / epilogue: two threads per query, 32 key columns each ----------------
    const int qd = warp & 3, half = (warp - 2) >> 2;
    const int row = qd * 32 + lane;
    const bool row_ok = row < qn;
    const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
    const int i = i0 + row;
    const float sc = CAP ? 1.0f : query_scale(p, i) * LOG2E;
    const float cap_mul = CAP ? query_scale(p, i) / p.softcap : 0.f, cap = p.softcap * LOG2E;
    const int iw0 = i0 + qd * 32, iw1 = iw0 + 31;             // positions of the warp's first and last query
    const int lo = p.window > i ? 0 : i - p.window + 1;
    const int lo_w1 = p.window > iw1 ? 0 : iw1 - p.window + 1;
    const float* bias = p.bias == nullptr ? nullptr : p.bias + (size_t)head * (p.far + 1);
    const float far_bias = bias == nullptr ? 0.f : bias[p.far];
    const float slope = p.slope == nullptr ? 0.f : p.slope[head];
    const int blocks = pooled ? visible_blocks(i, p.window, p.pool) : 0;
    float m_ref = -INFINITY, l = 0.f;
    for (int n = 0; n < total_blocks; ++n) {
      const int j0 = (n < kb ? n : w0 + n - kb) * BK + half * 32;        // first key column of this thread
      mbar_wait(s_full, n & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
      tc_fence_after();
      float sv[32];
      tmem_ld32(tmem_s + lane_off + half * 32, sv);
      tmem_ld_wait();
      const int dmin = iw0 - (j0 + 31), dmax = iw1 - j0;                 // distances inside the warp's 32 x 32 patch
      const bool means = pooled && n < kb;
      if constexpr (CAP) soft_cap32(sv, cap_mul, cap);
      if constexpr (TIED) {
        if (p.factor != nullptr && !means) {
          const int st = n % C::NSTAGE;
          mbar_wait(&kv_full[st], (n / C::NSTAGE) & 1, abort_flag, p.status, STATUS_TIMEOUT_TMA_FULL);
          const float4* f4 = reinterpret_cast<const float4*>(factor_s + st * BK + half * 32);
#pragma unroll
          for (int c = 0; c < 8; ++c) {
            const float4 f = f4[c];
            sv[4 * c] *= f.x; sv[4 * c + 1] *= f.y; sv[4 * c + 2] *= f.z; sv[4 * c + 3] *= f.w;
          }
        }
      }
      if (p.slope != nullptr) {
        const float d0 = -slope * (float)(i - j0);
#pragma unroll
        for (int c = 0; c < 32; ++c) sv[c] = fmaf(sv[c], sc, fmaf(slope, (float)c, d0));
      } else if (CAP && bias == nullptr) {
      } else if (bias == nullptr || dmin >= p.far) {
#pragma unroll
        for (int c = 0; c < 32; ++c) sv[c] = fmaf(sv[c], sc, far_bias);
      } else if (dmin >= 0 && dmax <= p.far) {
        const float* b = bias + (i - j0);
#pragma unroll
        for (int c = 0; c < 32; ++c) sv[c] = fmaf(sv[c], sc, __ldg(b - c));
      } else {
#pragma unroll
        for (int c = 0; c < 32; ++c) sv[c] = fmaf(sv[c], sc, __ldg(bias + min(max(i - j0 - c, 0), p.far)));
      }
      if (means) {
#pragma unroll
        for (int c = 0; c < 32; ++c)
          if (j0 + c >= blocks) sv[c] = -INFINITY;
      } else if (!(dmin >= 0 && (j0 >= lo_w1 || j0 + 31 < p.keep_first))) {
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          const int j = j0 + c;
          if (j > i || (j < lo && j >= p.keep_first)) sv[c] = -INFINITY;
        }
      }
      float mx = sv[0];
#pragma unroll
      for (int c = 1; c < 32; ++c) mx = fmaxf(mx, sv[c]);
      const uint32_t xcol = tmem_base + lane_off + C::XCOL + (n & 1) * 2;
      tmem_st1(xcol + half, mx);
      tmem_st_wait();
      tc_fence_before();
      named_bar_sync(1, 256);
      tc_fence_after();
      mx = fmaxf(mx, tmem_ld1(xcol + (half ^ 1)));
      const bool grow = mx > m_ref + 8.0f;
      const float m_new = grow ? mx : m_ref;
      const float f = (grow && m_ref != -INFINITY) ? exp2f(m_ref - m_new) : 1.0f;
      if (n > 0) mbar_wait(pv_done, (n - 1) & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
      tc_fence_after();
      if (n > 0 && __any_sync(0xffffffffu, f != 1.0f)) {
#pragma unroll 1
        for (int c = 0; c < HV * 32; c += 32) {
          float o[32];
          tmem_ld32(tmem_o + lane_off + half * (HV * 32) + c, o);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; ++e) o[e] *= f;
          tmem_st32(tmem_o + lane_off + half * (HV * 32) + c, o);
        }
        tmem_st_wait();
      }
      l *= f;
      m_ref = m_new;
      const float neg_m = (m_ref == -INFINITY) ? 0.f : -m_ref;
      float ps0 = 0.f, ps1 = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint4 pk;
        __nv_bfloat162* p2 = reinterpret_cast<__nv_bfloat162*>(&pk);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float a = ex2_approx(sv[c * 8 + 2 * e] + neg_m);
          const float b = ex2_approx(sv[c * 8 + 2 * e + 1] + neg_m);
          p2[e] = __floats2bfloat162_rn(a, b);
          ps0 += a;
          ps1 += b;
        }
        *reinterpret_cast<uint4*>(p_s + row * 128 + (((half * 4 + c) ^ (row & 7)) << 4)) = pk;
      }
      l += ps0 + ps1;
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(p_ready);
    }
    if (total_blocks > 0) mbar_wait(pv_done, (total_blocks - 1) & 1, abort_flag, p.status, STATUS_TIMEOUT_ACCUM);
    tc_fence_after();
    {
      const uint32_t xcol = tmem_base + lane_off + C::XCOL;
      named_bar_sync(1, 256);
      tmem_st1(xcol + half, l);
      tmem_st_wait();
      tc_fence_before();
      named_bar_sync(1, 256);
      tc_fence_after();
      l += tmem_ld1(xcol + (half ^ 1));
    }
    const float inv = row_ok ? finish_scale(p, q0 + row, head, m_ref, l) : 0.f;
    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(q0 + row) * p.ld_out + (size_t)head * p.dv;
#pragma unroll 1
    for (int c = half * (HV * 32); c < (half + 1) * (HV * 32); c += 32) {
      float o[32];
      tmem_ld32(tmem_o + lane_off + c, o);
      tmem_ld_wait();
      if (row_ok) {
#pragma unroll
        for (int v = 0; v < 4; ++v) {
          if (c + v * 8 < p.dv) {
            uint4 pk;
            __nv_bfloat162* p2 = reinterpret_cast<__nv_bfloat162*>(&pk);
            if (p.wide_gate != nullptr) {
              float z[8];
              load8(reinterpret_cast<const __nv_bfloat16*>(p.wide_gate) + (size_t)(q0 + row) * p.ld_gate + (size_t)head * p.dv + c + v * 8, z);
#pragma unroll
              for (int e = 0; e < 8; ++e) o[v * 8 + e] = __fdividef(o[v * 8 + e], 1.0f + __expf(-z[e]));
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) p2[e] = __floats2bfloat162_rn(o[v * 8 + 2 * e] * inv, o[v * 8 + 2 * e + 1] * inv);
            *reinterpret_cast<uint4*>(dst + c + v * 8) = pk;
          }
        }
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, C::TMEM_COLS);
  }
}

cudaError_t launch_window_merge(const WindowAttnParams& p, cudaStream_t stream) {
  return launch_chain(window_decode_merge_kernel, dim3(p.n * p.nq), dim3(128), 0, stream, p);
}

template <int VEC, int GB, bool EXACT, bool CAP>
static int launch_window_decode_as(const WindowAttnParams& p, cudaStream_t stream) {
  const int groups = (p.nq / p.nkv + GB - 1) / GB;
  const size_t ring = (size_t)WD_NSTAGE * WD_STAGE_PAGES * WD_PAGE * (p.dk + p.dv) * 2 + 128;
  const size_t merge = (size_t)16 * GB * (p.dv + 2) * 4;
  const size_t smem = ring > merge ? ring : merge;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(window_decode_kernel<VEC, GB, EXACT, CAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess)
      return -10;
    configured = true;
  }
  if (smem > 160 * 1024) return -11;
  cudaError_t e = launch_chain(window_decode_kernel<VEC, GB, EXACT, CAP>, dim3(p.nkv * groups, p.n, p.n_split), dim3(160), smem, stream, p);
  if (e == cudaSuccess && p.n_split > 1) e = launch_window_merge(p, stream);
  return e == cudaSuccess ? 0 : -3;
}

template <int VEC, int GB>
static int launch_window_decode(const WindowAttnParams& p, cudaStream_t stream) {
  const bool exact = p.dk == VEC * 64 && p.dv == VEC * 64;
  if (p.softcap > 0.f)
    return exact ? launch_window_decode_as<VEC, GB, true, true>(p, stream) : launch_window_decode_as<VEC, GB, false, true>(p, stream);
  return exact ? launch_window_decode_as<VEC, GB, true, false>(p, stream) : launch_window_decode_as<VEC, GB, false, false>(p, stream);
}

template <int HK, int HV, bool CAP, bool TIED = false>
static int launch_window_prefill_as(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv,
                                 const WindowAttnParams& p, const WindowTiles& tl, int n_tiles, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(window_prefill_kernel<HK, HV, CAP, TIED>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             WpCfg<HK, HV, TIED>::SMEM_BYTES) != cudaSuccess)
      return -10;
    configured = true;
  }
  window_prefill_kernel<HK, HV, CAP, TIED><<<dim3(n_tiles, p.nq), WP_THREADS, WpCfg<HK, HV, TIED>::SMEM_BYTES, stream>>>(mq, mk, mv, p, tl);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <int HK, int HV>
static int launch_window_prefill(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv,
                                 const WindowAttnParams& p, const WindowTiles& tl, int n_tiles, cudaStream_t stream) {
  if constexpr (HK == HV) {
    if (p.tied) return launch_window_prefill_as<HK, HV, false, true>(mq, mk, mv, p, tl, n_tiles, stream);
  }
  return p.softcap > 0.f ? launch_window_prefill_as<HK, HV, true>(mq, mk, mv, p, tl, n_tiles, stream)
                         : launch_window_prefill_as<HK, HV, false>(mq, mk, mv, p, tl, n_tiles, stream);
}

// queries as a [n, cols] matrix of row pitch ld, read in boxes of 128 tokens x 64 columns
static int make_query_map(CUtensorMap* m, const void* base, int n, long long cols, long long ld) {
  PfEncodeFn fn = pf_encode_fn();
  if (fn == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || ld % 8) return -2;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)n};
  cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
  cuuint32_t box[2] = {64u, 128u}, estr[2] = {1u, 1u};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -3;
}

int check_window_attn(const WindowAttnParams* p) {
  // tied layers: one size; pooled blocks are a tied layer's, in the place of kept tokens, and have no position
  if (p->tied && (p->tied != 1 || p->dk != p->dv || p->softcap != 0.f)) return -2;
  if (!p->tied && (p->factor != nullptr || p->pooled != nullptr)) return -2;
  if (p->pooled != nullptr && (p->pool < 1 || p->pool_rows < 1 || p->pool_rows > p->page_size || (p->pool_rows & (p->pool_rows - 1)) ||
                               (long long)p->pool_rows * p->pool < p->page_size || p->keep_first != 0 || p->factor != nullptr || p->slope != nullptr || p->bias != nullptr))
    return -2;
  if (p->slope != nullptr && p->bias != nullptr) return -2;
  if (p->gate != nullptr && p->wide_gate != nullptr) return -2;
  return p->nkv <= 0 || p->nq % p->nkv || p->dk > 256 || p->dv > 256 || p->dk % 8 || p->dv % 8 || p->window < 1 || p->far < 0 ||
         p->keep_first < 0 || p->ld_q < (long long)p->nq * p->dk || p->softcap < 0.f ||
         (p->temp_coef != 0.f && !(p->temp_every > 0.0)) ? -2 : 0;
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

// Host-side description of one launch (same fields as QkvPostParams).
extern "C" int tahb_qkv_post(const QkvPostParams* q, int f32, cudaStream_t stream) {
  const QkvPostParams& p = *q;
  if (p.M <= 0) return 0;
  if (p.dk > 256 || p.dv > 256 || p.dk % 8 || p.dv % 8 || p.dim > p.dk) return -2;
  if (p.rope != nullptr && (p.rot % 2 || p.rot < 2 || p.rot > p.dim)) return -2;
  if (p.v_first != nullptr && p.lambda == nullptr) return -2;
  const long long warps = (long long)p.M * (p.nq + 2 * p.nkv);
  const dim3 grid((unsigned)((warps + 3) / 4));
  cudaError_t e = f32 ? launch_chain(qkv_post_kernel<float>, grid, dim3(128), 0, stream, p)
                      : launch_chain(qkv_post_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p);
  return e == cudaSuccess ? 0 : -3;
}

// Host-side description of one attention launch (same fields as WindowAttnParams).
extern "C" int tahb_window_attn_plain(const WindowAttnParams* p, int f32, cudaStream_t stream) {
  if (p->n <= 0) return 0;
  if (check_window_attn(p)) return -2;
  const long long warps = (long long)p->n * p->nq;
  const dim3 grid((unsigned)((warps + 3) / 4));
  cudaError_t e = f32 ? launch_chain(window_attn_plain_kernel<float>, grid, dim3(128), 0, stream, *p)
                      : launch_chain(window_attn_plain_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}

// One query per entry (decode).  bias and sink in log2 units; ws: n * nq * n_split * (dv + 2) floats when n_split > 1.
extern "C" int tahb_window_attn_decode(const WindowAttnParams* p, cudaStream_t stream) {
  if (p->n <= 0) return 0;
  if (check_window_attn(p) || p->n > 65535 || p->n_split < 1 || p->n_split > 64) return -2;
  if (p->page_size != WD_PAGE) return -5;
  if (p->n_split > 1 && p->ws == nullptr) return -4;
  if (p->tied) return launch_tied_decode(*p, stream);
  const int d = p->dk > p->dv ? p->dk : p->dv, vec = d <= 64 ? 1 : d <= 128 ? 2 : 4;
  const int G = p->nq / p->nkv, gb = G == 1 ? 1 : (G == 2 || vec == 4) ? 2 : 4;
#define TAHB_WD(V_, G_) if (vec == V_ && gb == G_) return launch_window_decode<V_, G_>(*p, stream);
  TAHB_WD(1, 1) TAHB_WD(1, 2) TAHB_WD(1, 4)
  TAHB_WD(2, 1) TAHB_WD(2, 2) TAHB_WD(2, 4)
  TAHB_WD(4, 1) TAHB_WD(4, 2)
#undef TAHB_WD
  return -2;
}

// Query tiles of portions; n_pages = pages of the layer's pool; kv_ld: see WindowTiles.  bias and sink in log2 units.
// Tied layers with pooled blocks: p->pooled is a matrix [16 * n_pool_pages, nkv * dk] whose page pool_base[tile] is the first of the
// tile's row.
extern "C" int tahb_window_attn_tiles(const WindowAttnParams* p, const int* q0, const int* qn, int n_tiles, int n_pages,
                                      long long kv_ld, const int* pool_base, int n_pool_pages, cudaStream_t stream) {
  if (p->n <= 0 || n_tiles <= 0) return 0;
  if (check_window_attn(p) || p->ld_out % 8 || (p->wide_gate != nullptr && (p->ld_gate % 8 || (reinterpret_cast<uintptr_t>(p->wide_gate) & 15))))
    return -2;
  if (kv_ld != 0 && kv_ld < (long long)p->nkv * (p->dk + p->dv)) return -2;
  if (p->tied && (kv_ld != 0 || n_pages < 1 || (p->pooled != nullptr && pool_base == nullptr))) return -2;
  if (p->page_size != WD_PAGE) return -5;
  const size_t page_elems = (size_t)p->nkv * WD_PAGE * (p->dk + (p->tied ? 0 : p->dv));
  CUtensorMap mq, mk, mv;
  int rc;
  if ((rc = make_query_map(&mq, p->q, p->n, (long long)p->nq * p->dk, p->ld_q))) return rc;
  auto kv = reinterpret_cast<const __nv_bfloat16*>(p->cache);
  if (kv_ld) {
    if ((rc = make_page_map(&mk, kv, p->dk, p->nkv, n_pages, kv_ld, p->dk, WD_PAGE * kv_ld))) return rc;
    if ((rc = make_page_map(&mv, kv + (size_t)p->nkv * p->dk, p->dv, p->nkv, n_pages, kv_ld, p->dv, WD_PAGE * kv_ld))) return rc;
  } else {
    if ((rc = make_page_map(&mk, kv, p->dk, p->nkv, n_pages, p->dk, (size_t)WD_PAGE * p->dk, page_elems))) return rc;
    mv = mk;
    const long long pool_ld = (long long)p->nkv * p->dk;
    if (p->pooled != nullptr && n_pool_pages > 0 &&
        (rc = make_page_map(&mv, p->pooled, p->dk, p->nkv, n_pool_pages, pool_ld, p->dk, WD_PAGE * pool_ld)))
      return rc;
    if (!p->tied && (rc = make_page_map(&mv, kv + (size_t)p->nkv * WD_PAGE * p->dk, p->dv, p->nkv, n_pages, p->dv, (size_t)WD_PAGE * p->dv,
                            page_elems))) return rc;
  }
  WindowTiles tl{q0, qn, n_pages, kv_ld, pool_base, n_pool_pages};
  const int hk = p->dk <= 64 ? 1 : p->dk <= 128 ? 2 : 4, hv = p->dv <= 64 ? 1 : p->dv <= 128 ? 2 : 4;
  if (p->softcap == 0.f && p->dk > 128 && p->dk <= 192 && p->dv <= 128)
    return p->dv <= 64 ? launch_window_prefill_as<3, 1, false>(mq, mk, mv, *p, tl, n_tiles, stream)
                       : launch_window_prefill_as<3, 2, false>(mq, mk, mv, *p, tl, n_tiles, stream);
  if (hk == 4 || hv == 4) return launch_window_prefill<4, 4>(mq, mk, mv, *p, tl, n_tiles, stream);
  if (hk == 2) return hv == 2 ? launch_window_prefill<2, 2>(mq, mk, mv, *p, tl, n_tiles, stream)
                              : launch_window_prefill<2, 1>(mq, mk, mv, *p, tl, n_tiles, stream);
  return hv == 2 ? launch_window_prefill<1, 2>(mq, mk, mv, *p, tl, n_tiles, stream)
                 : launch_window_prefill<1, 1>(mq, mk, mv, *p, tl, n_tiles, stream);
}
