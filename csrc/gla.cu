// Gated linear attention: a matrix memory with a decay per key channel.  Per head, with log decays a_t [dk] <= 0:
//
//   a_t = logsigmoid(z_t) / tau,   z_t = W2 low_t + b           (low_t: a few fp32 features of the token)
//   S_t = diag(exp(a_t)) S_{t-1} + k_t v_t^T       [dk, dv]
//   o_t = S_t^T (q_scale q_t)
//   y_t = rms(o_t) * w * silu(g_t)                 (w shared by the heads)
//
// S lives in fp32, one slot per cache row: state[slot][head] = S [dk][dv].  A token at position 0 starts from zero, so a slot
// needs no clearing when it changes hands.  dk and dv are padded to multiples of 8 with zeros.
#include "chunk_common.cuh"

namespace tahb {

struct GlaParams {
  const void* qkvg;           // [n, ld]: heads * dk of q, heads * dk of k, heads * dv of v, heads * dv of g
  const float* low;           // [n, rank]
  const void* w2;             // [heads * dk, rank] in the activation type
  const float* b2;            // [heads * dk]
  const float* norm_w;        // [dv]
  void* out;                  // [n, ld_out], head h at column h * dv
  float* S;                   // [slots, heads, dk, dv]
  const int* seq_start;       // [n_seq] first packed token of each sequence, null = sequence s is token s
  const int* seq_len;         // [n_seq] tokens of each sequence, null = 1
  const int* pos;             // [n] position of each packed token
  const int* row;             // [n] state slot of each packed token
  const int* slot;            // [n] KV slot; negative = the row is idle and its state stays (may be null)
  int n_seq, heads, dk, dv, vdim, rank;       // vdim: real size; rank: a multiple of 4
  long long ld, ld_out;
  float inv_tau, eps, q_scale;
};

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// ---------------------------------------------------------------------------------------------
// Recurrent form: grid (heads, n_seq), 256 threads; the tokens of a sequence one after another.  Thread (rg, c) owns the
// float4 column c of the rows rg, rg + nrg, ... of S, read and written in place (one token: the state streams through
// once, which is the whole cost of a decode step).
// ---------------------------------------------------------------------------------------------
constexpr int GR_THREADS = 256;
constexpr int GR_MAX_D = 1024;

template <typename T>
__global__ void __launch_bounds__(GR_THREADS, 3) gla_recurrent_kernel(const GlaParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x, s = blockIdx.y;
  const int dk = p.dk, dv = p.dv, ncol = dv / 4, nrg = GR_THREADS / ncol;
  float* s_q = sm;                       // [dk]
  float* s_k = s_q + dk;                 // [dk]
  float* s_a = s_k + dk;                 // [dk] decay
  float* s_red = s_a + dk;               // [nrg][dv]
  float* s_w = s_red + (size_t)nrg * dv; // [8] warp partials
  const int t0 = p.seq_start ? p.seq_start[s] : s, len = p.seq_len ? p.seq_len[s] : 1;
  if (len <= 0) return;
  if (p.slot != nullptr && p.slot[t0] < 0) {     // idle row: leave the state alone
    T* o = reinterpret_cast<T*>(p.out) + (size_t)t0 * p.ld_out + (size_t)h * dv;
    for (int d = tid; d < dv; d += GR_THREADS) stf(o + d, 0.f);
    return;
  }
  float* S = p.S + ((size_t)p.row[t0] * p.heads + h) * dk * dv;
  bool fresh = p.pos[t0] == 0;
  const int rg = tid / ncol, c = tid % ncol;
  for (int t = t0; t < t0 + len; ++t) {
    const T* base = reinterpret_cast<const T*>(p.qkvg) + (size_t)t * p.ld;
    const T* q = base + (size_t)h * dk;
    const T* k = base + (size_t)(p.heads + h) * dk;
    const T* v = base + (size_t)2 * p.heads * dk + (size_t)h * dv;
    const T* g = base + (size_t)2 * p.heads * dk + (size_t)(p.heads + h) * dv;
    __syncthreads();                     // the previous token's s_q / s_k / s_a / s_red have been read
    for (int d = tid; d < dk; d += GR_THREADS) {
      const T* w2 = reinterpret_cast<const T*>(p.w2) + ((size_t)h * dk + d) * p.rank;
      const float* low = p.low + (size_t)t * p.rank;
      float z = 0.f;
      for (int r = 0; r < p.rank; r += 4) {
        const float4 a = ldf4(w2 + r), b = ldf4(low + r);
        z += a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w;
      }
      s_a[d] = expf(log_sigmoid(z + p.b2[(size_t)h * dk + d]) * p.inv_tau);
      s_q[d] = ldf(q + d) * p.q_scale;
      s_k[d] = ldf(k + d);
    }
    __syncthreads();
    if (rg < nrg) {
      const float4 vv = ldf4(v + c * 4);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      constexpr int U = 8;               // rows in flight: all their loads are issued before the first store
      for (int r0 = rg; r0 < dk; r0 += U * nrg) {
        float4 a[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = r0 + u * nrg;
          a[u] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (!fresh && r < dk) a[u] = *(reinterpret_cast<const float4*>(S + (size_t)r * dv) + c);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = r0 + u * nrg;
          if (r < dk) {
            const float kr = s_k[r], qr = s_q[r], ar = s_a[r];
            a[u].x = fmaf(ar, a[u].x, kr * vv.x); a[u].y = fmaf(ar, a[u].y, kr * vv.y);
            a[u].z = fmaf(ar, a[u].z, kr * vv.z); a[u].w = fmaf(ar, a[u].w, kr * vv.w);
            o.x = fmaf(a[u].x, qr, o.x); o.y = fmaf(a[u].y, qr, o.y); o.z = fmaf(a[u].z, qr, o.z); o.w = fmaf(a[u].w, qr, o.w);
            *(reinterpret_cast<float4*>(S + (size_t)r * dv) + c) = a[u];
          }
        }
      }
      *reinterpret_cast<float4*>(s_red + (size_t)rg * dv + c * 4) = o;
    }
    fresh = false;
    __syncthreads();
    float ss = 0.f;
    for (int d = tid; d < dv; d += GR_THREADS) {
      float o = 0.f;
      for (int r = 0; r < nrg; ++r) o += s_red[(size_t)r * dv + d];
      s_red[d] = o;                      // row 0 is rewritten by the thread that read this column of every row
      ss = fmaf(o, o, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) s_w[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < GR_THREADS / 32; ++w) ss += s_w[w];
    const float r = 1.0f / sqrtf(ss / (float)p.vdim + p.eps);
    T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + (size_t)h * dv;
    for (int d = tid; d < dv; d += GR_THREADS) {
      const float z = ldf(g + d);
      stf(out + d, s_red[d] * r * p.norm_w[d] * z / (1.0f + expf(-z)));
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Chunkwise form for prompt portions (bf16 activations) on the tensor cores.  A portion is cut into chunks of up to 128
// tokens.  Inside a chunk with incoming state S0 and G_t [dk] the running sum of the log decays:
//
//   o_t  = sum_{s <= t} P_ts v_s + S0^T (q_t exp(G_t)),    P_ts = sum_d q_t k_s exp(G_t - G_s)
//   S_L  = diag(exp(G_L)) S0 + sum_s (k_s exp(G_L - G_s)) v_s^T
//
// P splits into (q_t exp(G_t)) . (k_s exp(-G_s)) as long as exp(-G_s) stays finite: a key channel whose G falls below
// -GC_RANGE inside the chunk ("steep") is left out of that product and added pair by pair from exp(G_t - G_s) <= 1, so every
// decay is covered and a chunk without steep channels pays nothing for them.
//
// Launches, every chunk of every portion in parallel except for the element-wise scan:
//   gla_decay_kernel         G of every token and channel (fp32)
//   gla_chunk_state_kernel   the sum of S_L                                      [K^T V by tcgen05]
//   gla_chunk_scan_kernel    the incoming state of every chunk and the state the portion leaves behind (fp32)
//   gla_chunk_out_kernel     P by tcgen05, O = Q S0 + P V by tcgen05, head norm and output gate in the epilogue
//
// fp32 operands of a matrix product (decayed queries and keys, P, the incoming state) enter as a bf16 pair hi + lo: two or
// three accumulating products (relative error 2^-16 or less); values are bf16 to begin with.
// ---------------------------------------------------------------------------------------------
struct GlaChunkParams {
  const int* c_start;         // [n_chunks] first packed token
  const int* c_len;           // [n_chunks] tokens (<= 128)
  const int* seq_chunk0;      // [n_seq] first chunk of each portion
  const int* seq_chunks;      // [n_seq] chunks of each portion
  float* G;                   // [n, heads * dk]
  float* dS;                  // [n_chunks, heads, dk, dv]
  __nv_bfloat16* s0;          // [n_chunks, heads, 2 (hi, lo), dk, dv] incoming state
  int n_chunks;
  int* status;
};

constexpr float GC_RANGE = 60.0f;

// The same as log_sigmoid with log1p(x) = 2 artanh(x / (2 + x)) by the series of artanh: x <= 1, so eight terms leave 1.5e-9
// of the value, at any size of x.
__device__ __forceinline__ float log_sigmoid_series(float z) {
  const float x = __expf(-fabsf(z)), s = __fdividef(x, 2.0f + x), q = s * s;
  float r = 2.0f / 15.0f;
  r = fmaf(r, q, 2.0f / 13.0f);
  r = fmaf(r, q, 2.0f / 11.0f);
  r = fmaf(r, q, 2.0f / 9.0f);
  r = fmaf(r, q, 2.0f / 7.0f);
  r = fmaf(r, q, 2.0f / 5.0f);
  r = fmaf(r, q, 2.0f / 3.0f);
  r = fmaf(r, q, 2.0f);
  return fmaf(-r, s, fminf(z, 0.f));
}

// grid (n_chunks, ceil(heads * dk / 32)), 256 threads: thread (segment of 16 tokens, channel)
constexpr int GD_CH = 32, GD_SEG = 16;
__global__ void __launch_bounds__(256) gla_decay_kernel(const GlaParams p, const GlaChunkParams c) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];
  float* s_low = sm;                                   // [128][rank]
  float* s_w = s_low + 128 * p.rank;                   // [rank][GD_CH]
  float* s_tot = s_w + GD_CH * p.rank;                 // [8][GD_CH]
  const int start = c.c_start[blockIdx.x], len = c.c_len[blockIdx.x];
  const int n_ch = p.heads * p.dk, c0 = blockIdx.y * GD_CH;
  for (int i = threadIdx.x; i < 128 * p.rank; i += 256) s_low[i] = i < len * p.rank ? p.low[(size_t)start * p.rank + i] : 0.f;
  for (int i = threadIdx.x; i < GD_CH * p.rank; i += 256) {
    const int ch = i / p.rank, r = i % p.rank;
    s_w[r * GD_CH + ch] = c0 + ch < n_ch ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.w2)[(size_t)(c0 + ch) * p.rank + r]) : 0.f;
  }
  __syncthreads();
  const int ch = threadIdx.x & (GD_CH - 1), seg = threadIdx.x / GD_CH;
  float a[GD_SEG];
  const float b = c0 + ch < n_ch ? p.b2[c0 + ch] : 0.f;
#pragma unroll
  for (int t = 0; t < GD_SEG; ++t) a[t] = b;
  const float4* low = reinterpret_cast<const float4*>(s_low + seg * GD_SEG * p.rank);
  for (int r = 0; r < p.rank; r += 4) {
    const float w0 = s_w[r * GD_CH + ch], w1 = s_w[(r + 1) * GD_CH + ch], w2 = s_w[(r + 2) * GD_CH + ch], w3 = s_w[(r + 3) * GD_CH + ch];
#pragma unroll
    for (int t = 0; t < GD_SEG; ++t) {
      const float4 l = low[(t * p.rank + r) / 4];
      a[t] += w0 * l.x + w1 * l.y + w2 * l.z + w3 * l.w;
    }
  }
  float sum = 0.f;
#pragma unroll
  for (int t = 0; t < GD_SEG; ++t) {
    sum += log_sigmoid_series(a[t]) * p.inv_tau;
    a[t] = sum;
  }
  s_tot[seg * GD_CH + ch] = sum;
  __syncthreads();
  float off = 0.f;
  for (int k = 0; k < seg; ++k) off += s_tot[k * GD_CH + ch];
  if (c0 + ch < n_ch) {
#pragma unroll
    for (int t = 0; t < GD_SEG; ++t)
      if (seg * GD_SEG + t < len) c.G[(size_t)(start + seg * GD_SEG + t) * n_ch + c0 + ch] = a[t] + off;
  }
}

__device__ __forceinline__ void ld8f(const float* p, float* o) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
}
__device__ __forceinline__ void unpack8(const uint4& u, float* o) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = __bfloat1622float2(h[j]);
    o[2 * j] = f.x;
    o[2 * j + 1] = f.y;
  }
}
// 8 values as hi and lo pieces of 16 bytes
__device__ __forceinline__ void split8(const float* v, uint4* hi, uint4* lo) {
  uint32_t a[4], b[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) split_bf16(v[2 * e], v[2 * e + 1], a[e], b[e]);
  *hi = make_uint4(a[0], a[1], a[2], a[3]);
  *lo = make_uint4(b[0], b[1], b[2], b[3]);
}

// 128 columns of the state sum of one (chunk, head): grid (n_chunks, heads, ceil(nv / 2)), 256 threads, two CTAs per SM.
// Shared: K hi and lo (2 chunks of 16 KiB each), V (2 chunks of 16 KiB).
struct GcStateSmem {
  static constexpr int K_HI = 0, K_LO = 2 * MC_KCH, V = 4 * MC_KCH, TAIL = 6 * MC_KCH;
  static constexpr int BYTES = TAIL + 1024;
};

__global__ void __launch_bounds__(256, 2)
gla_chunk_state_kernel(const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_dS, const GlaParams p,
                       const GlaChunkParams c, const int nk, const int nv_all) {
  extern __shared__ __align__(1024) uint8_t mc_smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ch = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 2, nv = min(2, nv_all - v0);
  if ((smem_u32(mc_smem) & 1023u) != 0) {
    pdl_wait();
    if (tid == 0) atomicCAS(c.status, 0, STATUS_BAD_INDEX);
    return;
  }
  float* s_last = reinterpret_cast<float*>(mc_smem + GcStateSmem::TAIL);   // [128] G of the chunk's last token
  uint64_t* full = reinterpret_cast<uint64_t*>(s_last + MC_TOK);
  uint64_t* done = full + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  if (tid == 0) {
    mbar_init(full, 1);
    mbar_init(done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 128);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();            // only now: a successor must not take the tensor memory first
  pdl_wait();
  const uint32_t tmem = *tmem_slot;
  const int start = c.c_start[ch], len = c.c_len[ch];
  if (tid == 0) {
    mbar_expect_tx(full, nv * MC_KCH);
    for (int k = 0; k < nv; ++k) tma_load_3d(mc_smem + GcStateSmem::V + k * MC_KCH, &tm_v, (v0 + k) * 64, h, start, full);
  }
  const int n_ch = p.heads * p.dk;
  if (tid < MC_TOK) s_last[tid] = tid < p.dk ? c.G[(size_t)(start + len - 1) * n_ch + h * p.dk + tid] : 0.f;
  __syncthreads();
  // weighted keys: 16 bytes = 8 dims of one token per step, swizzled as TMA would; the loads of four steps go out together
  constexpr int U = 4;
#pragma unroll 1
  for (int i0 = tid; i0 < MC_TOK * 16; i0 += 256 * U) {
    uint4 raw[U];
    float g[U][8];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * 256, tok = i >> 4, d = (i & 15) * 8;
      if (tok < len && d < p.dk) {
        raw[u] = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.qkvg) + (size_t)(start + tok) * p.ld +
                                                 (size_t)(p.heads + h) * p.dk + d);
        ld8f(c.G + (size_t)(start + tok) * n_ch + h * p.dk + d, g[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * 256, tok = i >> 4, piece = i & 15, d = piece * 8;
      uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
      if (tok < len && d < p.dk) {
        float k[8];
        unpack8(raw[u], k);
#pragma unroll
        for (int e = 0; e < 8; ++e) k[e] *= __expf(s_last[d + e] - g[u][e]);
        split8(k, &hi, &lo);
      }
      const int off = (piece >> 3) * MC_KCH + tok * 128 + (((piece & 7) ^ (tok & 7)) << 4);
      *reinterpret_cast<uint4*>(mc_smem + GcStateSmem::K_HI + off) = hi;
      *reinterpret_cast<uint4*>(mc_smem + GcStateSmem::K_LO + off) = lo;
    }
  }
  fence_proxy_async_smem();
  __syncthreads();
  if (tid == 32) {
    mbar_wait(full, 0, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
    tc_fence_after();
    const uint32_t v_addr = smem_u32(mc_smem + GcStateSmem::V);
    const uint32_t idesc = umma_idesc_bf16_amn_bmn(128, nv * 64);
    for (int part = 0; part < 2; ++part) {
      const uint32_t a_addr = smem_u32(mc_smem + (part == 0 ? GcStateSmem::K_HI : GcStateSmem::K_LO));
#pragma unroll
      for (int ks = 0; ks < MC_TOK / 16; ++ks)
        umma_bf16(tmem, umma_desc_mn_sw128(a_addr + ks * 2048, MC_KCH), umma_desc_mn_sw128(v_addr + ks * 2048, MC_KCH), idesc,
                  (part > 0 || ks > 0) ? 1u : 0u);
    }
    umma_commit(done);
  }
  __syncwarp();                       // the issuing lane of warp 1 rejoins
  mbar_wait(done, 0, abort_flag, c.status, STATUS_TIMEOUT_ACCUM);
  __syncwarp();
  tc_fence_after();
  {
    // [128 key dims][32 columns] fp32 tiles (128-byte swizzled rows) over the operands, then one TMA store per tile
    const int d = (warp & 3) * 32 + lane;                      // row of S (key dim)
    const uint32_t trow = tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16);
    __syncthreads();
#pragma unroll 1
    for (int col = (warp >> 2) * 32; col < nv * 64; col += 64) {
      float o[32];
      tmem_ld32(trow + col, o);
      tmem_ld_wait();
      uint8_t* tile = mc_smem + (col / 32) * MC_KCH;
#pragma unroll
      for (int e = 0; e < 8; ++e)
        *reinterpret_cast<float4*>(tile + d * 128 + ((e ^ (d & 7)) << 4)) = make_float4(o[4 * e], o[4 * e + 1], o[4 * e + 2], o[4 * e + 3]);
    }
    fence_proxy_async_smem();
    __syncthreads();
    if (tid == 0) {
      const size_t chh = (size_t)ch * p.heads + h;
      for (int k = 0; k < nv * 2; ++k)
        if (v0 * 64 + k * 32 < p.dv) tma_store_3d(&tm_dS, mc_smem + k * MC_KCH, v0 * 64 + k * 32, 0, (int)chh);
      tma_store_commit();
      tma_store_wait_read();
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 128);
  }
}

// Scan over the chunks of a portion, element by element: grid (ceil(dk * dv / 4 / 256), heads, n_seq).
__global__ void __launch_bounds__(256) gla_chunk_scan_kernel(const GlaParams p, const GlaChunkParams c) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, s = blockIdx.z;
  const int c0 = c.seq_chunk0[s], nc = c.seq_chunks[s];
  if (nc <= 0) return;
  const int t0 = c.c_start[c0];
  const size_t sh = (size_t)p.row[t0] * p.heads + h;
  const bool fresh = p.pos[t0] == 0;
  const size_t per = (size_t)p.dk * p.dv;
  const int e = blockIdx.x * 256 + threadIdx.x;
  if ((size_t)e * 4 >= per) return;
  const int d = e * 4 / p.dv, n_ch = p.heads * p.dk;
  float4* Sp = reinterpret_cast<float4*>(p.S + sh * per) + e;
  float4 S = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *Sp;
#pragma unroll 4
  for (int k = 0; k < nc; ++k) {
    const size_t chh = (size_t)(c0 + k) * p.heads + h;
    const float4 a = reinterpret_cast<const float4*>(c.dS + chh * per)[e];
    uint32_t hi0, lo0, hi1, lo1;
    split_bf16(S.x, S.y, hi0, lo0);
    split_bf16(S.z, S.w, hi1, lo1);
    reinterpret_cast<uint2*>(c.s0 + chh * 2 * per)[e] = make_uint2(hi0, hi1);
    reinterpret_cast<uint2*>(c.s0 + (chh * 2 + 1) * per)[e] = make_uint2(lo0, lo1);
    const float keep = expf(c.G[(size_t)(c.c_start[c0 + k] + c.c_len[c0 + k] - 1) * n_ch + h * p.dk + d]);
    S.x = fmaf(keep, S.x, a.x); S.y = fmaf(keep, S.y, a.y); S.z = fmaf(keep, S.z, a.z); S.w = fmaf(keep, S.w, a.w);
  }
  *Sp = S;
}

// Outputs of one (chunk, head): grid (n_chunks, heads), 320 threads: warp 0 TMA, warp 1 tensor memory + MMA, warps 2..9
// operands, P and epilogue, two threads per token.  Shared: Q hi, Q lo (2 x 16 KiB each), K hi then P hi, K lo then P lo, ring
// of 3 tiles of 32 KiB: the slices (128 columns) of the incoming state, hi and lo, then the slices of V, then those of the
// output gate, which the outputs replace in place on their way to a TMA store (a chunk of fewer than 128 tokens stores row
// by row).
struct GcOutSmem {
  static constexpr int QHI = 0, QLO = 2 * MC_KCH, KHI = 4 * MC_KCH, KLO = 6 * MC_KCH, RING = 8 * MC_KCH, TILE = 2 * MC_KCH, NRING = 3;
  static constexpr int TAIL = RING + NRING * TILE;
  static constexpr int BYTES = TAIL + 2304;
};
constexpr int GC_OUT_THREADS = 320;

__global__ void __launch_bounds__(GC_OUT_THREADS, 1)
gla_chunk_out_kernel(const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_s0,
                     const __grid_constant__ CUtensorMap tm_out, const GlaParams p, const GlaChunkParams c, const int nk, const int nv) {
  extern __shared__ __align__(1024) uint8_t mc_smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ch = blockIdx.x, h = blockIdx.y;
  if ((smem_u32(mc_smem) & 1023u) != 0) {
    pdl_wait();
    if (tid == 0) atomicCAS(c.status, 0, STATUS_BAD_INDEX);
    return;
  }
  float* s_keep = reinterpret_cast<float*>(mc_smem + GcOutSmem::TAIL);   // [128] 1, or 0 for a steep channel
  float* s_x = s_keep + MC_TOK;                                          // [128] exchange (low half -> high half and back)
  int* s_steep = reinterpret_cast<int*>(s_x + MC_TOK);                   // [128] steep channels
  int* s_count = s_steep + MC_TOK;                                       // [4] of each warp of 32 channels
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_count + 4);
  uint64_t* qk_full = bars;                      // operands written (256 arrivals)
  uint64_t* full = bars + 1;                     // [NRING]
  uint64_t* empty = full + GcOutSmem::NRING;     // [NRING]
  uint64_t* s_done = empty + GcOutSmem::NRING;   // Q K^T complete
  uint64_t* p_ready = s_done + 1;                // P written (256 arrivals)
  uint64_t* o_done = p_ready + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  if (tid == 0) {
    mbar_init(qk_full, 256);
    for (int s = 0; s < GcOutSmem::NRING; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    mbar_init(s_done, 1);
    mbar_init(p_ready, 256);
    mbar_init(o_done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();            // only now: a successor must not take the tensor memory first
  pdl_wait();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + 128;
  const int start = c.c_start[ch], len = c.c_len[ch];
  const size_t chh = (size_t)ch * p.heads + h;
  const int slices = (nv + 1) / 2;
  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      for (int i = 0; i < 4 * slices; ++i) {
        const int st = i % GcOutSmem::NRING;
        mbar_wait(&empty[st], ((i / GcOutSmem::NRING) & 1) ^ 1, abort_flag, c.status, STATUS_TIMEOUT_STAGE_EMPTY);
        if (*abort_flag) break;
        uint8_t* dst = mc_smem + GcOutSmem::RING + st * GcOutSmem::TILE;
        const bool state = i < 2 * slices;
        const int sl = state ? i / 2 : i % slices;              // 2 * slices and 3 * slices are multiples of slices
        const int cols = min(2, nv - 2 * sl);
        const int bytes = state ? nk * 8192 : MC_KCH;         // one 64-column chunk: nk * 64 state rows, or 128 tokens
        mbar_expect_tx(&full[st], cols * bytes);
        for (int k = 0; k < cols; ++k) {
          const int x = (2 * sl + k) * 64;
          if (state) {
            for (int r = 0; r < nk; ++r)
              tma_load_3d(dst + k * bytes + r * 8192, &tm_s0, x, r * 64, (int)(chh * 2 + (i & 1)), &full[st]);
          } else {
            tma_load_3d(dst + k * bytes, &tm_v, x, i < 3 * slices ? h : p.heads + h, start, &full[st]);
          }
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      const uint32_t qhi = smem_u32(mc_smem + GcOutSmem::QHI), qlo = smem_u32(mc_smem + GcOutSmem::QLO);
      const uint32_t khi = smem_u32(mc_smem + GcOutSmem::KHI), klo = smem_u32(mc_smem + GcOutSmem::KLO);
      mbar_wait(qk_full, 0, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
      tc_fence_after();
      for (int part = 0; part < 3; ++part) {
        const uint32_t a = part == 2 ? qlo : qhi, b = part == 1 ? klo : khi;
        for (int ks = 0; ks < nk * 4; ++ks) {
          const uint32_t off = (ks / 4) * MC_KCH + (ks % 4) * 32;
          umma_bf16(tmem_s, umma_desc_sw128(a + off), umma_desc_sw128(b + off), umma_idesc_bf16(128, 128), (part > 0 || ks > 0) ? 1u : 0u);
        }
      }
      umma_commit(s_done);
      for (int i = 0; i < 3 * slices; ++i) {
        const int st = i % GcOutSmem::NRING;
        if (i == 2 * slices) {
          mbar_wait(p_ready, 0, abort_flag, c.status, STATUS_TIMEOUT_ACCUM);
          tc_fence_after();
        }
        mbar_wait(&full[st], (i / GcOutSmem::NRING) & 1, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
        tc_fence_after();
        const uint32_t b_addr = smem_u32(mc_smem + GcOutSmem::RING + st * GcOutSmem::TILE);
        const bool state = i < 2 * slices;
        const int sl = state ? i / 2 : i - 2 * slices;
        const uint32_t idesc = umma_idesc_bf16_bmn(128, min(2, nv - 2 * sl) * 64);
        const uint32_t d = tmem_o + sl * 128;
        if (state) {                               // hi: Q hi and Q lo, lo: Q hi
          const uint32_t lbo = nk * 8192;
          for (int part = 0; part < ((i & 1) ? 1 : 2); ++part)
            for (int ks = 0; ks < nk * 4; ++ks)
              umma_bf16(d, umma_desc_sw128((part == 0 ? qhi : qlo) + (ks / 4) * MC_KCH + (ks % 4) * 32),
                        umma_desc_mn_sw128(b_addr + ks * 2048, lbo), idesc, (ks > 0 || part > 0 || (i & 1)) ? 1u : 0u);
        } else {
          for (int part = 0; part < 2; ++part)
            for (int ks = 0; ks < 8; ++ks)
              umma_bf16(d, umma_desc_sw128((part == 0 ? khi : klo) + (ks / 4) * MC_KCH + (ks % 4) * 32),
                        umma_desc_mn_sw128(b_addr + ks * 2048, MC_KCH), idesc, 1u);
        }
        umma_commit(&empty[st]);
      }
      umma_commit(o_done);
    }
    __syncwarp();
  } else {
    // ---------------- two threads per token ----------------
    const int qd = warp & 3, half = (warp - 2) >> 2;
    const int t = qd * 32 + lane, ct = tid - 64;     // ct: index among the 256 threads
    const bool ok = t < len;
    const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
    const int n_ch = p.heads * p.dk;
    const __nv_bfloat16* qk = reinterpret_cast<const __nv_bfloat16*>(p.qkvg) + (size_t)start * p.ld;   // q of head x, then k
    const float* G = c.G + (size_t)start * n_ch + h * p.dk;
    if (ct < MC_TOK) {
      const bool steep = ct < p.dk && G[(size_t)(len - 1) * n_ch + ct] < -GC_RANGE;
      s_keep[ct] = steep ? 0.f : 1.f;
      const unsigned ball = __ballot_sync(0xffffffffu, steep);
      if (steep) s_steep[(ct & ~31) + __popc(ball & ((1u << lane) - 1u))] = ct;
      if (lane == 0) s_count[ct >> 5] = __popc(ball);
    }
    named_bar_sync(1, 256);
    constexpr int U = 4;                             // steps whose loads go out together
#pragma unroll 1
    for (int i0 = ct; i0 < MC_TOK * 16; i0 += 256 * U) {
      uint4 rq[U], rk[U];
      float g[U][8];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i0 + u * 256, tok = i >> 4, d = (i & 15) * 8;
        if (tok < len && d < p.dk) {
          const __nv_bfloat16* row = qk + (size_t)tok * p.ld + d;
          rq[u] = *reinterpret_cast<const uint4*>(row + (size_t)h * p.dk);
          rk[u] = *reinterpret_cast<const uint4*>(row + (size_t)(p.heads + h) * p.dk);
          ld8f(G + (size_t)tok * n_ch + d, g[u]);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i0 + u * 256, tok = i >> 4, piece = i & 15, d = piece * 8;
        if (piece >= nk * 8) continue;
        uint4 ah = make_uint4(0u, 0u, 0u, 0u), al = ah, bh = ah, bl = ah;
        if (tok < len && d < p.dk) {
          float q[8], k[8];
          unpack8(rq[u], q);
          unpack8(rk[u], k);
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float f = __expf(g[u][e]);
            q[e] *= p.q_scale * f;
            k[e] = s_keep[d + e] != 0.f ? __fdividef(k[e], f) : 0.f;
          }
          split8(q, &ah, &al);
          split8(k, &bh, &bl);
        }
        const int off = (piece >> 3) * MC_KCH + tok * 128 + (((piece & 7) ^ (tok & 7)) << 4);
        *reinterpret_cast<uint4*>(mc_smem + GcOutSmem::QHI + off) = ah;
        *reinterpret_cast<uint4*>(mc_smem + GcOutSmem::QLO + off) = al;
        *reinterpret_cast<uint4*>(mc_smem + GcOutSmem::KHI + off) = bh;
        *reinterpret_cast<uint4*>(mc_smem + GcOutSmem::KLO + off) = bl;
      }
    }
    fence_proxy_async_smem();
    mbar_arrive(qk_full);
    // P for s <= t: this thread's 64 columns, written over K hi and lo
    mbar_wait(s_done, 0, abort_flag, c.status, STATUS_TIMEOUT_ACCUM);
    tc_fence_after();
#pragma unroll 1
    for (int c0 = 0; c0 < 64; c0 += 32) {
      const int s0 = half * 64 + c0;
      float sv[32];
      if (s0 > qd * 32 + 31) {                     // right of the diagonal for every token of the warp
        const uint4 z = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
        for (int v = 0; v < 4; ++v) {
          const int off = half * MC_KCH + t * 128 + (((c0 / 8 + v) ^ (t & 7)) << 4);
          *reinterpret_cast<uint4*>(mc_smem + GcOutSmem::KHI + off) = z;
          *reinterpret_cast<uint4*>(mc_smem + GcOutSmem::KLO + off) = z;
        }
        continue;
      }
      tmem_ld32(tmem_s + lane_off + s0, sv);
      tmem_ld_wait();
#pragma unroll
      for (int e = 0; e < 32; ++e) sv[e] = ok && s0 + e <= t ? sv[e] : 0.f;
      for (int w = 0; w < 4; ++w) {
        for (int j = 0; j < s_count[w]; ++j) {     // steep channels, pair by pair
          const int d = s_steep[w * 32 + j];
          const float gt = ok ? G[(size_t)t * n_ch + d] : 0.f;
          const float qt = ok ? __bfloat162float(qk[(size_t)t * p.ld + (size_t)h * p.dk + d]) * p.q_scale : 0.f;
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            const int s = min(s0 + e, len - 1);
            const float ks = __bfloat162float(qk[(size_t)s * p.ld + (size_t)(p.heads + h) * p.dk + d]);
            if (ok && s0 + e <= t) sv[e] = fmaf(qt * ks, __expf(gt - G[(size_t)s * n_ch + d]), sv[e]);
          }
        }
      }
#pragma unroll
      for (int v = 0; v < 4; ++v) {
        uint4 hi, lo;
        split8(sv + v * 8, &hi, &lo);
        const int off = half * MC_KCH + t * 128 + (((c0 / 8 + v) ^ (t & 7)) << 4);
        *reinterpret_cast<uint4*>(mc_smem + GcOutSmem::KHI + off) = hi;
        *reinterpret_cast<uint4*>(mc_smem + GcOutSmem::KLO + off) = lo;
      }
    }
    fence_proxy_async_smem();
    tc_fence_before();
    mbar_arrive(p_ready);
    mbar_wait(o_done, 0, abort_flag, c.status, STATUS_TIMEOUT_ACCUM);
    tc_fence_after();
    float ss = 0.f;
#pragma unroll 1
    for (int col = half * 32; col < nv * 64; col += 64) {
      float o[32];
      tmem_ld32(tmem_o + lane_off + col, o);
      tmem_ld_wait();
#pragma unroll
      for (int e = 0; e < 32; ++e) ss = fmaf(o[e], o[e], ss);
    }
    if (half == 1) s_x[t] = ss;
    named_bar_sync(1, 256);
    if (half == 0) { ss += s_x[t]; s_x[t] = ss; }
    named_bar_sync(1, 256);
    const float r = 1.0f / sqrtf(s_x[t] / (float)p.vdim + p.eps);
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(start + t) * p.ld_out + (size_t)h * p.dv;
    const bool whole = len == MC_TOK;
    for (int sl = 0; sl < slices; ++sl) {
      const int i = 3 * slices + sl, st = i % GcOutSmem::NRING;
      uint8_t* tile = mc_smem + GcOutSmem::RING + st * GcOutSmem::TILE;
      mbar_wait(&full[st], (i / GcOutSmem::NRING) & 1, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
#pragma unroll 1
      for (int c0 = half * 32; c0 < min(2, nv - 2 * sl) * 64; c0 += 64) {
        const int col = sl * 128 + c0;
        float o[32];
        tmem_ld32(tmem_o + lane_off + col, o);
        tmem_ld_wait();
#pragma unroll
        for (int v = 0; v < 32; v += 8) {
          uint4* slot = reinterpret_cast<uint4*>(tile + (c0 / 64) * MC_KCH + t * 128 + ((((c0 & 63) + v) / 8 ^ (t & 7)) << 4));
          const uint4 gu = *slot;
          const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gu);
          uint4 pk;
          __nv_bfloat162* p2 = reinterpret_cast<__nv_bfloat162*>(&pk);
          const bool in = col + v < p.dv;
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 z = __bfloat1622float2(g2[e]);
            const float2 w = in ? __ldg(reinterpret_cast<const float2*>(p.norm_w + col + v + 2 * e)) : make_float2(0.f, 0.f);
            p2[e] = __floats2bfloat162_rn(o[v + 2 * e] * r * w.x * silu(z.x), o[v + 2 * e + 1] * r * w.y * silu(z.y));
          }
          if (whole) *slot = pk;
          else if (ok && in) *reinterpret_cast<uint4*>(out + col + v) = pk;
        }
      }
      if (whole) {
        fence_proxy_async_smem();
        named_bar_sync(1, 256);
        if (warp == 2 && lane == 0) {
          for (int k = 0; k < min(2, nv - 2 * sl); ++k) tma_store_3d(&tm_out, tile + k * MC_KCH, (2 * sl + k) * 64, h, start);
          tma_store_commit();
        }
      }
    }
    if (warp == 2 && lane == 0) tma_store_wait_read();            // shared memory may go only when the stores have read it
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_s, 512);
  }
}

}  // namespace tahb

using namespace tahb;

extern "C" int tahb_gla_recurrent(const GlaParams* p, int f32, cudaStream_t stream) {
  if (p->n_seq <= 0) return 0;
  if (p->dk % 8 || p->dv % 8 || p->dv > GR_MAX_D || p->dk > GR_MAX_D || p->n_seq > 65535 || p->rank % 4 || p->rank < 4) return -2;
  const int nrg = GR_THREADS / (p->dv / 4);
  const size_t smem = ((size_t)3 * p->dk + (size_t)nrg * p->dv + 8) * 4;
  const dim3 grid(p->heads, p->n_seq);
  cudaError_t e = f32 ? launch_chain(gla_recurrent_kernel<float>, grid, dim3(GR_THREADS), smem, stream, *p)
                      : launch_chain(gla_recurrent_kernel<__nv_bfloat16>, grid, dim3(GR_THREADS), smem, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}

// Chunkwise form: bf16 activations, dk <= 128, dv <= 256.  `n_tokens` = rows of qkvg.
extern "C" int tahb_gla_chunks(const GlaParams* p, const GlaChunkParams* c, int n_tokens, cudaStream_t stream) {
  if (p->n_seq <= 0 || c->n_chunks <= 0) return 0;
  if (p->dk % 8 || p->dv % 8 || p->dk > 128 || p->dv > 256 || p->n_seq > 65535 || p->heads > 65535 || p->ld_out % 8 || p->ld % 8 ||
      p->rank % 4 || p->rank < 4)
    return -2;
  const int nk = (p->dk + 63) / 64, nv = (p->dv + 63) / 64;
  auto base = reinterpret_cast<const __nv_bfloat16*>(p->qkvg);
  CUtensorMap mv, ms, mo, md;
  int rc;
  if ((rc = make_head_map(&mv, base + (size_t)2 * p->heads * p->dk, p->dv, 2 * p->heads, n_tokens, p->ld))) return rc;
  if ((rc = make_state_map(&ms, c->s0, p->dk, p->dv, (long long)c->n_chunks * p->heads * 2))) return rc;
  if ((rc = make_head_map(&mo, reinterpret_cast<const __nv_bfloat16*>(p->out), p->dv, p->heads, n_tokens, p->ld_out))) return rc;
  if ((rc = make_dS_map(&md, c->dS, p->dk, p->dv, (long long)c->n_chunks * p->heads))) return rc;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(gla_decay_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(gla_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, GcStateSmem::BYTES) != cudaSuccess ||
        cudaFuncSetAttribute(gla_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, GcOutSmem::BYTES) != cudaSuccess)
      return -10;
    configured = true;
  }
  const size_t decay_smem = ((size_t)(128 + GD_CH) * p->rank + 8 * GD_CH) * 4;
  if (decay_smem > 200 * 1024) return -2;
  cudaError_t e = launch_chain(gla_decay_kernel, dim3(c->n_chunks, (p->heads * p->dk + GD_CH - 1) / GD_CH), dim3(256), decay_smem, stream, *p, *c);
  if (e == cudaSuccess)
    e = launch_chain(gla_chunk_state_kernel, dim3(c->n_chunks, p->heads, (nv + 1) / 2), dim3(256), GcStateSmem::BYTES, stream, mv, md, *p, *c, nk, nv);
  const int blocks = (int)(((long long)p->dk * p->dv / 4 + 255) / 256);
  if (e == cudaSuccess) e = launch_chain(gla_chunk_scan_kernel, dim3(blocks, p->heads, p->n_seq), dim3(256), 0, stream, *p, *c);
  if (e == cudaSuccess)
    e = launch_chain(gla_chunk_out_kernel, dim3(c->n_chunks, p->heads), dim3(GC_OUT_THREADS), GcOutSmem::BYTES, stream, mv, ms, mo, *p, *c, nk, nv);
  return e == cudaSuccess ? 0 : -3;
}
