// Matrix memory of mLSTM layers.  Per head, with log gates i_t = cap tanh(zi_t / cap), f_t = logsigmoid(cap tanh(zf_t / cap)):
//
//   m_t = max(f_t + m_{t-1}, i_t)                        (m starts at 0)
//   S_t = exp(f_t + m_{t-1} - m_t) S_{t-1} + exp(i_t - m_t) k_t v_t^T      [dk, dv]
//   n_t = exp(f_t + m_{t-1} - m_t) n_{t-1} + exp(i_t - m_t) k_t            [dk]
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
//   y_t = rms(o_t) * w * sigmoid(g_t)
//
// S, n and m live in fp32, one slot per cache row: state[slot][head] = S [dk][dv], n [dk], m.  A token at position 0
// starts from zero, so a slot needs no clearing when it changes hands.  dk and dv are padded to multiples of 8 with zeros.
#include <cuda.h>

#include "chunk_common.cuh"

namespace tahb {

struct MlstmParams {
  const void* qkvg;           // [n, ld]: heads * dk of q, heads * dk of k, heads * dv of v, heads * dv of g
  const float* gates;         // [n, 2 * heads]: zi of every head, then zf
  const float* norm_w;        // [heads * dv]
  void* out;                  // [n, ld_out], head h at column h * dv
  float* S;                   // [slots, heads, dk, dv]
  float* nvec;                // [slots, heads, dk]
  float* mval;                // [slots, heads]
  const int* seq_start;       // [n_seq] first packed token of each sequence, null = sequence s is token s
  const int* seq_len;         // [n_seq] tokens of each sequence, null = 1
  const int* pos;             // [n] position of each packed token
  const int* row;             // [n] state slot of each packed token
  const int* slot;            // [n] KV slot; negative = the row is idle and its state stays (may be null)
  int n_seq, heads, dk, dv, dim, vdim;        // dim, vdim: real sizes
  long long ld, ld_out;
  float cap, eps, q_scale;
};

__device__ __forceinline__ float mlstm_log_i(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float mlstm_log_f(float z, float cap) {
  const float u = cap * tanhf(z / cap);
  return fminf(u, 0.f) - log1pf(expf(-fabsf(u)));
}

// ---------------------------------------------------------------------------------------------
// Recurrent form: grid (heads, n_seq), 256 threads; the tokens of a sequence one after another.  Thread (rg, c) owns the
// float4 column c of the rows rg, rg + nrg, ... of S, read and written in place (one token: the state streams through
// once, which is the whole cost of a decode step).
// ---------------------------------------------------------------------------------------------
constexpr int MR_THREADS = 256;
constexpr int MR_MAX_D = 1024;

template <typename T>
__global__ void __launch_bounds__(MR_THREADS, 3) mlstm_recurrent_kernel(const MlstmParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x, s = blockIdx.y;
  const int dk = p.dk, dv = p.dv, ncol = dv / 4, nrg = MR_THREADS / ncol;
  float* s_q = sm;                       // [dk]
  float* s_k = s_q + dk;                 // [dk]
  float* s_n = s_k + dk;                 // [dk]
  float* s_red = s_n + dk;               // [nrg][dv]
  float* s_w = s_red + (size_t)nrg * dv; // [32] warp partials
  const int t0 = p.seq_start ? p.seq_start[s] : s, len = p.seq_len ? p.seq_len[s] : 1;
  if (len <= 0) return;
  if (p.slot != nullptr && p.slot[t0] < 0) {     // idle row: leave the state alone
    T* o = reinterpret_cast<T*>(p.out) + (size_t)t0 * p.ld_out + (size_t)h * dv;
    for (int d = tid; d < dv; d += MR_THREADS) stf(o + d, 0.f);
    return;
  }
  const size_t sh = (size_t)p.row[t0] * p.heads + h;
  float* S = p.S + sh * dk * dv;
  float* N = p.nvec + sh * dk;
  bool fresh = p.pos[t0] == 0;
  float m = fresh ? 0.f : p.mval[sh];
  for (int d = tid; d < dk; d += MR_THREADS) s_n[d] = fresh ? 0.f : N[d];
  const int rg = tid / ncol, c = tid % ncol;
  for (int t = t0; t < t0 + len; ++t) {
    const T* base = reinterpret_cast<const T*>(p.qkvg) + (size_t)t * p.ld;
    const T* q = base + (size_t)h * dk;
    const T* k = base + (size_t)(p.heads + h) * dk;
    const T* v = base + (size_t)2 * p.heads * dk + (size_t)h * dv;
    const T* g = base + (size_t)2 * p.heads * dk + (size_t)(p.heads + h) * dv;
    const float li = mlstm_log_i(p.gates[(size_t)t * 2 * p.heads + h], p.cap);
    const float lf = mlstm_log_f(p.gates[(size_t)t * 2 * p.heads + p.heads + h], p.cap);
    const float m_new = fmaxf(lf + m, li);
    const float keep = expf(lf + m - m_new), add = expf(li - m_new);
    m = m_new;
    __syncthreads();                     // the previous token's s_q / s_k / s_red have been read
    float nq = 0.f;
    for (int d = tid; d < dk; d += MR_THREADS) {
      const float qd = ldf(q + d) * p.q_scale, kd = ldf(k + d);
      const float nd = keep * s_n[d] + add * kd;
      s_q[d] = qd;
      s_k[d] = add * kd;
      s_n[d] = nd;
      nq = fmaf(nd, qd, nq);
    }
    nq = warp_sum(nq);
    if (lane == 0) s_w[warp] = nq;
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
            const float kr = s_k[r], qr = s_q[r];
            a[u].x = fmaf(keep, a[u].x, kr * vv.x); a[u].y = fmaf(keep, a[u].y, kr * vv.y);
            a[u].z = fmaf(keep, a[u].z, kr * vv.z); a[u].w = fmaf(keep, a[u].w, kr * vv.w);
            o.x = fmaf(a[u].x, qr, o.x); o.y = fmaf(a[u].y, qr, o.y); o.z = fmaf(a[u].z, qr, o.z); o.w = fmaf(a[u].w, qr, o.w);
            *(reinterpret_cast<float4*>(S + (size_t)r * dv) + c) = a[u];
          }
        }
      }
      *reinterpret_cast<float4*>(s_red + (size_t)rg * dv + c * 4) = o;
    }
    fresh = false;
    nq = 0.f;
#pragma unroll
    for (int w = 0; w < MR_THREADS / 32; ++w) nq += s_w[w];
    const float inv = 1.0f / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
    __syncthreads();
    float ss = 0.f;
    for (int d = tid; d < dv; d += MR_THREADS) {
      float o = 0.f;
      for (int r = 0; r < nrg; ++r) o += s_red[(size_t)r * dv + d];
      o *= inv;
      s_red[d] = o;                      // row 0 is rewritten by the thread that read this column of every row
      ss = fmaf(o, o, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) s_w[16 + warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < MR_THREADS / 32; ++w) ss += s_w[16 + w];
    const float r = 1.0f / sqrtf(ss / (float)p.vdim + p.eps);
    T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + (size_t)h * dv;
    for (int d = tid; d < dv; d += MR_THREADS) {
      const float z = ldf(g + d);
      stf(out + d, s_red[d] * r * p.norm_w[(size_t)h * dv + d] / (1.0f + expf(-z)));
    }
  }
  __syncthreads();
  for (int d = tid; d < dk; d += MR_THREADS) N[d] = s_n[d];
  if (tid == 0) p.mval[sh] = m;
}

// ---------------------------------------------------------------------------------------------
// Chunkwise form for prompt portions (bf16 activations) on the tensor cores.  A portion is cut into chunks of up to 128
// tokens.  Inside a chunk with incoming state (S0, n0, m0), F_t the running sum of the log forget gates and
// B_s = i_s - F_s:
//
//   m_t = F_t + max(m0, max_{s <= t} B_s)                                    the same running maximum as token by token
//   P_ts = (q_t . k_s) exp(F_t - m_t + B_s)        for s <= t
//   o_t  = (sum_s P_ts v_s + a_t S0^T q_t) / (max(|sum_s P_ts + a_t n0 . q_t|, exp(-m_t)) + 1e-6),  a_t = exp(F_t + m0 - m_t)
//
// Three launches, every chunk of every portion in parallel except for the element-wise scan:
//   mlstm_chunk_state_kernel   dS = sum_s exp(F_L + B_s - M) k_s v_s^T,  M = F_L + max_s B_s         [K^T V by tcgen05]
//   mlstm_chunk_scan_kernel    the incoming state of every chunk and the state the portion leaves behind (fp32)
//   mlstm_chunk_out_kernel     P by tcgen05 (Q K^T) and registers, O by tcgen05, head norm and output gate in the epilogue
//
// fp32 operands of a matrix product (P, the weighted keys, the incoming state) enter as a bf16 pair hi + lo, two
// accumulating products (relative error 2^-17 or less); queries, keys and values are bf16 to begin with.
// ---------------------------------------------------------------------------------------------
struct MlstmChunkParams {
  const int* c_start;         // [n_chunks] first packed token
  const int* c_len;           // [n_chunks] tokens (<= 128)
  const int* seq_chunk0;      // [n_seq] first chunk of each portion
  const int* seq_chunks;      // [n_seq] chunks of each portion
  float* dS;                  // [n_chunks, heads, dk, dv]
  float* dn;                  // [n_chunks, heads, dk]
  float* cg;                  // [n_chunks, heads, 2]: F_L, max_s B_s
  __nv_bfloat16* s0;          // [n_chunks, heads, 2 (hi, lo), dk, dv] incoming state
  float* n0;                  // [n_chunks, heads, dk]
  float* m0;                  // [n_chunks, heads]
  int n_chunks;
  int* status;
};

// Gate scan of a chunk by 256 threads (named barrier 1), t = their index; tokens are t < 128.
// F = inclusive sum of the log forget gates, B = log_i - F, Bmax = inclusive prefix maximum of B.  xw: 8 floats.
__device__ __forceinline__ void chunk_gates(const float* gates, int heads, int h, int start, int len, float cap, float* xw,
                                            int t, float& F, float& B, float& Bmax) {
  const int lane = t & 31, w = t >> 5;
  F = 0.f;
  B = -INFINITY;
  float li = -INFINITY;
  if (t < len) {
    li = mlstm_log_i(gates[(size_t)(start + t) * 2 * heads + h], cap);
    F = mlstm_log_f(gates[(size_t)(start + t) * 2 * heads + heads + h], cap);
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float v = __shfl_up_sync(0xffffffffu, F, o);
    if (lane >= o) F += v;
  }
  if (w < 4 && lane == 31) xw[w] = F;
  named_bar_sync(1, 256);
  for (int k = 0; k < min(w, 4); ++k) F += xw[k];
  if (t < len) B = li - F;
  Bmax = B;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float v = __shfl_up_sync(0xffffffffu, Bmax, o);
    if (lane >= o) Bmax = fmaxf(Bmax, v);
  }
  if (w < 4 && lane == 31) xw[4 + w] = Bmax;
  named_bar_sync(1, 256);
  for (int k = 0; k < min(w, 4); ++k) Bmax = fmaxf(Bmax, xw[4 + k]);
}

// 128 columns of dS of one (chunk, head): grid (n_chunks, heads, ceil(nv / 2)), 256 threads, two CTAs per SM.  Shared: K hi
// and lo (2 chunks of 16 KiB each), V (2 chunks of 16 KiB).
struct McStateSmem {
  static constexpr int K_HI = 0, K_LO = 2 * MC_KCH, V = 4 * MC_KCH, TAIL = 6 * MC_KCH;
  static constexpr int BYTES = TAIL + 2048;
};

__global__ void __launch_bounds__(256, 2)
mlstm_chunk_state_kernel(const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                         const __grid_constant__ CUtensorMap tm_dS, const MlstmParams p, const MlstmChunkParams c, const int nv_all) {
  extern __shared__ __align__(1024) uint8_t mc_smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ch = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 2, nv = min(2, nv_all - v0);
  if ((smem_u32(mc_smem) & 1023u) != 0) {
    if (tid == 0) atomicCAS(c.status, 0, STATUS_BAD_INDEX);
    return;
  }
  float* s_w = reinterpret_cast<float*>(mc_smem + McStateSmem::TAIL);   // [128] weight of each token
  float* s_dn = s_w + MC_TOK;                                  // [128] half sums of dn
  float* s_x = s_dn + MC_TOK;                                  // [8]
  uint64_t* full = reinterpret_cast<uint64_t*>(s_x + 8);
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
  const uint32_t tmem = *tmem_slot;
  const int start = c.c_start[ch], len = c.c_len[ch];
  if (tid == 0) {
    mbar_expect_tx(full, (2 + nv) * MC_KCH);
    for (int k = 0; k < 2; ++k) tma_load_3d(mc_smem + McStateSmem::K_HI + k * MC_KCH, &tm_k, k * 64, p.heads + h, start, full);
    for (int k = 0; k < nv; ++k) tma_load_3d(mc_smem + McStateSmem::V + k * MC_KCH, &tm_v, (v0 + k) * 64, h, start, full);
  }
  float F, B, Bmax;
  chunk_gates(p.gates, p.heads, h, start, len, p.cap, s_x, tid, F, B, Bmax);
  float* s_last = reinterpret_cast<float*>(tmem_slot + 2);     // [2] F and prefix maximum of the chunk's last token
  if (tid == len - 1) { s_last[0] = F; s_last[1] = Bmax; }
  __syncthreads();
  const size_t chh = (size_t)ch * p.heads + h;
  if (tid < MC_TOK) s_w[tid] = tid < len ? expf(B - s_last[1]) : 0.f;
  if (tid == 0 && v0 == 0) { c.cg[chh * 2] = s_last[0]; c.cg[chh * 2 + 1] = s_last[1]; }
  __syncthreads();
  mbar_wait(full, 0, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
  // weighted keys: hi in place, lo beside them (16 bytes = 8 dims of one token per step; the swizzle only permutes
  // 16-byte pieces inside a token's 128 bytes)
  for (int i = tid; i < 2 * MC_TOK * 8; i += 256) {
    const int tok = (i >> 3) & (MC_TOK - 1);
    const float w = s_w[tok];
    uint4* kp = reinterpret_cast<uint4*>(mc_smem + McStateSmem::K_HI) + i;
    const uint4 kv = *kp;
    const __nv_bfloat162* k2 = reinterpret_cast<const __nv_bfloat162*>(&kv);
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(k2[e]);
      split_bf16(tok < len ? f.x * w : 0.f, tok < len ? f.y * w : 0.f, hi[e], lo[e]);
    }
    *kp = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    reinterpret_cast<uint4*>(mc_smem + McStateSmem::K_LO)[i] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  fence_proxy_async_smem();
  __syncthreads();
  if (tid == 32) {
    tc_fence_after();
    const uint32_t v_addr = smem_u32(mc_smem + McStateSmem::V);
    const uint32_t idesc = umma_idesc_bf16_amn_bmn(128, nv * 64);
    for (int part = 0; part < 2; ++part) {
      const uint32_t a_addr = smem_u32(mc_smem + (part == 0 ? McStateSmem::K_HI : McStateSmem::K_LO));
#pragma unroll
      for (int ks = 0; ks < MC_TOK / 16; ++ks)
        umma_bf16(tmem, umma_desc_mn_sw128(a_addr + ks * 2048, MC_KCH), umma_desc_mn_sw128(v_addr + ks * 2048, MC_KCH), idesc,
                  (part > 0 || ks > 0) ? 1u : 0u);
    }
    umma_commit(done);
  }
  __syncwarp();                       // the issuing lane of warp 1 rejoins
  // dn[d] = sum of the weighted keys of dim d: two threads per dim, 64 tokens each
  if (v0 == 0) {
    const int d = tid & (MC_TOK - 1), th = tid >> 7;
    float s0 = 0.f, s1 = 0.f;
    const uint8_t* base = mc_smem + (d >> 6) * MC_KCH;
    const int piece = (d & 63) >> 3, within = (d & 7) * 2;
#pragma unroll 8
    for (int t = th * 64; t < th * 64 + 64; ++t) {             // tokens past the end weigh zero
      const int off = t * 128 + ((piece ^ (t & 7)) << 4) + within;
      s0 += __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(base + McStateSmem::K_HI + off));
      s1 += __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(base + McStateSmem::K_LO + off));
    }
    if (th == 1) s_dn[d] = s0 + s1;
    __syncthreads();
    if (th == 0 && d < p.dk) c.dn[chh * p.dk + d] = s0 + s1 + s_dn[d];
  }
  mbar_wait(done, 0, abort_flag, c.status, STATUS_TIMEOUT_ACCUM);
  __syncwarp();
  tc_fence_after();
  {
    // [128 key dims][32 columns] fp32 tiles (128-byte swizzled rows) over the operands, then one TMA store per tile
    const int d = (warp & 3) * 32 + lane;                      // row of S (key dim)
    const uint32_t trow = tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16);
    __syncthreads();                                           // every thread has read the weighted keys
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

// Scan over the chunks of a portion, element by element: grid (ceil(dk * dv / 4 / 256) + 1, heads, n_seq).  The last
// block of x handles n and m.
__global__ void __launch_bounds__(256) mlstm_chunk_scan_kernel(const MlstmParams p, const MlstmChunkParams c) {
  const int h = blockIdx.y, s = blockIdx.z;
  const int c0 = c.seq_chunk0[s], nc = c.seq_chunks[s];
  if (nc <= 0) return;
  const int t0 = c.c_start[c0];
  const size_t sh = (size_t)p.row[t0] * p.heads + h;
  const bool fresh = p.pos[t0] == 0;
  float m = fresh ? 0.f : p.mval[sh];
  const size_t per = (size_t)p.dk * p.dv;
  if (blockIdx.x + 1 < gridDim.x) {
    const int e = blockIdx.x * 256 + threadIdx.x;
    if ((size_t)e * 4 >= per) return;
    float4* Sp = reinterpret_cast<float4*>(p.S + sh * per) + e;
    float4 S = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *Sp;
#pragma unroll 4
    for (int k = 0; k < nc; ++k) {
      const size_t chh = (size_t)(c0 + k) * p.heads + h;
      const float4 d = reinterpret_cast<const float4*>(c.dS + chh * per)[e];
      uint32_t hi0, lo0, hi1, lo1;
      split_bf16(S.x, S.y, hi0, lo0);
      split_bf16(S.z, S.w, hi1, lo1);
      reinterpret_cast<uint2*>(c.s0 + chh * 2 * per)[e] = make_uint2(hi0, hi1);
      reinterpret_cast<uint2*>(c.s0 + (chh * 2 + 1) * per)[e] = make_uint2(lo0, lo1);
      const float FL = c.cg[chh * 2], Bm = c.cg[chh * 2 + 1];
      const float m_new = FL + fmaxf(m, Bm);
      const float keep = expf(FL + m - m_new), add = expf(FL + Bm - m_new);
      S.x = keep * S.x + add * d.x; S.y = keep * S.y + add * d.y;
      S.z = keep * S.z + add * d.z; S.w = keep * S.w + add * d.w;
      m = m_new;
    }
    *Sp = S;
    return;
  }
  // n and the chunks' m (the slot's m itself is read by every block of this grid; the output kernel rewrites it)
  float n[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int d = threadIdx.x + j * 256;
    n[j] = d < p.dk && !fresh ? p.nvec[sh * p.dk + d] : 0.f;
  }
  for (int k = 0; k < nc; ++k) {
    const size_t chh = (size_t)(c0 + k) * p.heads + h;
    const float FL = c.cg[chh * 2], Bm = c.cg[chh * 2 + 1];
    const float m_new = FL + fmaxf(m, Bm);
    const float keep = expf(FL + m - m_new), add = expf(FL + Bm - m_new);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = threadIdx.x + j * 256;
      if (d < p.dk) {
        c.n0[chh * p.dk + d] = n[j];
        n[j] = keep * n[j] + add * c.dn[chh * p.dk + d];
      }
    }
    if (threadIdx.x == 0) c.m0[chh] = m;
    m = m_new;
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int d = threadIdx.x + j * 256;
    if (d < p.dk) p.nvec[sh * p.dk + d] = n[j];
  }
}

// Outputs of one (chunk, head): grid (n_chunks, heads), 320 threads: warp 0 TMA, warp 1 tensor memory + MMA, warps 2..9
// two threads per token.  Shared: Q (2 x 16 KiB), K then P hi (2 x 16 KiB), P lo (2 x 16 KiB), ring of 3 tiles of
// 32 KiB: the slices (128 columns) of the incoming state, hi and lo, then the slices of V, then those of the output gate,
// which the outputs replace in place on their way to a TMA store (a chunk of fewer than 128 tokens stores row by row).
struct McOutSmem {
  static constexpr int Q = 0, K = 2 * MC_KCH, PLO = 4 * MC_KCH, RING = 6 * MC_KCH, TILE = 2 * MC_KCH, NRING = 3;
  static constexpr int TAIL = RING + NRING * TILE;
  static constexpr int BYTES = TAIL + 2304;
};
constexpr int MC_OUT_THREADS = 320;

__global__ void __launch_bounds__(MC_OUT_THREADS, 1)
mlstm_chunk_out_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_v,
                       const __grid_constant__ CUtensorMap tm_s0, const __grid_constant__ CUtensorMap tm_out,
                       const MlstmParams p, const MlstmChunkParams c, const int nk, const int nv) {
  extern __shared__ __align__(1024) uint8_t mc_smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ch = blockIdx.x, h = blockIdx.y;
  if ((smem_u32(mc_smem) & 1023u) != 0) {
    if (tid == 0) atomicCAS(c.status, 0, STATUS_BAD_INDEX);
    return;
  }
  float* s_B = reinterpret_cast<float*>(mc_smem + McOutSmem::TAIL);   // [128] B_s
  float* s_A = s_B + MC_TOK;                                          // [128] F_t - m_t
  float* s_n0 = s_A + MC_TOK;                                         // [128]
  float* s_x = s_n0 + MC_TOK;                                         // [128] exchange (low half -> high half and back)
  float* s_g = s_x + MC_TOK;                                          // [8]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_g + 8);
  uint64_t* qk_full = bars;
  uint64_t* full = bars + 1;                     // [NRING]
  uint64_t* empty = full + McOutSmem::NRING;     // [NRING]
  uint64_t* s_done = empty + McOutSmem::NRING;   // Q K^T complete
  uint64_t* o2_done = s_done + 1;                // Q S0 complete
  uint64_t* p_ready = o2_done + 1;               // P written, O scaled (256 arrivals)
  uint64_t* o_done = p_ready + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  if (tid == 0) {
    mbar_init(qk_full, 1);
    for (int s = 0; s < McOutSmem::NRING; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    mbar_init(s_done, 1);
    mbar_init(o2_done, 1);
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
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + 128;
  const int start = c.c_start[ch], len = c.c_len[ch];
  const size_t chh = (size_t)ch * p.heads + h;
  const int slices = (nv + 1) / 2;
  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      mbar_expect_tx(qk_full, 2 * nk * MC_KCH);
      for (int k = 0; k < nk; ++k) {
        tma_load_3d(mc_smem + McOutSmem::Q + k * MC_KCH, &tm_q, k * 64, h, start, qk_full);
        tma_load_3d(mc_smem + McOutSmem::K + k * MC_KCH, &tm_q, k * 64, p.heads + h, start, qk_full);
      }
      for (int i = 0; i < 4 * slices; ++i) {
        const int st = i % McOutSmem::NRING;
        mbar_wait(&empty[st], ((i / McOutSmem::NRING) & 1) ^ 1, abort_flag, c.status, STATUS_TIMEOUT_STAGE_EMPTY);
        if (*abort_flag) break;
        uint8_t* dst = mc_smem + McOutSmem::RING + st * McOutSmem::TILE;
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
      const uint32_t q_addr = smem_u32(mc_smem + McOutSmem::Q), k_addr = smem_u32(mc_smem + McOutSmem::K);
      const uint32_t plo_addr = smem_u32(mc_smem + McOutSmem::PLO);
      mbar_wait(qk_full, 0, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
      tc_fence_after();
      for (int ks = 0; ks < nk * 4; ++ks) {
        const uint32_t off = (ks / 4) * MC_KCH + (ks % 4) * 32;
        umma_bf16(tmem_s, umma_desc_sw128(q_addr + off), umma_desc_sw128(k_addr + off), umma_idesc_bf16(128, 128), ks > 0 ? 1u : 0u);
      }
      umma_commit(s_done);
      for (int i = 0; i < 3 * slices; ++i) {
        const int st = i % McOutSmem::NRING;
        if (i == 2 * slices) {
          umma_commit(o2_done);
          mbar_wait(p_ready, 0, abort_flag, c.status, STATUS_TIMEOUT_ACCUM);
          tc_fence_after();
        }
        mbar_wait(&full[st], (i / McOutSmem::NRING) & 1, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
        tc_fence_after();
        const uint32_t b_addr = smem_u32(mc_smem + McOutSmem::RING + st * McOutSmem::TILE);
        const bool state = i < 2 * slices;
        const int sl = state ? i / 2 : i - 2 * slices;
        const uint32_t idesc = umma_idesc_bf16_bmn(128, min(2, nv - 2 * sl) * 64);
        const uint32_t d = tmem_o + sl * 128;
        if (state) {
          const uint32_t lbo = nk * 8192;
          for (int ks = 0; ks < nk * 4; ++ks)
            umma_bf16(d, umma_desc_sw128(q_addr + (ks / 4) * MC_KCH + (ks % 4) * 32), umma_desc_mn_sw128(b_addr + ks * 2048, lbo),
                      idesc, (ks > 0 || (i & 1)) ? 1u : 0u);
        } else {
          for (int part = 0; part < 2; ++part) {
            const uint32_t a_addr = part == 0 ? k_addr : plo_addr;
            for (int ks = 0; ks < 8; ++ks)
              umma_bf16(d, umma_desc_sw128(a_addr + (ks / 4) * MC_KCH + (ks % 4) * 32),
                        umma_desc_mn_sw128(b_addr + ks * 2048, MC_KCH), idesc, 1u);
          }
        }
        umma_commit(&empty[st]);
      }
      umma_commit(o_done);
    }
    __syncwarp();
  } else {
    // ---------------- two threads per token ----------------
    const int qd = warp & 3, half = (warp - 2) >> 2;
    const int t = qd * 32 + lane;
    const bool ok = t < len;
    const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
    const float m0 = c.m0[chh];
    {
      const int ct = half * 128 + t;               // index among the 256 threads; tokens are the first 128
      float F, B, Bmax;
      chunk_gates(p.gates, p.heads, h, start, len, p.cap, s_g, ct, F, B, Bmax);
      if (half == 0) {
        s_B[t] = B * MC_LOG2E;
        s_A[t] = -fmaxf(m0, Bmax);                 // F_t - m_t
        s_n0[t] = t < p.dk ? c.n0[chh * p.dk + t] : 0.f;
        s_x[t] = F;
      }
      named_bar_sync(1, 256);
    }
    const float At = s_A[t], At2 = At * MC_LOG2E;
    const float m_t = s_x[t] - At;
    const float a_t = ok ? expf(At + m0) * p.q_scale : 0.f;       // weight of the incoming state, q scaling included
    named_bar_sync(1, 256);                                       // s_x is read; it becomes the exchange buffer
    // n0 . q_t: this thread's 64 dims
    mbar_wait(qk_full, 0, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
    float nq = 0.f;
    if (half < nk) {
      const uint8_t* qr = mc_smem + McOutSmem::Q + half * MC_KCH + t * 128;
#pragma unroll
      for (int piece = 0; piece < 8; ++piece) {
        const uint4 u = *reinterpret_cast<const uint4*>(qr + ((piece ^ (t & 7)) << 4));
        const __nv_bfloat162* q2 = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = __bfloat1622float2(q2[e]);
          nq = fmaf(f.x, s_n0[half * 64 + piece * 8 + 2 * e], nq);
          nq = fmaf(f.y, s_n0[half * 64 + piece * 8 + 2 * e + 1], nq);
        }
      }
    }
    nq *= a_t;
    // P = (q . k) * q_scale * exp(F_t - m_t + B_s) for s <= t: this thread's 64 columns, written over K and beside it
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
          *reinterpret_cast<uint4*>(mc_smem + McOutSmem::K + off) = z;
          *reinterpret_cast<uint4*>(mc_smem + McOutSmem::PLO + off) = z;
        }
        continue;
      }
      tmem_ld32(tmem_s + lane_off + s0, sv);
      tmem_ld_wait();
#pragma unroll
      for (int e = 0; e < 32; e += 4) {
        const float4 b4 = *reinterpret_cast<const float4*>(s_B + s0 + e);
        const float bb[4] = {b4.x, b4.y, b4.z, b4.w};
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          sv[e + u] = ok && s0 + e + u <= t ? sv[e + u] * p.q_scale * ex2_approx(At2 + bb[u]) : 0.f;
          nq += sv[e + u];
        }
      }
#pragma unroll
      for (int v = 0; v < 4; ++v) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split_bf16(sv[v * 8 + 2 * e], sv[v * 8 + 2 * e + 1], hi[e], lo[e]);
        const int off = half * MC_KCH + t * 128 + (((c0 / 8 + v) ^ (t & 7)) << 4);
        *reinterpret_cast<uint4*>(mc_smem + McOutSmem::K + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(mc_smem + McOutSmem::PLO + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    }
    fence_proxy_async_smem();
    // O = a_t * (Q S0): this thread's columns are half, half + 2, ... of the 32-column pieces
    mbar_wait(o2_done, 0, abort_flag, c.status, STATUS_TIMEOUT_ACCUM);
    tc_fence_after();
#pragma unroll 1
    for (int col = half * 32; col < nv * 64; col += 64) {
      float o[32];
      tmem_ld32(tmem_o + lane_off + col, o);
      tmem_ld_wait();
#pragma unroll
      for (int e = 0; e < 32; ++e) o[e] *= a_t;
      tmem_st32(tmem_o + lane_off + col, o);
    }
    tmem_st_wait();
    tc_fence_before();
    mbar_arrive(p_ready);
    // n . q of the token: both halves
    if (half == 1) s_x[t] = nq;
    named_bar_sync(1, 256);
    if (half == 0) { nq += s_x[t]; s_x[t] = nq; }
    named_bar_sync(1, 256);
    nq = s_x[t];
    const float inv = 1.0f / (fmaxf(fabsf(nq), expf(-m_t)) + 1e-6f);
    named_bar_sync(1, 256);
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
    ss = s_x[t] * inv * inv;
    const float r = inv / sqrtf(ss / (float)p.vdim + p.eps);
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(start + t) * p.ld_out + (size_t)h * p.dv;
    const float* nw = p.norm_w + (size_t)h * p.dv;
    const bool whole = len == MC_TOK;
    for (int sl = 0; sl < slices; ++sl) {
      const int i = 3 * slices + sl, st = i % McOutSmem::NRING;
      uint8_t* tile = mc_smem + McOutSmem::RING + st * McOutSmem::TILE;
      mbar_wait(&full[st], (i / McOutSmem::NRING) & 1, abort_flag, c.status, STATUS_TIMEOUT_TMA_FULL);
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
            const float2 w = in ? __ldg(reinterpret_cast<const float2*>(nw + col + v + 2 * e)) : make_float2(0.f, 0.f);
            p2[e] = __floats2bfloat162_rn(__fdividef(o[v + 2 * e] * r * w.x, 1.0f + __expf(-z.x)),
                                          __fdividef(o[v + 2 * e + 1] * r * w.y, 1.0f + __expf(-z.y)));
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
    // the state's running maximum after the portion (the scan reads the old one): its last chunk writes it
    if (half == 0 && t == len - 1) {
      const bool last = ch + 1 == c.n_chunks || p.row[c.c_start[ch + 1]] != p.row[start];
      if (last) p.mval[(size_t)p.row[start] * p.heads + h] = m_t;
    }
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

extern "C" int tahb_mlstm_recurrent(const MlstmParams* p, int f32, cudaStream_t stream) {
  if (p->n_seq <= 0) return 0;
  if (p->dk % 8 || p->dv % 8 || p->dv > MR_MAX_D || p->dk > MR_MAX_D || p->n_seq > 65535) return -2;
  const int nrg = MR_THREADS / (p->dv / 4);
  const size_t smem = ((size_t)3 * p->dk + (size_t)nrg * p->dv + 32) * 4;
  const dim3 grid(p->heads, p->n_seq);
  cudaError_t e = f32 ? launch_chain(mlstm_recurrent_kernel<float>, grid, dim3(MR_THREADS), smem, stream, *p)
                      : launch_chain(mlstm_recurrent_kernel<__nv_bfloat16>, grid, dim3(MR_THREADS), smem, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}

// Chunkwise form: bf16 activations, dk <= 128, dv <= 256.  `n_tokens` = rows of qkvg.
extern "C" int tahb_mlstm_chunks(const MlstmParams* p, const MlstmChunkParams* c, int n_tokens, cudaStream_t stream) {
  if (p->n_seq <= 0 || c->n_chunks <= 0) return 0;
  if (p->dk % 8 || p->dv % 8 || p->dk > 128 || p->dv > 256 || p->n_seq > 65535 || p->heads > 65535 || p->ld_out % 8) return -2;
  const int nk = (p->dk + 63) / 64, nv = (p->dv + 63) / 64;
  auto base = reinterpret_cast<const __nv_bfloat16*>(p->qkvg);
  CUtensorMap mq, mv, ms, mo, md;
  int rc;
  if ((rc = make_head_map(&mq, base, p->dk, 2 * p->heads, n_tokens, p->ld))) return rc;
  if ((rc = make_head_map(&mv, base + (size_t)2 * p->heads * p->dk, p->dv, 2 * p->heads, n_tokens, p->ld))) return rc;
  if ((rc = make_state_map(&ms, c->s0, p->dk, p->dv, (long long)c->n_chunks * p->heads * 2))) return rc;
  if ((rc = make_head_map(&mo, reinterpret_cast<const __nv_bfloat16*>(p->out), p->dv, p->heads, n_tokens, p->ld_out))) return rc;
  if ((rc = make_dS_map(&md, c->dS, p->dk, p->dv, (long long)c->n_chunks * p->heads))) return rc;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(mlstm_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, McStateSmem::BYTES) != cudaSuccess ||
        cudaFuncSetAttribute(mlstm_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, McOutSmem::BYTES) != cudaSuccess)
      return -10;
    configured = true;
  }
  const dim3 grid(c->n_chunks, p->heads);
  mlstm_chunk_state_kernel<<<dim3(c->n_chunks, p->heads, (nv + 1) / 2), 256, McStateSmem::BYTES, stream>>>(mq, mv, md, *p, *c, nv);
  const int blocks = (int)(((long long)p->dk * p->dv / 4 + 255) / 256) + 1;
  mlstm_chunk_scan_kernel<<<dim3(blocks, p->heads, p->n_seq), 256, 0, stream>>>(*p, *c);
  mlstm_chunk_out_kernel<<<grid, MC_OUT_THREADS, McOutSmem::BYTES, stream>>>(mq, mv, ms, mo, *p, *c, nk, nv);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
