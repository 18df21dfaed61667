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
#include "common.cuh"

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

// ---------------------------------------------------------------------------------------------
// Recurrent form: grid (heads, n_seq), 256 threads; the tokens of a sequence one after another.  Thread (rg, c) owns the
// float4 column c of the rows rg, rg + nrg, ... of S, read and written in place (one token: the state streams through
// once, which is the whole cost of a decode step).
// ---------------------------------------------------------------------------------------------
constexpr int MR_THREADS = 256;
constexpr int MR_MAX_D = 1024;

template <typename T>
__global__ void __launch_bounds__(MR_THREADS) mlstm_recurrent_kernel(const MlstmParams p) {
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
#pragma unroll 4
      for (int r = rg; r < dk; r += nrg) {
        float4* sp = reinterpret_cast<float4*>(S + (size_t)r * dv) + c;
        float4 a = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *sp;
        const float kr = s_k[r], qr = s_q[r];
        a.x = fmaf(keep, a.x, kr * vv.x); a.y = fmaf(keep, a.y, kr * vv.y);
        a.z = fmaf(keep, a.z, kr * vv.z); a.w = fmaf(keep, a.w, kr * vv.w);
        o.x = fmaf(a.x, qr, o.x); o.y = fmaf(a.y, qr, o.y); o.z = fmaf(a.z, qr, o.z); o.w = fmaf(a.w, qr, o.w);
        *sp = a;
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
