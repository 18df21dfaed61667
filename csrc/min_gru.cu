// minGRU: an elementwise gated recurrence whose gates read the current token only.
//
//   z = sigmoid(zr + zb),  u = xr + xb,  candidate c(u) = u + 1/2 for u >= 0, sigmoid(u) for u < 0
//   S <- (1 - z) S + z c(u),   out = out_scale * S * silu(gr)
//
// zr, xr, gr are columns [z | x | g] of d each of the layer's projection (d padded to a multiple of 8; padding columns of the
// output meet zero weight columns).  The state is one fp32 vector per cache row; a token at position 0 starts from zeros.
// Gates, candidate and recurrence are fp32.
//
//   min_gru_step     one token per row
//   min_gru_scan     portions.  A CTA owns 64 channels of a portion (or of a segment of one) and walks it in tiles of 64 tokens:
//                    every warp composes the 8 affine maps S -> a S + b of its tokens, the warps' compositions meet in shared
//                    memory, and each warp replays its tokens from the state in front of them.  A long portion is cut into
//                    segments: a first launch leaves the composition of every segment, a second one starts each segment from
//                    the state behind those in front of it.
#include "common.cuh"

namespace tahb {

struct MinGruParams {
  const void* proj;           // [n, ld], first column of z
  const float* zb;            // [d]
  const float* xb;
  void* out;                  // [n, ld_out]
  float* S;                   // [rows, d]
  const int* seq_start;       // [n_seq] first token and number of tokens of every portion (scan)
  const int* seq_len;
  const int* pos;             // [n]
  const int* row;             // [n]
  const int* slot;            // [n], negative = idle row (step), or null
  float* ws;                  // [n_seq][n_split][2][d], with n_split > 1
  int n, d, n_split;
  long long ld, ld_out;
  float out_scale;
};

// two elements as they lie in memory
template <typename T> struct Pair2;
template <> struct Pair2<float> { using type = float2; };
template <> struct Pair2<__nv_bfloat16> { using type = __nv_bfloat162; };
__device__ __forceinline__ float2 widen(float2 v) { return v; }
__device__ __forceinline__ float2 widen(__nv_bfloat162 v) { return __bfloat1622float2(v); }

template <typename T> __device__ __forceinline__ float2 load2(const T* p);
template <> __device__ __forceinline__ float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 load2<__nv_bfloat16>(const __nv_bfloat16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

__device__ __forceinline__ float rcp_approx(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
constexpr float MG_LOG2E = 1.4426950408889634f;
// exp(-x), at most 2^40 (a sigmoid stops at 2^-40), so that the product of two of them plus one stays finite
__device__ __forceinline__ float exp_neg(float x) { return ex2_approx(fminf(-x * MG_LOG2E, 40.0f)); }

// The map of a token, S -> a S + b.
template <typename T>
__device__ __forceinline__ void token_map(float z, float u, float& a, float& b) {
  if constexpr (sizeof(T) == 4) {
    a = 1.0f / (1.0f + expf(z));
    b = 1.0f / (1.0f + expf(-z)) * (u >= 0.f ? u + 0.5f : 1.0f / (1.0f + expf(-u)));
  } else {                                       // two sigmoids with one reciprocal
    const float ez = exp_neg(z), eu = exp_neg(u), dz = 1.0f + ez, du = 1.0f + eu;
    const float r = rcp_approx(dz * du), p = r * du;
    a = ez * p;
    b = p * (u >= 0.f ? u + 0.5f : r * dz);
  }
}
template <typename T>
__device__ __forceinline__ float silu_of(float g) {
  return sizeof(T) == 4 ? g / (1.0f + expf(-g)) : g * rcp_approx(1.0f + exp_neg(g));
}

template <typename T>
__global__ void __launch_bounds__(128) min_gru_step_kernel(const MinGruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.y, c = 2 * (blockIdx.x * 128 + threadIdx.x);
  if (c >= p.d || (p.slot != nullptr && p.slot[t] < 0)) return;
  const T* x = reinterpret_cast<const T*>(p.proj) + (size_t)t * p.ld + c;
  const float2 z = load2(x), u = load2(x + p.d), g = load2(x + 2 * p.d);
  const float2 zb = load2(p.zb + c), xb = load2(p.xb + c);
  float* st = p.S + (size_t)p.row[t] * p.d + c;
  float2 S = p.pos[t] == 0 ? make_float2(0.f, 0.f) : load2(st);
  float a, b;
  token_map<T>(z.x + zb.x, u.x + xb.x, a, b);
  S.x = fmaf(a, S.x, b);
  token_map<T>(z.y + zb.y, u.y + xb.y, a, b);
  S.y = fmaf(a, S.y, b);
  store2(st, S.x, S.y);
  store2(reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + c, p.out_scale * S.x * silu_of<T>(g.x), p.out_scale * S.y * silu_of<T>(g.y));
}

constexpr int MG_WARPS = 8, MG_PER = 8, MG_TILE = MG_WARPS * MG_PER, MG_CH = 64;

// Grid (channel blocks, portions, segments).  SUMMARY: only the composition of the segment, to ws.
template <typename T, bool SUMMARY>
__global__ void __launch_bounds__(MG_WARPS * 32, sizeof(T) == 2 ? 2 : 1) min_gru_scan_kernel(const MinGruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float4 s_map[2][MG_WARPS][32];      // (a, b) of two channels
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * MG_CH + 2 * lane, seq = blockIdx.y, seg = blockIdx.z;
  const bool live = c < p.d;
  const int first = p.seq_start[seq], len = p.seq_len[seq];
  const int per = (len + p.n_split * MG_TILE - 1) / (p.n_split * MG_TILE) * MG_TILE;      // tokens of a segment
  const int t_begin = min(len, seg * per), t_end = min(len, t_begin + per);
  float* ws = p.ws + (size_t)seq * p.n_split * 2 * p.d + c;                    // segment s: a at 2 s d, b at (2 s + 1) d
  float* st = p.S + (size_t)p.row[first] * p.d + c;
  const bool fresh = p.pos[first] == 0;
  float2 zb = make_float2(0.f, 0.f), xb = zb, carry = zb, prod = make_float2(1.f, 1.f);
  if (live) {
    zb = load2(p.zb + c);
    xb = load2(p.xb + c);
    if constexpr (SUMMARY) {
      // the slot of the last segment, which no other needs, keeps the state in front of the portion: the last segment of the
      // second launch writes the new one while others may not have started
      if (seg == 0) {
        const float2 S = fresh ? make_float2(0.f, 0.f) : load2(st);
        store2(ws + (size_t)(2 * (p.n_split - 1)) * p.d, S.x, S.y);
      }
    } else if (p.n_split > 1) {
      carry = load2(ws + (size_t)(2 * (p.n_split - 1)) * p.d);
      for (int s = 0; s < seg; ++s) {
        const float2 a = load2(ws + (size_t)(2 * s) * p.d), b = load2(ws + (size_t)(2 * s + 1) * p.d);
        carry.x = fmaf(a.x, carry.x, b.x);
        carry.y = fmaf(a.y, carry.y, b.y);
      }
    } else if (!fresh) {
      carry = load2(st);
    }
  }
  const T* x = reinterpret_cast<const T*>(p.proj) + (size_t)first * p.ld + (live ? c : 0);
  T* out = reinterpret_cast<T*>(p.out) + (size_t)first * p.ld_out + c;
  using Raw = typename Pair2<T>::type;
  Raw zr[MG_PER], ur[MG_PER], gr[MG_PER];        // of the next tile, while the one before is at work
  auto fetch = [&](int t0, int col, Raw* r) {    // unconditional loads, so that all of them are on their way together
#pragma unroll
    for (int k = 0; k < MG_PER; ++k)
      r[k] = *reinterpret_cast<const Raw*>(x + (size_t)min(t0 + warp * MG_PER + k, len - 1) * p.ld + col);
  };
  fetch(t_begin, 0, zr);
  fetch(t_begin, p.d, ur);
  if constexpr (!SUMMARY) fetch(t_begin, 2 * p.d, gr);
  int buf = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += MG_TILE, buf ^= 1) {
    float2 a[MG_PER], b[MG_PER];
    float4 m = make_float4(1.f, 0.f, 1.f, 0.f);
#pragma unroll
    for (int k = 0; k < MG_PER; ++k) {
      const float2 z = widen(zr[k]), u = widen(ur[k]);
      token_map<T>(z.x + zb.x, u.x + xb.x, a[k].x, b[k].x);
      token_map<T>(z.y + zb.y, u.y + xb.y, a[k].y, b[k].y);
      if (t0 + warp * MG_PER + k >= t_end) {     // behind the segment: S stays what it is
        a[k] = make_float2(1.f, 1.f);
        b[k] = make_float2(0.f, 0.f);
      }
      m = make_float4(a[k].x * m.x, fmaf(a[k].x, m.y, b[k].x), a[k].y * m.z, fmaf(a[k].y, m.w, b[k].y));
    }
    s_map[buf][warp][lane] = m;
    if (t0 + MG_TILE < t_end) {
      fetch(t0 + MG_TILE, 0, zr);
      fetch(t0 + MG_TILE, p.d, ur);
    }
    __syncthreads();
    float2 S = carry;
#pragma unroll
    for (int w = 0; w < MG_WARPS; ++w) {
      if (w == warp) S = carry;
      const float4 q = s_map[buf][w][lane];
      carry.x = fmaf(q.x, carry.x, q.y);
      carry.y = fmaf(q.z, carry.y, q.w);
      if constexpr (SUMMARY) {
        prod.x *= q.x;
        prod.y *= q.z;
      }
    }
    if constexpr (!SUMMARY) {
#pragma unroll
      for (int k = 0; k < MG_PER; ++k) {
        const int t = t0 + warp * MG_PER + k;
        const float2 g = widen(gr[k]);
        S.x = fmaf(a[k].x, S.x, b[k].x);
        S.y = fmaf(a[k].y, S.y, b[k].y);
        if (live && t < t_end)
          store2(out + (size_t)t * p.ld_out, p.out_scale * S.x * silu_of<T>(g.x), p.out_scale * S.y * silu_of<T>(g.y));
      }
      if (t0 + MG_TILE < t_end) fetch(t0 + MG_TILE, 2 * p.d, gr);
    }
  }
  if (!live || warp != 0) return;
  if constexpr (SUMMARY) {
    store2(ws + (size_t)(2 * seg) * p.d, prod.x, prod.y);
    store2(ws + (size_t)(2 * seg + 1) * p.d, carry.x, carry.y);
  } else if (seg == p.n_split - 1) {
    store2(st, carry.x, carry.y);
  }
}

static int check_min_gru(const MinGruParams* p) {
  return p->d % 2 || p->d < 2 || p->ld % 2 || p->ld < 3ll * p->d || p->ld_out % 2 || p->n_split < 1 || p->n_split > 64 ? -2 : 0;
}

}  // namespace tahb

using namespace tahb;

// One token per entry.
extern "C" int tahb_min_gru_step(const MinGruParams* p, int f32, cudaStream_t stream) {
  if (p->n <= 0) return 0;
  if (check_min_gru(p) || p->n > 65535) return -2;
  const dim3 grid((p->d + 255) / 256, p->n);
  cudaError_t e = f32 ? launch_chain(min_gru_step_kernel<float>, grid, dim3(128), 0, stream, *p)
                      : launch_chain(min_gru_step_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}

// Portions seq_start / seq_len (n_seq of them); n_split segments each.
extern "C" int tahb_min_gru_scan(const MinGruParams* p, int n_seq, int f32, cudaStream_t stream) {
  if (n_seq <= 0) return 0;
  if (check_min_gru(p) || n_seq > 65535 || (p->n_split > 1 && p->ws == nullptr)) return -2;
  const dim3 block(MG_WARPS * 32);
  const unsigned cb = (p->d + MG_CH - 1) / MG_CH;
  cudaError_t e = cudaSuccess;
  if (p->n_split > 1)
    e = f32 ? launch_chain(min_gru_scan_kernel<float, true>, dim3(cb, n_seq, p->n_split - 1), block, 0, stream, *p)
            : launch_chain(min_gru_scan_kernel<__nv_bfloat16, true>, dim3(cb, n_seq, p->n_split - 1), block, 0, stream, *p);
  if (e != cudaSuccess) return -3;
  e = f32 ? launch_chain(min_gru_scan_kernel<float, false>, dim3(cb, n_seq, p->n_split), block, 0, stream, *p)
          : launch_chain(min_gru_scan_kernel<__nv_bfloat16, false>, dim3(cb, n_seq, p->n_split), block, 0, stream, *p);
  return e == cudaSuccess ? 0 : -3;
}
