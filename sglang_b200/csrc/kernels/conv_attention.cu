// What lies between a q / k / v projection and the attention kernel when the projections run through a short causal convolution over time and
// every head may carry several maps (differential attention has two):
//
//   conv_attention_prepare : projection rows [q (H*M*D) | k (G*M*D) | v (G*Dv)] ->
//     u_t      = sum_j w[c, j] * x_(t - taps + 1 + j)      per channel c; before the portion: the request's rolling state; before the sequence: zeros
//     q, k     <- unit RMS over the D values of every (head, map), times a weight [D]
//     q, k     <- pairs (i, i + half), i < half, turned by position * inv_freq[i]; cosine and sine times rot_mult
//     k row    : head g takes M segments side by side, one per map;  v row: head g
//     q        : [T, H * M, M * segment]: query row h * M + m holds its map in segment m and zeros elsewhere, so that its product with the whole key
//                head is its own map's score: M maps over shared values become M times the query heads of ordinary grouped-query attention
//   A segment is D columns (64 when the heads are laid out 128 wide for the tcgen05 kernels: M = 2; 128 for M = 1), values Dv (or 128).
//
// Mapping: a CTA takes a run of tokens of the flat batch and a share of the units (one unit = a (head, map) of q or k, or a head of v); the
// sines and cosines of the run are computed once into shared memory; a warp walks the run for one unit with its taps' history in registers, so
// a projection row is read once per run (plus the taps before it).  A lane owns column pairs (2 lane, 2 lane + 1) + 64 e.  Decode calls
// (cu_q == nullptr: one token per request) also roll the request's state forward here: a channel is read and written by one lane.  Prompt
// portions roll it in a second launch (mamba.cu causal_conv1d_state), after every run has read the old one.  All math is fp32.
#include <algorithm>
#include <stdexcept>

#include "api.h"
#include "common.cuh"
#include "tma_host.h"

namespace sglb {
namespace {

constexpr int CA_NT = 256;            // 8 warps
constexpr int CA_MAX_N = 256;         // widest head
constexpr int CA_VW = 64;             // columns of a value unit in the four-column kernel

struct ConvPrepParams {
  const void* qkv; int ld;
  int T, H, G, M, D, Dv;
  const void* w; int taps;            // [C, taps]
  void* state;                        // [slots, C, taps - 1]
  const int* positions; const int* cu_q; const int* req_slots; const int* seq_lens; int B;
  const void* qw; const void* kw; float eps;      // null: no norm
  const float* inv_freq; int half; float rot_mult;
  void* kc; void* vc; size_t ldc; const int* loc;
  void* q_out; int seg, wv;           // segment of a map, width of a value head
  int run, units, units_per_cta, vpieces;         // vpieces: value units per head (four-column kernel)
};

template <typename T> __device__ __forceinline__ float ca_ld(const T* p);
template <> __device__ __forceinline__ float ca_ld<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ca_ld<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void ca_st(T* p, float v);
template <> __device__ __forceinline__ void ca_st<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void ca_st<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float2 ca_ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ca_ld2(const __nv_bfloat16* p) {
  const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(bf16_lo(v), bf16_hi(v));
}
__device__ __forceinline__ void ca_st2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void ca_st2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16(a, b); }

// EP: column pairs per lane (64 EP >= head width); KM: taps held in registers (taps <= KM); VEC: every width, stride and base is even
template <typename T, int EP, int KM, bool VEC>
__global__ void __launch_bounds__(CA_NT) conv_attention_prepare_kernel(const ConvPrepParams p) {
  extern __shared__ float sm[];
  float* s_cs = sm;                                         // [run][half][cos, sin]
  float* s_row = sm + (size_t)p.run * p.half * 2;           // [8 warps][64 EP]
  int* s_b = reinterpret_cast<int*>(s_row + 8 * 64 * EP);   // request of the run's first token
  const int t0 = blockIdx.x * p.run, t1 = min(p.T, t0 + p.run);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    int b = t0;
    if (p.cu_q) {                                           // last request that starts at or before t0 (empty ones share a start: take the last)
      int lo = 0, hi = p.B - 1;
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (p.cu_q[mid] <= t0) lo = mid; else hi = mid - 1;
      }
      b = lo;
    }
    *s_b = b;
  }
  for (int i = threadIdx.x; i < (t1 - t0) * p.half; i += CA_NT) {
    const int tt = i / p.half, f = i - tt * p.half;
    float sn, cs;
    sincosf((float)p.positions[t0 + tt] * p.inv_freq[f], &sn, &cs);
    s_cs[2 * i] = cs * p.rot_mult;
    s_cs[2 * i + 1] = sn * p.rot_mult;
  }
  __syncthreads();
  const int K = p.taps, hist_n = K - 1;
  const int C = (p.H + p.G) * p.M * p.D + p.G * p.Dv;
  const T* x = reinterpret_cast<const T*>(p.qkv);
  const T* w = reinterpret_cast<const T*>(p.w);
  T* state = reinterpret_cast<T*>(p.state);
  float* row = s_row + warp * 64 * EP;
  const int u_end = min(p.units, ((int)blockIdx.y + 1) * p.units_per_cta);
  for (int u = blockIdx.y * p.units_per_cta + warp; u < u_end; u += CA_NT / 32) {
    const int nq = p.H * p.M, nk = p.G * p.M;
    const int kind = u < nq ? 0 : u < nq + nk ? 1 : 2;      // q, k, v
    const int n = kind == 2 ? p.Dv : p.D;
    const int c0 = kind == 2 ? (nq + nk) * p.D + (u - nq - nk) * p.Dv : u * p.D;      // first channel (q and k units follow one another)
    const T* nw = reinterpret_cast<const T*>(kind == 0 ? p.qw : p.kw);
    // taps and inputs are right-aligned: slot KM - 1 belongs to the current token, slots below KM - K carry weight zero
    float wt[KM][2 * EP], win[KM][2 * EP];
#pragma unroll
    for (int e = 0; e < EP; ++e)
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        const int i = 2 * lane + 64 * e + s;
#pragma unroll
        for (int j = 0; j < KM; ++j) {
          const int tap = j - (KM - K);
          wt[j][2 * e + s] = (tap >= 0 && i < n) ? ca_ld<T>(w + (size_t)(c0 + i) * K + tap) : 0.f;
          win[j][2 * e + s] = 0.f;
        }
      }
    auto load_row = [&](const T* src, float (&dst)[2 * EP]) {         // src: first channel of the unit in one projection row
#pragma unroll
      for (int e = 0; e < EP; ++e) {
        const int i = 2 * lane + 64 * e;
        if (VEC) {
          const float2 v = i < n ? ca_ld2(src + i) : make_float2(0.f, 0.f);
          dst[2 * e] = v.x; dst[2 * e + 1] = v.y;
        } else {
          dst[2 * e] = i < n ? ca_ld<T>(src + i) : 0.f;
          dst[2 * e + 1] = i + 1 < n ? ca_ld<T>(src + i + 1) : 0.f;
        }
      }
    };
    int b = *s_b, bq0 = 0, bend = 0;
    bool enter = true;
    for (int t = t0; t < t1; ++t) {
      if (p.cu_q) {
        while (b + 1 < p.B && t >= p.cu_q[b + 1]) { ++b; enter = true; }      // tokens behind the last request (padded batches) count to it
      } else if (t > t0) {
        b = t;
        enter = true;
      }
      if (enter) {                                          // first token of this run in request b: gather the inputs before it
        enter = false;
        bq0 = p.cu_q ? p.cu_q[b] : b;
        bend = p.cu_q ? p.cu_q[b + 1] : b + 1;
        const bool fresh = p.seq_lens[b] - (bend - bq0) == 0;
        const T* st = state + ((size_t)p.req_slots[b] * C + c0) * hist_n;
#pragma unroll
        for (int j = 0; j < KM - 1; ++j) {
          const int tt = t - (KM - 1) + j;                  // flat index of the input in slot j
          if (j >= KM - K) {
            if (tt >= bq0) {
              load_row(x + (size_t)tt * p.ld + c0, win[j]);
            } else {
#pragma unroll
              for (int e = 0; e < EP; ++e)
#pragma unroll
                for (int s = 0; s < 2; ++s) {
                  const int i = 2 * lane + 64 * e + s;
                  win[j][2 * e + s] = (!fresh && i < n) ? ca_ld<T>(st + (size_t)i * hist_n + (hist_n + tt - bq0)) : 0.f;
                }
            }
          }
        }
      }
      float y[2 * EP];
      load_row(x + (size_t)t * p.ld + c0, win[KM - 1]);
#pragma unroll
      for (int i = 0; i < 2 * EP; ++i) {
        y[i] = 0.f;
#pragma unroll
        for (int j = 0; j < KM; ++j) y[i] += wt[j][i] * win[j][i];
      }
#pragma unroll
      for (int j = 0; j < KM - 1; ++j)                      // the window moves on
#pragma unroll
        for (int i = 0; i < 2 * EP; ++i) win[j][i] = win[j + 1][i];
      if (p.cu_q == nullptr && hist_n > 0) {
        T* st = state + ((size_t)p.req_slots[b] * C + c0) * hist_n;
#pragma unroll
        for (int j = 0; j < KM - 1; ++j) {
          if (j >= KM - K) {
#pragma unroll
            for (int e = 0; e < EP; ++e)
#pragma unroll
              for (int s = 0; s < 2; ++s) {
                const int i = 2 * lane + 64 * e + s;
                if (i < n) ca_st<T>(st + (size_t)i * hist_n + (j - (KM - K)), win[j][2 * e + s]);
              }
          }
        }
      }
      const size_t slot = (size_t)p.loc[t];
      if (kind < 2) {
        if (nw) {
          float ss = 0.f;
#pragma unroll
          for (int i = 0; i < 2 * EP; ++i) ss += y[i] * y[i];                  // columns >= n are zero
          const float r = 1.0f / sqrtf(warp_sum(ss) / (float)n + p.eps);
#pragma unroll
          for (int e = 0; e < EP; ++e)
#pragma unroll
            for (int s = 0; s < 2; ++s) {
              const int i = 2 * lane + 64 * e + s;
              y[2 * e + s] *= i < n ? r * ca_ld<T>(nw + i) : 0.f;
            }
        }
        if (p.half > 0) {
          __syncwarp();
#pragma unroll
          for (int e = 0; e < EP; ++e) *reinterpret_cast<float2*>(row + 2 * lane + 64 * e) = make_float2(y[2 * e], y[2 * e + 1]);
          __syncwarp();
          const float* cs = s_cs + (size_t)(t - t0) * p.half * 2;
#pragma unroll
          for (int e = 0; e < EP; ++e)
#pragma unroll
            for (int s = 0; s < 2; ++s) {
              const int i = 2 * lane + 64 * e + s;
              if (i < p.half) y[2 * e + s] = y[2 * e + s] * cs[2 * i] - row[i + p.half] * cs[2 * i + 1];
              else if (i < 2 * p.half) y[2 * e + s] = y[2 * e + s] * cs[2 * (i - p.half)] + row[i - p.half] * cs[2 * (i - p.half) + 1];
            }
        }
      }
      // ---- store: the unit's values (zeros up to the segment's end); a query row also gets zeros in the other maps' segments
      T* dst;
      int width, lead = 0;                                  // row of ``width`` columns whose columns lead .. lead + n - 1 are the values
      if (kind == 0) {
        dst = reinterpret_cast<T*>(p.q_out) + ((size_t)t * nq + u) * (p.M * p.seg);
        width = p.M * p.seg;
        lead = (u % p.M) * p.seg;
      } else if (kind == 1) {
        const int uk = u - nq;
        dst = reinterpret_cast<T*>(p.kc) + slot * p.ldc + (size_t)uk * p.seg;
        width = p.seg;
      } else {
        dst = reinterpret_cast<T*>(p.vc) + slot * p.ldc + (size_t)(u - nq - nk) * p.wv;
        width = p.wv;
      }
#pragma unroll
      for (int e = 0; e < EP; ++e) {
        const int i = 2 * lane + 64 * e;
        if (VEC) {
          if (i < n) ca_st2(dst + lead + i, y[2 * e], y[2 * e + 1]);
        } else {
          if (i < n) ca_st<T>(dst + lead + i, y[2 * e]);
          if (i + 1 < n) ca_st<T>(dst + lead + i + 1, y[2 * e + 1]);
        }
      }
      if (VEC) {
        for (int i = 2 * lane; i < width; i += 64)
          if (i < lead || i >= lead + n) ca_st2(dst + i, 0.f, 0.f);
      } else {
        for (int i = lane; i < width; i += 32)
          if (i < lead || i >= lead + n) ca_st<T>(dst + i, 0.f);
      }
    }
  }
}

// four columns of a row
__device__ __forceinline__ void ca_ld4(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void ca_ld4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 a = *reinterpret_cast<const uint2*>(p);
  v[0] = bf16_lo(a.x); v[1] = bf16_hi(a.x); v[2] = bf16_lo(a.y); v[3] = bf16_hi(a.y);
}
__device__ __forceinline__ void ca_st4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void ca_st4(__nv_bfloat16* p, const float (&v)[4]) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3])); }

// The same work for maps at most 64 wide, at most four taps and sizes in multiples of four: a half-warp owns a unit (a (head, map) of q or k, or a
// 64-column piece of a value head), a lane four neighbouring columns; a group of AHEAD tokens that lies in one request convolves straight from
// the loaded rows, with no moves between them, and its norms and rotations run side by side.
template <typename T, int AHEAD>
__global__ void __launch_bounds__(CA_NT) conv_attention_prepare_x4_kernel(const ConvPrepParams p) {
  constexpr int KM = 4;
  extern __shared__ float sm[];
  float* s_cs = sm;                                         // [run][half][cos, sin]
  int* s_loc = reinterpret_cast<int*>(s_cs + (size_t)p.run * p.half * 2);      // [run] cache slots
  int* s_b = s_loc + p.run;                                 // request of the run's first token
  const int t0 = blockIdx.x * p.run, t1 = min(p.T, t0 + p.run);
  const int lane = threadIdx.x & 31, hl = lane & 15, col = 4 * hl;
  if (threadIdx.x == 0) {
    int b = t0;
    if (p.cu_q) {                                           // last request that starts at or before t0
      int lo = 0, hi = p.B - 1;
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (p.cu_q[mid] <= t0) lo = mid; else hi = mid - 1;
      }
      b = lo;
    }
    *s_b = b;
  }
  for (int i = threadIdx.x; i < t1 - t0; i += CA_NT) s_loc[i] = p.loc[t0 + i];
  for (int i = threadIdx.x; i < (t1 - t0) * p.half; i += CA_NT) {
    const int tt = i / p.half, f = i - tt * p.half;
    float sn, cs;
    sincosf((float)p.positions[t0 + tt] * p.inv_freq[f], &sn, &cs);
    s_cs[2 * i] = cs * p.rot_mult;
    s_cs[2 * i + 1] = sn * p.rot_mult;
  }
  __syncthreads();
  const int K = p.taps, hist_n = K - 1;
  const int nq = p.H * p.M, nk = p.G * p.M;
  const int C = (nq + nk) * p.D + p.G * p.Dv;
  const T* w = reinterpret_cast<const T*>(p.w);
  const int u_end = min(p.units, ((int)blockIdx.y + 1) * p.units_per_cta);
  // both halves of a warp walk the same number of rounds; a half without a unit repeats the other's and stores nothing
  for (int ub = blockIdx.y * p.units_per_cta + 2 * (threadIdx.x >> 5); ub < u_end; ub += CA_NT / 16) {
    const bool mine = ub + (lane >> 4) < u_end;
    const int u = mine ? ub + (lane >> 4) : ub;
    const int kind = u < nq ? 0 : u < nq + nk ? 1 : 2;      // q, k, v
    const int vh = kind == 2 ? (u - nq - nk) / p.vpieces : 0, vo = kind == 2 ? ((u - nq - nk) - vh * p.vpieces) * CA_VW : 0;      // value head, first column
    const int n = kind == 2 ? min(CA_VW, p.Dv - vo) : p.D;
    const int c0 = kind == 2 ? (nq + nk) * p.D + vh * p.Dv + vo : u * p.D;
    const bool live = col < n;                              // n is a multiple of four: a lane's columns all count or none
    const T* nw = reinterpret_cast<const T*>(kind == 0 ? p.qw : p.kw);
    // taps right-aligned (slots below KM - K carry weight zero); the KM - 1 inputs before the group, then the group's rows
    float wt[KM][4], seq[KM - 1 + AHEAD][4], nwv[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      nwv[i] = live ? ((kind < 2 && nw) ? ca_ld<T>(nw + col + i) : 1.f) : 0.f;
#pragma unroll
      for (int j = 0; j < KM; ++j) {
        const int tap = j - (KM - K);
        wt[j][i] = (tap >= 0 && live) ? ca_ld<T>(w + (size_t)(c0 + col + i) * K + tap) : 0.f;
      }
    }
#pragma unroll
    for (int j = 0; j < KM - 1 + AHEAD; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) seq[j][i] = 0.f;
    const T* x = reinterpret_cast<const T*>(p.qkv) + c0 + col;
    T* dst;                                                 // where token t0's (q) or slot 0's (k, v) columns go; lead: columns before the values
    int width, lead = 0;
    size_t step;
    if (kind == 0) {
      width = p.M * p.seg; lead = (u % p.M) * p.seg; step = (size_t)nq * width;
      dst = reinterpret_cast<T*>(p.q_out) + ((size_t)t0 * nq + u) * width;
    } else if (kind == 1) {
      width = p.seg; step = p.ldc;
      dst = reinterpret_cast<T*>(p.kc) + (size_t)(u - nq) * p.seg;
    } else {                                                // a head's last piece also writes the zeros behind the values
      width = vo + CA_VW >= p.Dv ? p.wv - vo : n; step = p.ldc;
      dst = reinterpret_cast<T*>(p.vc) + (size_t)vh * p.wv + vo;
    }
    const bool rot = kind < 2 && col < 2 * p.half;
    const bool first = col < p.half;                        // half is a multiple of four: partners sit half / 4 lanes apart
    const int partner = (lane & 16) | ((first ? hl + (p.half >> 2) : hl - (p.half >> 2)) & 15);
    const float sg = first ? -1.f : 1.f;
    int b = *s_b, bend = -1;                                // request at hand and its end (none yet)
    for (int tg = t0; tg < t1; tg += AHEAD) {
      if (live) {
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) ca_ld4(x + (size_t)min(tg + g, t1 - 1) * p.ld, seq[KM - 1 + g]);
      }
      float y[AHEAD][4];
      if (min(tg + AHEAD, t1) <= bend) {                    // the whole group continues the request at hand
#pragma unroll
        for (int g = 0; g < AHEAD; ++g)
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < KM; ++j) acc += wt[j][i] * seq[g + j][i];
            y[g][i] = acc;
          }
      } else {                                              // a request begins in the group: token by token, the inputs before it gathered anew
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) {
          const int t = tg + g;
          if (t < t1 && t >= bend) {
            if (p.cu_q) {
              while (b + 1 < p.B && t >= p.cu_q[b + 1]) ++b;          // tokens behind the last request (padded batches) count to it
            } else {
              b = t;
            }
            const int bq0 = p.cu_q ? p.cu_q[b] : b, bq1 = p.cu_q ? p.cu_q[b + 1] : b + 1;
            bend = b + 1 < p.B ? bq1 : 0x7fffffff;
            const bool fresh = p.seq_lens[b] - (bq1 - bq0) == 0;
            const T* st = reinterpret_cast<const T*>(p.state) + ((size_t)p.req_slots[b] * C + c0 + col) * hist_n;
#pragma unroll
            for (int j = 0; j < KM - 1; ++j) {
              const int tt = t - (KM - 1) + j;              // flat index of the input in slot j
              if (j >= KM - K && live) {
                if (tt >= bq0) {
                  ca_ld4(x + (size_t)tt * p.ld, seq[g + j]);
                } else {
#pragma unroll
                  for (int i = 0; i < 4; ++i) seq[g + j][i] = fresh ? 0.f : ca_ld<T>(st + (size_t)i * hist_n + (hist_n + tt - bq0));
                }
              }
            }
          }
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < KM; ++j) acc += wt[j][i] * seq[g + j][i];
            y[g][i] = acc;
          }
          if (p.cu_q == nullptr && hist_n > 0 && t < t1 && live && mine) {
            T* st = reinterpret_cast<T*>(p.state) + ((size_t)p.req_slots[b] * C + c0 + col) * hist_n;
#pragma unroll
            for (int j = 1; j < KM; ++j)
              if (j >= KM - hist_n) {
#pragma unroll
                for (int i = 0; i < 4; ++i) ca_st<T>(st + (size_t)i * hist_n + (j - (KM - hist_n)), seq[g + j][i]);
              }
          }
        }
      }
      if (p.qw) {                                           // unit RMS (the value units' sums go unused)
        float ss[AHEAD];
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) ss[g] = y[g][0] * y[g][0] + y[g][1] * y[g][1] + y[g][2] * y[g][2] + y[g][3] * y[g][3];
#pragma unroll
        for (int o = 8; o > 0; o >>= 1)
#pragma unroll
          for (int g = 0; g < AHEAD; ++g) ss[g] += __shfl_xor_sync(0xffffffffu, ss[g], o);
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) {
          const float r = kind < 2 ? 1.0f / sqrtf(ss[g] / (float)n + p.eps) : 1.f;
#pragma unroll
          for (int i = 0; i < 4; ++i) y[g][i] *= r * nwv[i];
        }
      }
      if (p.half > 0) {
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) {
          float o[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) o[i] = __shfl_sync(0xffffffffu, y[g][i], partner);
          if (rot) {
            const float* cs = s_cs + (size_t)min(tg + g - t0, t1 - t0 - 1) * p.half * 2 + 2 * (first ? col : col - p.half);
            const float4 a = *reinterpret_cast<const float4*>(cs), c = *reinterpret_cast<const float4*>(cs + 4);          // cos, sin of four angles
            y[g][0] = y[g][0] * a.x + sg * o[0] * a.y;
            y[g][1] = y[g][1] * a.z + sg * o[1] * a.w;
            y[g][2] = y[g][2] * c.x + sg * o[2] * c.y;
            y[g][3] = y[g][3] * c.z + sg * o[3] * c.w;
          }
        }
      }
#pragma unroll
      for (int g = 0; g < AHEAD; ++g) {
        if (tg + g < t1 && mine) {
          T* d = dst + (size_t)(kind == 0 ? tg + g - t0 : s_loc[tg + g - t0]) * step;
          if (live) ca_st4(d + lead + col, y[g]);
          const float zero[4] = {0.f, 0.f, 0.f, 0.f};
          for (int i = col; i < width; i += 64)
            if (i < lead || i >= lead + n) ca_st4(d + i, zero);
        }
      }
#pragma unroll
      for (int j = 0; j < KM - 1; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) seq[j][i] = seq[j + AHEAD][i];
    }
  }
}

template <typename T, int EP, int KM>
void launch_prep(const ConvPrepParams& p, bool vec, dim3 grid, size_t smem, cudaStream_t stream) {
  auto go = [&](auto kern) {
    if (smem > 48 * 1024) SGLB_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kern<<<grid, CA_NT, smem, stream>>>(p);
  };
  if (vec) go(conv_attention_prepare_kernel<T, EP, KM, true>);
  else go(conv_attention_prepare_kernel<T, EP, KM, false>);
}

template <typename T>
void dispatch_prep(const ConvPrepParams& p, bool vec, dim3 grid, size_t smem, cudaStream_t stream) {
  const int n = std::max(p.D, p.Dv);
  const bool few = p.taps <= 4;
  if (n <= 64) { if (few) launch_prep<T, 1, 4>(p, vec, grid, smem, stream); else launch_prep<T, 1, 16>(p, vec, grid, smem, stream); }
  else if (n <= 128) { if (few) launch_prep<T, 2, 4>(p, vec, grid, smem, stream); else launch_prep<T, 2, 16>(p, vec, grid, smem, stream); }
  else { if (few) launch_prep<T, 4, 4>(p, vec, grid, smem, stream); else launch_prep<T, 4, 16>(p, vec, grid, smem, stream); }
}

}  // namespace

void conv_attention_prepare(const void* qkv, int ld, bool bf16, int T, int H, int G, int M, int D, int Dv, const void* conv_w, int taps, void* conv_state,
                            const int* positions, const int* cu_q, const int* req_slots, const int* seq_lens, int B, const void* q_norm_w,
                            const void* k_norm_w, float eps, const float* inv_freq, int half, float rot_mult, void* kc, void* vc, size_t ldc,
                            const int* loc, void* q_out, int pad, int num_sms, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return;
  if (D > CA_MAX_N || Dv > CA_MAX_N || taps < 1 || taps > 16) throw std::runtime_error("sglb conv_attention_prepare: heads up to 256 wide, 1 to 16 taps");
  if (pad > 0 && (pad % M || D > pad / M || Dv > pad)) throw std::runtime_error("sglb conv_attention_prepare: heads do not fit the padded layout");
  ConvPrepParams p;
  p.qkv = qkv; p.ld = ld; p.T = T; p.H = H; p.G = G; p.M = M; p.D = D; p.Dv = Dv; p.w = conv_w; p.taps = taps; p.state = conv_state;
  p.positions = positions; p.cu_q = cu_q; p.req_slots = req_slots; p.seq_lens = seq_lens; p.B = B; p.qw = q_norm_w; p.kw = k_norm_w; p.eps = eps;
  p.inv_freq = inv_freq; p.half = inv_freq ? half : 0; p.rot_mult = rot_mult; p.kc = kc; p.vc = vc; p.ldc = ldc; p.loc = loc; p.q_out = q_out;
  p.seg = pad > 0 ? pad / M : D; p.wv = pad > 0 ? pad : Dv;
  const size_t a2 = bf16 ? 4 : 8;
  auto al = [&](const void* q, size_t n) { return ((uintptr_t)q % n) == 0; };
  auto even = [&](int k) {                                  // every width and stride a multiple of k elements, every base aligned to as much
    const size_t n = a2 * k / 2;
    return D % k == 0 && Dv % k == 0 && ld % k == 0 && ldc % k == 0 && p.seg % k == 0 && p.wv % k == 0 && al(qkv, n) && al(kc, n) && al(vc, n) && al(q_out, n);
  };
  const bool x4 = D <= 64 && taps <= 4 && p.half % 4 == 0 && even(4);
  p.vpieces = x4 ? (Dv + CA_VW - 1) / CA_VW : 1;
  p.units = (H + G) * M + G * p.vpieces;
  // few tokens: one per CTA and the units spread over many CTAs; long batches: runs of tokens, all the history reads amortised
  p.run = cu_q == nullptr ? 1 : T >= 16 * num_sms ? 32 : T >= 4 * num_sms ? 16 : 4;
  const int cols = (T + p.run - 1) / p.run, step = x4 ? 16 : 8;          // units a CTA walks at once
  int ys = std::max(1, std::min((p.units + step - 1) / step, (4 * num_sms + cols - 1) / cols));
  p.units_per_cta = ((p.units + ys - 1) / ys + step - 1) / step * step;
  ys = (p.units + p.units_per_cta - 1) / p.units_per_cta;
  dim3 grid(cols, ys);
  if (x4) {
    const size_t smem = sizeof(float) * (size_t)p.run * p.half * 2 + sizeof(int) * (p.run + 4);      // at most 17 KB
    if (cu_q == nullptr) {
      if (bf16) conv_attention_prepare_x4_kernel<__nv_bfloat16, 1><<<grid, CA_NT, smem, stream>>>(p);
      else conv_attention_prepare_x4_kernel<float, 1><<<grid, CA_NT, smem, stream>>>(p);
    } else {
      if (bf16) conv_attention_prepare_x4_kernel<__nv_bfloat16, 4><<<grid, CA_NT, smem, stream>>>(p);
      else conv_attention_prepare_x4_kernel<float, 4><<<grid, CA_NT, smem, stream>>>(p);
    }
  } else {
    const int n = std::max(D, Dv), ep = n <= 64 ? 1 : n <= 128 ? 2 : 4;
    const size_t smem = sizeof(float) * ((size_t)p.run * p.half * 2 + 8 * 64 * ep) + sizeof(int) * 4;
    if (bf16) dispatch_prep<__nv_bfloat16>(p, even(2), grid, smem, stream);
    else dispatch_prep<float>(p, even(2), grid, smem, stream);
  }
  SGLB_CUDA_CHECK(cudaGetLastError());
  if (cu_q != nullptr) causal_conv1d_state(qkv, ld, conv_state, cu_q, req_slots, seq_lens, B, (H + G) * M * D + G * Dv, taps, bf16, stream);
}

}  // namespace sglb
