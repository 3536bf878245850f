// Real-gated linear recurrent unit over a ragged batch (prompt portions and decode tokens alike), per channel:
//   r = sigmoid(gr + br), i = sigmoid(gi + bi);  log a = -power r softplus(lam);  S <- a S + sqrt(1 - a^2) i u;  out = S gelu_tanh(y)
// gr / gi are the block-diagonal gate products in fp32 (gemm_tc.cu EPI_F32_DIAG): [T, blocks, 2, n].  State fp32 [slots, C]; a request whose cached
// length is zero starts from S = 0 whatever its slot holds.
//
// Prompt portions: the recurrence is linear, so a CTA (32 channels of one request, NW warps) walks the request in tiles of NW * L tokens, warp w
// taking the tile's w-th run of L tokens (a lane is a channel: coalesced rows).  A warp forms a and b = sqrt(1 - a^2) i u of its L tokens in
// registers and their composition (A, H): S_out = A S_in + H; the NW compositions meet in shared memory (two buffers, one barrier per tile), every
// warp folds the ones before it into its own incoming state and runs its L tokens again from there.  The gates' transcendentals, the bulk of the
// work, are thus spread over all warps, and a tile costs 2 L + NW dependent multiply-adds instead of NW * L.  How tiles fall depends on how the
// prompt was cut, which moves results by fp32 rounding only.  Decode: one thread per (request, channel).
//
// bf16 serving evaluates exponentials, reciprocals and the root with the fast instructions (a few 2^-23 relative; one reciprocal serves the two
// gates and the output branch); fp32 serving calls the library functions.  1 - a^2 = -expm1(2 log a) is summed as a series where a is near 1.
#include <stdexcept>

#include "common.cuh"
#include "tma_host.h"

namespace sglb {
namespace {

struct RglruParams {
  const float* gates; const float* bias;       // [T, blocks, 2, n], [blocks, 2, n] or null
  const void* u; int ldu;
  const float* lam;
  const void* y; int ldy;
  float* state;
  const int* req_slots; const int* seq_lens; const int* cu_q;
  void* out;
  int C, n;                                    // channels, channels per block
  float power;
};

template <typename T> __device__ __forceinline__ float rg_ld(const T* p);
template <> __device__ __forceinline__ float rg_ld<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float rg_ld<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void rg_st(T* p, float v);
template <> __device__ __forceinline__ void rg_st<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void rg_st<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ float rg_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// one token of one channel from the gate products (biases br, bi), u and y: a, b = sqrt(1 - a^2) i u, and g = gelu_tanh(y) = y sigmoid(2 z) with
// z = sqrt(2 / pi) (y + 0.044715 y^3).  c = -power softplus(lam): log a = c r.
constexpr float RG_2Z = 1.5957691216057308f;          // 2 sqrt(2 / pi)
constexpr float RG_LOG2E = 1.4426950408889634f;

template <bool FAST>
__device__ __forceinline__ void rg_token(float gr, float br, float gi, float bi, float u, float y, float c, float& a, float& b, float& g) {
  if constexpr (FAST) {
    // sigmoid(x) = 1 / (1 + 2^(-x log2 e)), exponents held below 40 (sigmoid < 1e-12) so that the product of three denominators stays finite
    const float x1 = fmaf(gr, -RG_LOG2E, -RG_LOG2E * br), x2 = fmaf(gi, -RG_LOG2E, -RG_LOG2E * bi);
    const float x3 = y * fmaf(y * y, -RG_LOG2E * RG_2Z * 0.044715f, -RG_LOG2E * RG_2Z);
    const float e1 = 1.f + ex2_approx(fminf(x1, 40.f)), e2 = 1.f + ex2_approx(fminf(x2, 40.f)), e3 = 1.f + ex2_approx(fminf(x3, 40.f));
    const float e12 = e1 * e2, inv = rcp_approx(e12 * e3), inv12 = inv * e3;
    g = y * (e12 * inv);
    const float la = c * (e2 * inv12);               // log a <= 0
    a = ex2_approx(la * RG_LOG2E);
    // 1 - a^2 = -expm1(t), t = 2 log a: the series -t (1 + t/2 (1 + t/3 (1 + t/4))) where a is near 1
    const float t = la + la;
    const float series = -t * fmaf(t * 0.5f, fmaf(t * (1.f / 3.f), fmaf(t, 0.25f, 1.f), 1.f), 1.f);
    const float om = t > -0.06f ? series : fmaf(-a, a, 1.f);
    b = sqrt_approx(om) * (e1 * inv12) * u;
  } else {
    const float r = 1.f / (1.f + expf(-(gr + br))), i = 1.f / (1.f + expf(-(gi + bi)));
    g = y / (1.f + expf(-RG_2Z * (y + 0.044715f * y * y * y)));
    const float la = c * r;
    a = expf(la);
    b = sqrtf(-expm1f(2.f * la)) * i * u;
  }
}

template <typename T, int NW, int L>
__global__ void __launch_bounds__(NW * 32) rglru_scan_kernel(const RglruParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  __shared__ float sA[2][NW][32], sH[2][NW][32];
  const int bq = blockIdx.y;
  const int q0 = p.cu_q ? p.cu_q[bq] : bq;
  const int n = p.cu_q ? p.cu_q[bq + 1] - q0 : 1;
  if (n <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * 32 + lane;
  const bool live = c < p.C;
  const int cc = live ? c : p.C - 1;
  const int blk = cc / p.n, j = cc - blk * p.n;
  const size_t gld = 2 * (size_t)p.C;
  const float* gr = p.gates + (size_t)blk * 2 * p.n + j;
  const float br = p.bias ? p.bias[(size_t)blk * 2 * p.n + j] : 0.f, bi = p.bias ? p.bias[(size_t)blk * 2 * p.n + p.n + j] : 0.f;
  const float cf = -p.power * rg_softplus(p.lam[cc]);
  const T* u = reinterpret_cast<const T*>(p.u) + cc;
  const T* y = reinterpret_cast<const T*>(p.y) + cc;
  T* out = reinterpret_cast<T*>(p.out) + cc;
  float* st = p.state + (size_t)p.req_slots[bq] * p.C + cc;
  float S = p.seq_lens[bq] - n == 0 ? 0.f : *st;          // every warp carries the state at the tile's start
  int buf = 0;
  for (int t0 = 0; t0 < n; t0 += NW * L, buf ^= 1) {
    const int w0 = t0 + warp * L;
    float a[L], b[L], g[L];
    {
      float vr[L], vi[L], vu[L], vy[L];
#pragma unroll
      for (int k = 0; k < L; ++k) {
        const size_t t = (size_t)(q0 + min(w0 + k, n - 1));          // beyond the end: a valid row whose numbers are dropped below
        vr[k] = gr[t * gld];
        vi[k] = gr[t * gld + p.n];
        vu[k] = rg_ld<T>(u + t * p.ldu);
        vy[k] = rg_ld<T>(y + t * p.ldy);
      }
#pragma unroll
      for (int k = 0; k < L; ++k) {
        rg_token<FAST>(vr[k], br, vi[k], bi, vu[k], vy[k], cf, a[k], b[k], g[k]);
        if (w0 + k >= n) { a[k] = 1.f; b[k] = 0.f; }
      }
    }
    float A = a[0], Hs = b[0];
#pragma unroll
    for (int k = 1; k < L; ++k) {
      Hs = a[k] * Hs + b[k];
      A *= a[k];
    }
    sA[buf][warp][lane] = A;
    sH[buf][warp][lane] = Hs;
    __syncthreads();                                      // the other buffer is free again: its readers passed this barrier
    float s = S;
#pragma unroll
    for (int w = 0; w < NW; ++w) {
      if (w == warp) s = S;                               // the state this warp's tokens start from
      S = sA[buf][w][lane] * S + sH[buf][w][lane];
    }
#pragma unroll
    for (int k = 0; k < L; ++k) {
      s = a[k] * s + b[k];
      if (live && w0 + k < n) rg_st<T>(out + (size_t)(q0 + w0 + k) * p.C, s * g[k]);
    }
  }
  if (live && warp == 0) *st = S;
}

// The same with two channels per lane: a half-warp holds 32 channels and is a segment of its own, the two halves of a warp meet by shuffle, the next
// tile's inputs are loaded before the current one is worked on.
template <typename T> struct RgPair;
template <> struct RgPair<float> { typedef float2 raw; };
template <> struct RgPair<__nv_bfloat16> { typedef uint32_t raw; };
__device__ __forceinline__ float2 rg_unpack(float2 v) { return v; }
__device__ __forceinline__ float2 rg_unpack(uint32_t v) { return make_float2(bf16_lo(v), bf16_hi(v)); }
__device__ __forceinline__ void rg_st2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void rg_st2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16(a, b); }

template <typename T, int NW, int L>
__global__ void __launch_bounds__(NW * 32, 512 / (NW * 32)) rglru_scan_pair_kernel(const RglruParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int TILE = 2 * NW * L;
  typedef typename RgPair<T>::raw raw_t;
  __shared__ float4 sT[2][NW][16];                        // (A, H) of a warp's tokens, two channels
  const int bq = blockIdx.y;
  const int q0 = p.cu_q ? p.cu_q[bq] : bq;
  const int n = p.cu_q ? p.cu_q[bq + 1] - q0 : 1;
  if (n <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = lane >> 4, hl = lane & 15;
  const int c = blockIdx.x * 32 + hl * 2;
  const bool live = c < p.C;
  const int cc = live ? c : p.C - 2;
  const int blk = cc / p.n, j = cc - blk * p.n;
  const size_t go = (size_t)blk * 2 * p.n + j, gld = 2 * (size_t)p.C;
  const float2 zero2 = make_float2(0.f, 0.f);
  const float2 br = p.bias ? *reinterpret_cast<const float2*>(p.bias + go) : zero2, bi = p.bias ? *reinterpret_cast<const float2*>(p.bias + go + p.n) : zero2;
  const float cf0 = -p.power * rg_softplus(p.lam[cc]), cf1 = -p.power * rg_softplus(p.lam[cc + 1]);
  const float* gr = p.gates + (size_t)q0 * gld + go;
  const float* gi = gr + p.n;
  const T* u = reinterpret_cast<const T*>(p.u) + (size_t)q0 * p.ldu + cc;
  const T* y = reinterpret_cast<const T*>(p.y) + (size_t)q0 * p.ldy + cc;
  T* out = reinterpret_cast<T*>(p.out) + (size_t)q0 * p.C + cc;
  float* st = p.state + (size_t)p.req_slots[bq] * p.C + cc;
  float2 S = p.seq_lens[bq] - n == 0 ? zero2 : *reinterpret_cast<const float2*>(st);          // every lane carries the state at the tile's start
  const int seg = (warp * 2 + half) * L;
  float2 vr[L], vi[L];
  raw_t vu[L], vy[L];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < L; ++k) {
      const size_t t = (size_t)min(t0 + seg + k, n - 1);          // beyond the end: a valid row whose numbers are dropped below
      vr[k] = *reinterpret_cast<const float2*>(gr + t * gld);
      vi[k] = *reinterpret_cast<const float2*>(gi + t * gld);
      vu[k] = *reinterpret_cast<const raw_t*>(u + t * p.ldu);
      vy[k] = *reinterpret_cast<const raw_t*>(y + t * p.ldy);
    }
  };
  fetch(0);
  int buf = 0;
  for (int t0 = 0; t0 < n; t0 += TILE, buf ^= 1) {
    const int w0 = t0 + seg;
    float2 a[L], b[L], g[L];
    {
      float2 cr[L], ci[L];
      raw_t cu[L], cy[L];
#pragma unroll
      for (int k = 0; k < L; ++k) { cr[k] = vr[k]; ci[k] = vi[k]; cu[k] = vu[k]; cy[k] = vy[k]; }
      if (t0 + TILE < n) fetch(t0 + TILE);
#pragma unroll
      for (int k = 0; k < L; ++k) {
        const float2 uu = rg_unpack(cu[k]), yy = rg_unpack(cy[k]);
        rg_token<FAST>(cr[k].x, br.x, ci[k].x, bi.x, uu.x, yy.x, cf0, a[k].x, b[k].x, g[k].x);
        rg_token<FAST>(cr[k].y, br.y, ci[k].y, bi.y, uu.y, yy.y, cf1, a[k].y, b[k].y, g[k].y);
        if (w0 + k >= n) { a[k] = make_float2(1.f, 1.f); b[k] = zero2; }
      }
    }
    float2 A = a[0], Hs = b[0];
#pragma unroll
    for (int k = 1; k < L; ++k) {
      Hs.x = a[k].x * Hs.x + b[k].x; Hs.y = a[k].y * Hs.y + b[k].y;
      A.x *= a[k].x; A.y *= a[k].y;
    }
    // the lower half's tokens come first: its composition (lo) leads into the upper half's (hi)
    const float oAx = __shfl_xor_sync(0xffffffffu, A.x, 16), oAy = __shfl_xor_sync(0xffffffffu, A.y, 16);
    const float oHx = __shfl_xor_sync(0xffffffffu, Hs.x, 16), oHy = __shfl_xor_sync(0xffffffffu, Hs.y, 16);
    if (half == 0) sT[buf][warp][hl] = make_float4(A.x * oAx, oAx * Hs.x + oHx, A.y * oAy, oAy * Hs.y + oHy);
    __syncthreads();                                      // the other buffer is free again: its readers passed this barrier
    float2 s = S;
#pragma unroll
    for (int w = 0; w < NW; ++w) {
      if (w == warp) s = S;                               // the state this warp's tokens start from
      const float4 t = sT[buf][w][hl];
      S.x = t.x * S.x + t.y;
      S.y = t.z * S.y + t.w;
    }
    if (half) {
      s.x = oAx * s.x + oHx;
      s.y = oAy * s.y + oHy;
    }
#pragma unroll
    for (int k = 0; k < L; ++k) {
      s.x = a[k].x * s.x + b[k].x;
      s.y = a[k].y * s.y + b[k].y;
      if (live && w0 + k < n) rg_st2(out + (size_t)(w0 + k) * p.C, s.x * g[k].x, s.y * g[k].y);
    }
  }
  if (live && warp == 0 && half == 0) *reinterpret_cast<float2*>(st) = S;
}

template <typename T>
__global__ void __launch_bounds__(128) rglru_decode_kernel(const RglruParams p) {
  const int b = blockIdx.y, c = blockIdx.x * 128 + threadIdx.x;
  if (c >= p.C) return;
  const int blk = c / p.n, j = c - blk * p.n;
  const size_t go = (size_t)blk * 2 * p.n + j;
  const float* gr = p.gates + (size_t)b * 2 * p.C + go;
  float* st = p.state + (size_t)p.req_slots[b] * p.C + c;
  const float S = p.seq_lens[b] == 1 ? 0.f : *st;
  float a, x, g;
  rg_token<sizeof(T) == 2>(gr[0], p.bias ? p.bias[go] : 0.f, gr[p.n], p.bias ? p.bias[go + p.n] : 0.f,
                           rg_ld<T>(reinterpret_cast<const T*>(p.u) + (size_t)b * p.ldu + c), rg_ld<T>(reinterpret_cast<const T*>(p.y) + (size_t)b * p.ldy + c),
                           -p.power * rg_softplus(p.lam[c]), a, x, g);
  const float s = a * S + x;
  *st = s;
  rg_st<T>(reinterpret_cast<T*>(p.out) + (size_t)b * p.C + c, s * g);
}

template <typename T>
void launch_rglru(const RglruParams& p, int B, cudaStream_t stream) {
  if (!p.cu_q) {
    rglru_decode_kernel<T><<<dim3((p.C + 127) / 128, B), 128, 0, stream>>>(p);
    SGLB_CUDA_CHECK(cudaGetLastError());
    return;
  }
  dim3 grid((p.C + 31) / 32, B);
  auto al = [](const void* q, size_t n) { return q == nullptr || (uintptr_t)q % n == 0; };
  const bool pairs = p.C % 2 == 0 && p.n % 2 == 0 && p.ldu % 2 == 0 && p.ldy % 2 == 0 && al(p.gates, 8) && al(p.bias, 8) && al(p.state, 8) &&
                     al(p.u, 2 * sizeof(T)) && al(p.y, 2 * sizeof(T)) && al(p.out, 2 * sizeof(T));
  if (!pairs) {
    rglru_scan_kernel<T, 8, 8><<<grid, 256, 0, stream>>>(p);
  } else if ((long long)grid.x * B >= 148) {
    rglru_scan_pair_kernel<T, 8, 4><<<grid, 256, 0, stream>>>(p);
  } else {
    rglru_scan_pair_kernel<T, 16, 4><<<grid, 512, 0, stream>>>(p);          // fewer CTAs than SMs: longer tiles
  }
  SGLB_CUDA_CHECK(cudaGetLastError());
}

}  // namespace

void rglru_scan(const float* gates, const float* bias, const void* u, int ldu, const float* lam, const void* y, int ldy, bool bf16, float* state,
                const int* req_slots, const int* seq_lens, const int* cu_q, int B, int C, int blocks, float power, void* out, cudaStream_t stream) {
  if (B <= 0 || C <= 0) return;
  if (B > 65535 || blocks <= 0 || C % blocks) throw std::runtime_error("sglb rglru_scan: equal blocks, at most 65535 requests");
  RglruParams p;
  p.gates = gates; p.bias = bias; p.u = u; p.ldu = ldu; p.lam = lam; p.y = y; p.ldy = ldy; p.state = state; p.req_slots = req_slots; p.seq_lens = seq_lens;
  p.cu_q = cu_q; p.out = out; p.C = C; p.n = C / blocks; p.power = power;
  if (bf16) launch_rglru<__nv_bfloat16>(p, B, stream);
  else launch_rglru<float>(p, B, stream);
}

}  // namespace sglb
