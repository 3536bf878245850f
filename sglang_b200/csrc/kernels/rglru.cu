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
__device__ __forceinline__ float rg_sqrt_fast(float x) {
  float r;
  asm("sqrt.approx.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

// one token of one channel: a, b = sqrt(1 - a^2) i u, and g = gelu_tanh(y)
template <bool FAST>
__device__ __forceinline__ void rg_token(float gr, float gi, float u, float y, float c, float& a, float& b, float& g) {
  // gelu_tanh(y) = y sigmoid(2 z),  z = sqrt(2 / pi) (y + 0.044715 y^3)
  const float z2 = 1.5957691216057308f * (y + 0.044715f * y * y * y);
  if constexpr (FAST) {
    // sigmoid(x) = 1 / (1 + exp(-x)), arguments held above -28 (sigmoid < 1e-12) so that the product of three denominators stays finite
    const float e1 = 1.f + __expf(-fmaxf(gr, -28.f)), e2 = 1.f + __expf(-fmaxf(gi, -28.f)), e3 = 1.f + __expf(-fmaxf(z2, -28.f));
    const float e12 = e1 * e2, inv = __fdividef(1.f, e12 * e3), inv12 = inv * e3;
    const float r = e2 * inv12, i = e1 * inv12;
    g = y * e12 * inv;
    const float la = c * r;                          // log a <= 0
    a = __expf(la);
    const float t = 2.f * la;
    const float series = -t * (1.f + t * 0.5f * (1.f + t * (1.f / 3.f) * (1.f + t * 0.25f * (1.f + t * 0.2f * (1.f + t * (1.f / 6.f))))));
    const float om = t > -0.25f ? series : 1.f - a * a;
    b = rg_sqrt_fast(om) * i * u;
  } else {
    const float r = 1.f / (1.f + expf(-gr)), i = 1.f / (1.f + expf(-gi));
    g = y / (1.f + expf(-z2));
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
        rg_token<FAST>(vr[k] + br, vi[k] + bi, vu[k], vy[k], cf, a[k], b[k], g[k]);
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
  rg_token<sizeof(T) == 2>(gr[0] + (p.bias ? p.bias[go] : 0.f), gr[p.n] + (p.bias ? p.bias[go + p.n] : 0.f),
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
  } else {
    dim3 grid((p.C + 31) / 32, B);
    if ((long long)grid.x * B >= 296) rglru_scan_kernel<T, 8, 8><<<grid, 256, 0, stream>>>(p);
    else rglru_scan_kernel<T, 16, 8><<<grid, 512, 0, stream>>>(p);          // few CTAs: longer tiles
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
