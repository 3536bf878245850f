// fp32 residual stream helpers.
//
//   add_rmsnorm_f32 : residual (fp32, in place) += delta (bf16 | fp32 | none); out = residual / rms(residual) * (w | 1 + w) in bf16 | fp32.
//                     One block per row; the sum, the mean of squares and the scaling are fp32, eps sits inside the root.  The weight is a
//                     vector or one number for all coordinates.
//   stream_mix_norm : several parallel fp32 streams instead of one (hyper-connections): mixing, the update and the next sublayer's normed input.
//   clamped_glu     : [gate | up] halves -> min(g, limit) * sigmoid(alpha * g) * (clamp(u, -limit, limit) + 1), fp32 math.
#include <stdexcept>

#include "common.cuh"
#include "tma_host.h"

namespace sglb {
namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void stf(T* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <typename TD, typename TO>
__global__ void __launch_bounds__(256) add_rmsnorm_f32_kernel(float* __restrict__ res, const TD* __restrict__ delta, const TO* __restrict__ w,
                                                              TO* __restrict__ out, int H, float eps, int zero_centred, int ws) {
  __shared__ float red[8];
  __shared__ float s_rs;
  float* r = res + (size_t)blockIdx.x * H;
  const TD* d = delta ? delta + (size_t)blockIdx.x * H : nullptr;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    float v = r[i];
    if (d) {
      v += ldf<TD>(d + i);
      r[i] = v;
    }
    ss += v * v;
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  if (threadIdx.x < 32) {
    float t = threadIdx.x < 8 ? red[threadIdx.x] : 0.f;
    t = warp_sum(t);
    if (threadIdx.x == 0) s_rs = 1.0f / sqrtf(t / (float)H + eps);
  }
  __syncthreads();
  const float rs = s_rs;
  TO* o = out + (size_t)blockIdx.x * H;
  for (int i = threadIdx.x; i < H; i += 256) {          // each thread re-reads exactly the elements it wrote
    float wv = ldf<TO>(w + i * ws);                   // ws = 0: one gain for all coordinates
    if (zero_centred) wv += 1.f;
    stf<TO>(o + i, r[i] * rs * wv);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const T* __restrict__ gu, T* __restrict__ out, int I, float limit, float alpha) {
  const T* row = gu + (size_t)blockIdx.x * 2 * I;
  const int i = blockIdx.y * 256 + threadIdx.x;
  if (i >= I) return;
  const float g = fminf(ldf<T>(row + i), limit);
  const float u = fminf(fmaxf(ldf<T>(row + I + i), -limit), limit);
  stf<T>(out + (size_t)blockIdx.x * I + i, g / (1.f + expf(-alpha * g)) * (u + 1.f));
}

// 16-byte lanes: 8 bf16 gate values and the 8 matching up values per thread
__global__ void __launch_bounds__(256) clamped_glu_bf16x8_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out, int I,
                                                                 float limit, float alpha) {
  const int i = (blockIdx.y * 256 + threadIdx.x) * 8;
  if (i >= I) return;
  const __nv_bfloat16* row = gu + (size_t)blockIdx.x * 2 * I;
  const U4 g = ldg128(row + i), u = ldg128(row + I + i);
  const uint32_t gw[4] = {g.x, g.y, g.z, g.w}, uw[4] = {u.x, u.y, u.z, u.w};
  uint32_t o[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float g0 = fminf(bf16_lo(gw[k]), limit), g1 = fminf(bf16_hi(gw[k]), limit);
    const float u0 = fminf(fmaxf(bf16_lo(uw[k]), -limit), limit), u1 = fminf(fmaxf(bf16_hi(uw[k]), -limit), limit);
    o[k] = pack_bf16(g0 / (1.f + __expf(-alpha * g0)) * (u0 + 1.f), g1 / (1.f + __expf(-alpha * g1)) * (u1 + 1.f));
  }
  st128(out + (size_t)blockIdx.x * I + i, U4{o[0], o[1], o[2], o[3]});
}

// block-wide sum for 256 threads (every thread gets the total)
__device__ __forceinline__ float block_sum_256(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();                       // red may still be read from an earlier call
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) t += red[i];
  return t;
}

// residual += rmsnorm(delta) * (1 + post_w);  out = rmsnorm(residual) * (1 + w): the post-norm of a branch, the residual add and the next
// pre-norm of a sandwich-normed block in one pass over the row.  ``one`` = 1 for weights stored around zero, 0 for plain weights; a weight
// stride of 0 means one gain for all coordinates.
template <typename TD, typename TO>
__global__ void __launch_bounds__(256) postnorm_add_rmsnorm_f32_kernel(float* __restrict__ res, const TD* __restrict__ delta, const TO* __restrict__ post_w,
                                                                       const TO* __restrict__ w, TO* __restrict__ out, int H, float eps, float one,
                                                                       int wsp, int ws) {
  __shared__ float red[8];
  float* r = res + (size_t)blockIdx.x * H;
  const TD* d = delta + (size_t)blockIdx.x * H;
  float sd = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    const float v = ldf<TD>(d + i);
    sd += v * v;
  }
  const float rd = 1.0f / sqrtf(block_sum_256(sd, red) / (float)H + eps);
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    const float v = r[i] + ldf<TD>(d + i) * rd * (one + ldf<TO>(post_w + i * wsp));
    r[i] = v;
    ss += v * v;
  }
  const float rs = 1.0f / sqrtf(block_sum_256(ss, red) / (float)H + eps);
  TO* o = out + (size_t)blockIdx.x * H;
  for (int i = threadIdx.x; i < H; i += 256) stf<TO>(o + i, r[i] * rs * (one + ldf<TO>(w + i * ws)));      // each thread re-reads what it wrote
}


// residual += d1 + d2 + d3 (each optional; d1 / d2 in the model dtype, d3 fp32; the deltas are summed first);  out1 = rmsnorm(residual) * (one + w1),
// out2 likewise under w2 (optional): the residual update of a block whose two branches read the same input, with both pre-norms of the next
// block, in one pass over the row.  Four columns per access; a thread keeps up to four accesses of the row in registers.
template <typename T> __device__ __forceinline__ float4 ld4f(const T* p);
template <> __device__ __forceinline__ float4 ld4f<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 ld4f<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
template <typename T> __device__ __forceinline__ void st4f(T* p, float4 v);
template <> __device__ __forceinline__ void st4f<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void st4f<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

template <typename TD, typename TO, int VEC>
__global__ void __launch_bounds__(256) parallel_add_rmsnorm_f32_kernel(float* __restrict__ res, const TD* __restrict__ d1, const TD* __restrict__ d2,
                                                                       const float* __restrict__ d3, const TO* __restrict__ w1, const TO* __restrict__ w2,
                                                                       TO* __restrict__ out1, TO* __restrict__ out2, int H, float eps, float one) {
  __shared__ float red[8];
  const size_t off = (size_t)blockIdx.x * H;
  float* r = res + off;
  const bool any = d1 || d2 || d3;
  float ss = 0.f;
  if constexpr (VEC == 4) {
    constexpr int KEEP = 4;
    float4 keep[KEEP];
    const int n4 = H >> 2;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = (threadIdx.x + k * 256) * 4;
      keep[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < H) {
        float4 v = *reinterpret_cast<const float4*>(r + i);
        if (any) {
          float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
          if (d1) { const float4 t = ld4f<TD>(d1 + off + i); d.x += t.x; d.y += t.y; d.z += t.z; d.w += t.w; }
          if (d2) { const float4 t = ld4f<TD>(d2 + off + i); d.x += t.x; d.y += t.y; d.z += t.z; d.w += t.w; }
          if (d3) { const float4 t = *reinterpret_cast<const float4*>(d3 + off + i); d.x += t.x; d.y += t.y; d.z += t.z; d.w += t.w; }
          v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w;
          *reinterpret_cast<float4*>(r + i) = v;
        }
        keep[k] = v;
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      }
    }
    for (int c = threadIdx.x + KEEP * 256; c < n4; c += 256) {          // rows wider than 4096: the rest is read again below
      const int i = c * 4;
      float4 v = *reinterpret_cast<const float4*>(r + i);
      if (any) {
        float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d1) { const float4 t = ld4f<TD>(d1 + off + i); d.x += t.x; d.y += t.y; d.z += t.z; d.w += t.w; }
        if (d2) { const float4 t = ld4f<TD>(d2 + off + i); d.x += t.x; d.y += t.y; d.z += t.z; d.w += t.w; }
        if (d3) { const float4 t = *reinterpret_cast<const float4*>(d3 + off + i); d.x += t.x; d.y += t.y; d.z += t.z; d.w += t.w; }
        v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w;
        *reinterpret_cast<float4*>(r + i) = v;
      }
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float rs = 1.0f / sqrtf(block_sum_256(ss, red) / (float)H + eps);
    auto emit = [&](int i, float4 v) {
      const float4 a = ld4f<TO>(w1 + i);
      st4f<TO>(out1 + off + i, make_float4(v.x * rs * (one + a.x), v.y * rs * (one + a.y), v.z * rs * (one + a.z), v.w * rs * (one + a.w)));
      if (out2) {
        const float4 b = ld4f<TO>(w2 + i);
        st4f<TO>(out2 + off + i, make_float4(v.x * rs * (one + b.x), v.y * rs * (one + b.y), v.z * rs * (one + b.z), v.w * rs * (one + b.w)));
      }
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = (threadIdx.x + k * 256) * 4;
      if (i < H) emit(i, keep[k]);
    }
    for (int c = threadIdx.x + KEEP * 256; c < n4; c += 256) emit(c * 4, *reinterpret_cast<const float4*>(r + c * 4));      // each thread re-reads what it wrote
  } else {
    for (int i = threadIdx.x; i < H; i += 256) {
      float v = r[i];
      if (any) {
        float d = 0.f;
        if (d1) d += ldf<TD>(d1 + off + i);
        if (d2) d += ldf<TD>(d2 + off + i);
        if (d3) d += d3[off + i];
        v += d;
        r[i] = v;
      }
      ss += v * v;
    }
    const float rs = 1.0f / sqrtf(block_sum_256(ss, red) / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += 256) {          // each thread re-reads exactly the elements it wrote
      const float y = r[i] * rs;
      stf<TO>(out1 + off + i, y * (one + ldf<TO>(w1 + i)));
      if (out2) stf<TO>(out2 + off + i, y * (one + ldf<TO>(w2 + i)));
    }
  }
}

// x += rmsnorm(src) * (one + w), or x = ... when ``ids`` picks the source row from a table (embedding);  out = x in TO (optional): the residual update
// of a block that norms a sublayer's output only, so that the next sublayer reads the stream itself.  VEC = 4: four columns per access, up to four
// accesses of the row in registers.
template <typename TS, typename TO, int VEC>
__global__ void __launch_bounds__(256) norm_add_f32_kernel(float* __restrict__ x, const TS* __restrict__ src, const int* __restrict__ ids, int rows,
                                                           const TO* __restrict__ w, TO* __restrict__ out, int H, float eps, float one) {
  __shared__ float red[8];
  const size_t off = (size_t)blockIdx.x * H;
  const TS* s = ids ? src + (size_t)min(max(ids[blockIdx.x], 0), rows - 1) * H : src + off;
  float ss = 0.f;
  if constexpr (VEC == 4) {
    constexpr int KEEP = 4;
    float4 keep[KEEP];
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = (threadIdx.x + k * 256) * 4;
      keep[k] = i < H ? ld4f<TS>(s + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += keep[k].x * keep[k].x + keep[k].y * keep[k].y + keep[k].z * keep[k].z + keep[k].w * keep[k].w;
    }
    for (int i = (threadIdx.x + KEEP * 256) * 4; i < H; i += 1024) {          // rows wider than 4096: the rest is read again below
      const float4 v = ld4f<TS>(s + i);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float rs = 1.0f / sqrtf(block_sum_256(ss, red) / (float)H + eps);
    auto emit = [&](int i, float4 v) {
      const float4 a = ld4f<TO>(w + i);
      float4 r = ids ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(x + off + i);
      r.x += v.x * rs * (one + a.x); r.y += v.y * rs * (one + a.y); r.z += v.z * rs * (one + a.z); r.w += v.w * rs * (one + a.w);
      *reinterpret_cast<float4*>(x + off + i) = r;
      if (out) st4f<TO>(out + off + i, r);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = (threadIdx.x + k * 256) * 4;
      if (i < H) emit(i, keep[k]);
    }
    for (int i = (threadIdx.x + KEEP * 256) * 4; i < H; i += 1024) emit(i, ld4f<TS>(s + i));
  } else {
    for (int i = threadIdx.x; i < H; i += 256) { const float v = ldf<TS>(s + i); ss += v * v; }
    const float rs = 1.0f / sqrtf(block_sum_256(ss, red) / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += 256) {
      const float r = (ids ? 0.f : x[off + i]) + ldf<TS>(s + i) * rs * (one + ldf<TO>(w + i));
      x[off + i] = r;
      if (out) stf<TO>(out + off + i, r);
    }
  }
}

// gate activations of grouped_rmsnorm; bf16 gates take the fast exponential and reciprocal (a few 2^-23 relative)
template <typename TO>
__device__ __forceinline__ float gate_act(float g, int silu) {
  const float s = sizeof(TO) == 2 ? __fdividef(1.f, 1.f + __expf(-g)) : 1.f / (1.f + expf(-g));
  return silu ? g * s : s;
}

// x fp32 [T, C] in ``groups`` equal parts: part / sqrt(mean(part^2) + eps) [* w] [* sigmoid(gate) | * silu(gate)] * out_scale; grid (T, groups); gate and
// out are rows of ldg / ldo elements
template <typename TO>
__global__ void __launch_bounds__(256) grouped_rmsnorm_kernel(const float* __restrict__ x, const TO* __restrict__ w, TO* __restrict__ out, int C, int per,
                                                              float eps, const TO* __restrict__ gate, int ldg, int ldo, float out_scale, int silu) {
  __shared__ float red[8];
  const size_t base = (size_t)blockIdx.x * C + (size_t)blockIdx.y * per;
  float ss = 0.f;
  for (int i = threadIdx.x; i < per; i += 256) {
    const float v = x[base + i];
    ss += v * v;
  }
  const float rs = 1.0f / sqrtf(block_sum_256(ss, red) / (float)per + eps) * out_scale;
  const int c0 = blockIdx.y * per;
  TO* o = out + (size_t)blockIdx.x * ldo + c0;
  const TO* gr = gate ? gate + (size_t)blockIdx.x * ldg + c0 : nullptr;
  for (int i = threadIdx.x; i < per; i += 256) {
    float v = x[base + i] * rs;
    if (w) v *= ldf<TO>(w + c0 + i);
    if (gr) v *= gate_act<TO>(ldf<TO>(gr + i), silu);
    stf<TO>(o + i, v);
  }
}

// the same with one warp per (row, part): a CTA of 8 warps walks the parts of its row (many small parts: no CTA-wide barrier, four columns per
// access); a part of up to KEEP * 128 columns stays in registers between the two passes
template <typename TO, int KEEP>
__global__ void __launch_bounds__(256) grouped_rmsnorm_warp_kernel(const float* __restrict__ x, const TO* __restrict__ w, TO* __restrict__ out, int C,
                                                                   int per, int groups, float eps, const TO* __restrict__ gate, int ldg, int ldo,
                                                                   float out_scale, int silu) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n4 = per / 4;
  for (int g = warp; g < groups; g += 8) {
    const float4* xv = reinterpret_cast<const float4*>(x + (size_t)blockIdx.x * C + (size_t)g * per);
    const size_t c0 = (size_t)g * per;
    const TO* gr = gate ? gate + (size_t)blockIdx.x * ldg + c0 : nullptr;
    float4 keep[KEEP], gk[KEEP];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = lane + k * 32;
      gk[k] = gr && i < n4 ? ld4f<TO>(gr + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
      keep[k] = i < n4 ? xv[i] : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += keep[k].x * keep[k].x + keep[k].y * keep[k].y + keep[k].z * keep[k].z + keep[k].w * keep[k].w;
    }
    for (int i = lane + KEEP * 32; i < n4; i += 32) {
      const float4 v = xv[i];
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)per + eps) * out_scale;
    auto emit = [&](int i, float4 v, float4 a) {
      v.x *= rs; v.y *= rs; v.z *= rs; v.w *= rs;
      if (w) {
        const float4 ww = ld4f<TO>(w + c0 + 4 * i);
        v.x *= ww.x; v.y *= ww.y; v.z *= ww.z; v.w *= ww.w;
      }
      if (gr) {
        v.x *= gate_act<TO>(a.x, silu); v.y *= gate_act<TO>(a.y, silu); v.z *= gate_act<TO>(a.z, silu); v.w *= gate_act<TO>(a.w, silu);
      }
      st4f<TO>(out + (size_t)blockIdx.x * ldo + c0 + 4 * i, v);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int i = lane + k * 32;
      if (i < n4) emit(i, keep[k], gk[k]);
    }
    for (int i = lane + KEEP * 32; i < n4; i += 32) emit(i, xv[i], gr ? ld4f<TO>(gr + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f));
  }
}

// S parallel fp32 residual streams x [T, S, W] (hyper-connections).  coef = mix [from, to] (S x S) | out (S) | in (S):
//   x'_t = sum_s mix[s, t] x_s + out[t] y      all streams from the old ones (without y: x' = x);   written to xn when given
//   u    = sum_t in[t] x'_t;   h = (u - mean) / sqrt(mean((u - mean)^2) + eps) * w       (centre = 0: u / sqrt(mean(u^2) + eps) * w)
// x == nullptr: every old stream is the embedding row table[ids].  One CTA per token; a thread owns the same columns of every stream, so x' may
// replace x in place.  u stays in registers (4 accesses per thread) and, for wider rows, in shared memory; mean and variance are two passes.
// SN: number of streams at compile time (0: at run time, up to 16).  VEC = 4: four columns per access.
template <int VEC> struct StreamVec;
template <> struct StreamVec<1> {
  float v[1];
};
template <> struct StreamVec<4> {
  float v[4];
};
template <int VEC> __device__ __forceinline__ StreamVec<VEC> sv_ld(const float* p) {
  StreamVec<VEC> r;
  if constexpr (VEC == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
  } else r.v[0] = *p;
  return r;
}
template <int VEC> __device__ __forceinline__ StreamVec<VEC> sv_ld(const __nv_bfloat16* p) {
  StreamVec<VEC> r;
  if constexpr (VEC == 4) {
    const float4 t = ld4f<__nv_bfloat16>(p);
    r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
  } else r.v[0] = __bfloat162float(*p);
  return r;
}
template <int VEC> __device__ __forceinline__ void sv_st(float* p, const StreamVec<VEC>& r) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int VEC> __device__ __forceinline__ void sv_st(__nv_bfloat16* p, const StreamVec<VEC>& r) {
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(r.v[0], r.v[1]), pack_bf16(r.v[2], r.v[3]));
  else *p = __float2bfloat16(r.v[0]);
}

constexpr int STREAM_MAX = 16;
template <int SN> constexpr int STREAM_KEEP = SN > 0 ? 4 : 0;          // accesses per thread whose u stays in registers

template <typename T, int SN, int VEC>
__global__ void __launch_bounds__(256) stream_mix_norm_kernel(const float* x, const T* __restrict__ table, const int* __restrict__ ids, int rows,
                                                              const T* __restrict__ y, const float* __restrict__ coef, int streams, const T* __restrict__ w,
                                                              float* xn, T* __restrict__ h, int W, float eps, int centre) {
  constexpr int SM = SN > 0 ? SN : STREAM_MAX;
  constexpr int KEEP = STREAM_KEEP<SN>;
  const int S = SN > 0 ? SN : streams;
  extern __shared__ float su[];                     // u beyond the registers' columns
  __shared__ float red[8];
  __shared__ float sc[SM * SM + 2 * SM];
  for (int i = threadIdx.x; i < S * S + 2 * S; i += 256) sc[i] = coef[i];
  __syncthreads();
  const float* cout = sc + S * S;
  const float* cin = cout + S;
  const int t = blockIdx.x;
  const float* xr = x ? x + (size_t)t * S * W : nullptr;
  const T* er = x ? nullptr : table + (size_t)min(max(ids[t], 0), rows - 1) * W;
  const T* yr = y ? y + (size_t)t * W : nullptr;
  float* nr = xn ? xn + (size_t)t * S * W : nullptr;

  auto form = [&](int i) {                          // columns i .. i + VEC - 1: the new streams, and their weighted sum
    StreamVec<VEC> u, yv, old[SM];
#pragma unroll
    for (int e = 0; e < VEC; ++e) u.v[e] = 0.f;
    if (yr) yv = sv_ld<VEC>(yr + i);
    if (xr) {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) old[s] = sv_ld<VEC>(xr + (size_t)s * W + i);
    } else {
      const StreamVec<VEC> e = sv_ld<VEC>(er + i);
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) old[s] = e;
    }
#pragma unroll(SN > 0 ? SM : 1)
    for (int d = 0; d < S; ++d) {
      StreamVec<VEC> nv;
      if (yr) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) nv.v[e] = cout[d] * yv.v[e];
#pragma unroll
        for (int s = 0; s < SM; ++s) {
          if (s < S) {
            const float m = sc[s * S + d];
#pragma unroll
            for (int e = 0; e < VEC; ++e) nv.v[e] += m * old[s].v[e];
          }
        }
      } else if constexpr (SN > 0) nv = old[d];
      else nv = xr ? sv_ld<VEC>(xr + (size_t)d * W + i) : old[0];
      if (nr) sv_st<VEC>(nr + (size_t)d * W + i, nv);
#pragma unroll
      for (int e = 0; e < VEC; ++e) u.v[e] += cin[d] * nv.v[e];
    }
    return u;
  };

  StreamVec<VEC> keep[KEEP > 0 ? KEEP : 1];
  constexpr int KCOLS = KEEP * 256 * VEC;
  float sum = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = (threadIdx.x + k * 256) * VEC;
#pragma unroll
    for (int e = 0; e < VEC; ++e) keep[k].v[e] = 0.f;
    if (i < W) {
      keep[k] = form(i);
#pragma unroll
      for (int e = 0; e < VEC; ++e) sum += keep[k].v[e];
    }
  }
  for (int i = KCOLS + threadIdx.x * VEC; i < W; i += 256 * VEC) {
    const StreamVec<VEC> u = form(i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) { su[i - KCOLS + e] = u.v[e]; sum += u.v[e]; }
  }
  const float mean = centre ? block_sum_256(sum, red) / (float)W : 0.f;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = (threadIdx.x + k * 256) * VEC;
    if (i < W) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) { keep[k].v[e] -= mean; ss += keep[k].v[e] * keep[k].v[e]; }
    }
  }
  for (int i = KCOLS + threadIdx.x * VEC; i < W; i += 256 * VEC) {          // each thread re-reads what it wrote
#pragma unroll
    for (int e = 0; e < VEC; ++e) { const float d = su[i - KCOLS + e] - mean; ss += d * d; }
  }
  const float rs = 1.0f / sqrtf(block_sum_256(ss, red) / (float)W + eps);
  T* hr = h + (size_t)t * W;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = (threadIdx.x + k * 256) * VEC;
    if (i < W) {
      const StreamVec<VEC> a = sv_ld<VEC>(w + i);
      StreamVec<VEC> o;
#pragma unroll
      for (int e = 0; e < VEC; ++e) o.v[e] = keep[k].v[e] * rs * a.v[e];
      sv_st<VEC>(hr + i, o);
    }
  }
  for (int i = KCOLS + threadIdx.x * VEC; i < W; i += 256 * VEC) {
    const StreamVec<VEC> a = sv_ld<VEC>(w + i);
    StreamVec<VEC> o;
#pragma unroll
    for (int e = 0; e < VEC; ++e) o.v[e] = (su[i - KCOLS + e] - mean) * rs * a.v[e];
    sv_st<VEC>(hr + i, o);
  }
}

template <typename T, int SN, int VEC>
void launch_stream_mix(const float* x, const T* table, const int* ids, int rows, const T* y, const float* coef, int S, const T* w, float* xn, T* h, int n,
                       int W, float eps, bool centre, cudaStream_t stream) {
  const int over = W - STREAM_KEEP<SN> * 256 * VEC;
  const size_t smem = over > 0 ? sizeof(float) * (size_t)over : 0;
  if (smem > 200 * 1024) throw std::runtime_error("sglb stream_mix_norm: rows up to 52,000 columns");
  auto kern = stream_mix_norm_kernel<T, SN, VEC>;
  if (smem > 32 * 1024) SGLB_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  kern<<<n, 256, smem, stream>>>(x, table, ids, rows, y, coef, S, w, xn, h, W, eps, centre ? 1 : 0);
  SGLB_CUDA_CHECK(cudaGetLastError());
}

template <typename T>
void dispatch_stream_mix(const float* x, const T* table, const int* ids, int rows, const T* y, const float* coef, int S, const T* w, float* xn, T* h, int n,
                         int W, float eps, bool centre, cudaStream_t stream) {
  auto al = [](const void* p) { return p == nullptr || ((uintptr_t)p % 16) == 0; };
  const bool vec = W % 4 == 0 && al(x) && al(table) && al(y) && al(w) && al(xn) && al(h);
#define SGLB_SM(SN)                                                                                                                       \
  do {                                                                                                                                    \
    if (vec) launch_stream_mix<T, SN, 4>(x, table, ids, rows, y, coef, S, w, xn, h, n, W, eps, centre, stream);                             \
    else launch_stream_mix<T, SN, 1>(x, table, ids, rows, y, coef, S, w, xn, h, n, W, eps, centre, stream);                                 \
  } while (0)
  switch (S) {
    case 1: SGLB_SM(1); break;
    case 2: SGLB_SM(2); break;
    case 3: SGLB_SM(3); break;
    case 4: SGLB_SM(4); break;
    default: SGLB_SM(0);
  }
#undef SGLB_SM
}

}  // namespace

void postnorm_add_rmsnorm_f32(float* residual, const void* delta, bool delta_bf16, const void* post_w, const void* w, void* out, bool out_bf16, int T,
                              int H, float eps, bool zero_centred, int wsp, int ws, cudaStream_t stream) {
  if (T <= 0) return;
  using bf = __nv_bfloat16;
  const float one = zero_centred ? 1.f : 0.f;
  if (out_bf16) {
    if (delta_bf16)
      postnorm_add_rmsnorm_f32_kernel<bf, bf><<<T, 256, 0, stream>>>(residual, (const bf*)delta, (const bf*)post_w, (const bf*)w, (bf*)out, H, eps, one, wsp, ws);
    else
      postnorm_add_rmsnorm_f32_kernel<float, bf><<<T, 256, 0, stream>>>(residual, (const float*)delta, (const bf*)post_w, (const bf*)w, (bf*)out, H, eps, one, wsp, ws);
  } else {
    if (delta_bf16)
      postnorm_add_rmsnorm_f32_kernel<bf, float><<<T, 256, 0, stream>>>(residual, (const bf*)delta, (const float*)post_w, (const float*)w, (float*)out, H, eps, one, wsp, ws);
    else
      postnorm_add_rmsnorm_f32_kernel<float, float><<<T, 256, 0, stream>>>(residual, (const float*)delta, (const float*)post_w, (const float*)w,
                                                                           (float*)out, H, eps, one, wsp, ws);
  }
  SGLB_CUDA_CHECK(cudaGetLastError());
}

void norm_add_f32(float* x, const void* src, bool src_bf16, const int* ids, int rows, const void* w, void* out, bool w_bf16, int T, int H, float eps,
                  bool zero_centred, cudaStream_t stream) {
  if (T <= 0) return;
  using bf = __nv_bfloat16;
  const float one = zero_centred ? 1.f : 0.f;
  auto al = [](const void* p) { return p == nullptr || ((uintptr_t)p % 16) == 0; };
  const bool vec = H % 4 == 0 && al(x) && al(src) && al(w) && al(out);
#define SGLB_NA(TS, TO)                                                                                                                             \
  do {                                                                                                                                              \
    if (vec) norm_add_f32_kernel<TS, TO, 4><<<T, 256, 0, stream>>>(x, (const TS*)src, ids, rows, (const TO*)w, (TO*)out, H, eps, one);                \
    else norm_add_f32_kernel<TS, TO, 1><<<T, 256, 0, stream>>>(x, (const TS*)src, ids, rows, (const TO*)w, (TO*)out, H, eps, one);                    \
  } while (0)
  if (w_bf16) { if (src_bf16) SGLB_NA(bf, bf); else SGLB_NA(float, bf); }
  else { if (src_bf16) SGLB_NA(bf, float); else SGLB_NA(float, float); }
#undef SGLB_NA
  SGLB_CUDA_CHECK(cudaGetLastError());
}

void parallel_add_rmsnorm_f32(float* residual, const void* d1, const void* d2, bool delta_bf16, const float* d3, const void* w1, const void* w2, void* out1,
                              void* out2, bool out_bf16, int T, int H, float eps, bool zero_centred, cudaStream_t stream) {
  if (T <= 0) return;
  using bf = __nv_bfloat16;
  const float one = zero_centred ? 1.f : 0.f;
  auto al = [](const void* p) { return p == nullptr || ((uintptr_t)p % 16) == 0; };
  const bool vec = H % 4 == 0 && al(residual) && al(d1) && al(d2) && al(d3) && al(w1) && al(w2) && al(out1) && al(out2);
#define SGLB_PAR(TD, TO)                                                                                                                         \
  do {                                                                                                                                           \
    if (vec)                                                                                                                                     \
      parallel_add_rmsnorm_f32_kernel<TD, TO, 4><<<T, 256, 0, stream>>>(residual, (const TD*)d1, (const TD*)d2, d3, (const TO*)w1, (const TO*)w2, \
                                                                        (TO*)out1, (TO*)out2, H, eps, one);                                     \
    else                                                                                                                                         \
      parallel_add_rmsnorm_f32_kernel<TD, TO, 1><<<T, 256, 0, stream>>>(residual, (const TD*)d1, (const TD*)d2, d3, (const TO*)w1, (const TO*)w2, \
                                                                        (TO*)out1, (TO*)out2, H, eps, one);                                     \
  } while (0)
  if (out_bf16) { if (delta_bf16) SGLB_PAR(bf, bf); else SGLB_PAR(float, bf); }
  else { if (delta_bf16) SGLB_PAR(bf, float); else SGLB_PAR(float, float); }
#undef SGLB_PAR
  SGLB_CUDA_CHECK(cudaGetLastError());
}

void stream_mix_norm(const float* x, const void* table, const int* ids, int rows, const void* y, const float* coef, int streams, const void* w, float* xn,
                     void* h, bool bf16, int T, int W, float eps, bool centre, cudaStream_t stream) {
  if (T <= 0 || W <= 0) return;
  if (streams < 1 || streams > STREAM_MAX) throw std::runtime_error("sglb stream_mix_norm: 1 to 16 streams");
  using bf = __nv_bfloat16;
  if (bf16) dispatch_stream_mix<bf>(x, (const bf*)table, ids, rows, (const bf*)y, coef, streams, (const bf*)w, xn, (bf*)h, T, W, eps, centre, stream);
  else dispatch_stream_mix<float>(x, (const float*)table, ids, rows, (const float*)y, coef, streams, (const float*)w, xn, (float*)h, T, W, eps, centre, stream);
}

void grouped_rmsnorm(const float* x, const void* w, void* out, bool out_bf16, int T, int C, int groups, float eps, const void* gate, int ldg, int ldo,
                     float out_scale, bool silu, cudaStream_t stream) {
  if (T <= 0) return;
  if (groups <= 0 || C % groups || groups > 65535) throw std::runtime_error("sglb grouped_rmsnorm: the width must split into equal parts");
  const int per = C / groups, act = silu ? 1 : 0;
  const size_t a4 = out_bf16 ? 8 : 16;               // bytes of a four-column access
  auto al = [&](const void* p) { return p == nullptr || ((uintptr_t)p % a4) == 0; };
  using bf = __nv_bfloat16;
  if (groups >= 4 && per % 4 == 0 && per <= 4096 && ldo % 4 == 0 && (!gate || ldg % 4 == 0) && ((uintptr_t)x % 16) == 0 && al(w) && al(out) && al(gate)) {
#define SGLB_GN(TO, KEEP) \
  grouped_rmsnorm_warp_kernel<TO, KEEP><<<T, 256, 0, stream>>>(x, (const TO*)w, (TO*)out, C, per, groups, eps, (const TO*)gate, ldg, ldo, out_scale, act)
    if (out_bf16) { if (per <= 128) SGLB_GN(bf, 1); else if (per <= 256) SGLB_GN(bf, 2); else SGLB_GN(bf, 4); }
    else { if (per <= 128) SGLB_GN(float, 1); else if (per <= 256) SGLB_GN(float, 2); else SGLB_GN(float, 4); }
#undef SGLB_GN
    SGLB_CUDA_CHECK(cudaGetLastError());
    return;
  }
  dim3 g(T, groups);
  if (out_bf16) grouped_rmsnorm_kernel<bf><<<g, 256, 0, stream>>>(x, (const bf*)w, (bf*)out, C, per, eps, (const bf*)gate, ldg, ldo, out_scale, act);
  else grouped_rmsnorm_kernel<float><<<g, 256, 0, stream>>>(x, (const float*)w, (float*)out, C, per, eps, (const float*)gate, ldg, ldo, out_scale, act);
  SGLB_CUDA_CHECK(cudaGetLastError());
}

void add_rmsnorm_f32(float* residual, const void* delta, bool delta_bf16, const void* w, void* out, bool out_bf16, int T, int H, float eps,
                     bool zero_centred, int ws, cudaStream_t stream) {
  if (T <= 0) return;
  const int z = zero_centred ? 1 : 0;
  if (out_bf16) {
    if (delta_bf16)
      add_rmsnorm_f32_kernel<__nv_bfloat16, __nv_bfloat16><<<T, 256, 0, stream>>>(residual, (const __nv_bfloat16*)delta, (const __nv_bfloat16*)w,
                                                                                  (__nv_bfloat16*)out, H, eps, z, ws);
    else
      add_rmsnorm_f32_kernel<float, __nv_bfloat16><<<T, 256, 0, stream>>>(residual, (const float*)delta, (const __nv_bfloat16*)w, (__nv_bfloat16*)out, H,
                                                                          eps, z, ws);
  } else {
    if (delta_bf16)
      add_rmsnorm_f32_kernel<__nv_bfloat16, float><<<T, 256, 0, stream>>>(residual, (const __nv_bfloat16*)delta, (const float*)w, (float*)out, H, eps, z, ws);
    else
      add_rmsnorm_f32_kernel<float, float><<<T, 256, 0, stream>>>(residual, (const float*)delta, (const float*)w, (float*)out, H, eps, z, ws);
  }
  SGLB_CUDA_CHECK(cudaGetLastError());
}

void clamped_glu(const void* gu, void* out, bool bf16, int T, int I, float limit, float alpha, cudaStream_t stream) {
  if (T <= 0 || I <= 0) return;
  if ((I + 255) / 256 > 65535) throw std::runtime_error("sglb clamped_glu: feed-forward width too large for one launch");
  dim3 g(T, (I + 255) / 256);
  if (bf16 && I % 8 == 0 && ((uintptr_t)gu % 16) == 0 && ((uintptr_t)out % 16) == 0) {
    clamped_glu_bf16x8_kernel<<<dim3(T, (I / 8 + 255) / 256), 256, 0, stream>>>((const __nv_bfloat16*)gu, (__nv_bfloat16*)out, I, limit, alpha);
    SGLB_CUDA_CHECK(cudaGetLastError());
    return;
  }
  if (bf16)
    clamped_glu_kernel<__nv_bfloat16><<<g, 256, 0, stream>>>((const __nv_bfloat16*)gu, (__nv_bfloat16*)out, I, limit, alpha);
  else
    clamped_glu_kernel<float><<<g, 256, 0, stream>>>((const float*)gu, (float*)out, I, limit, alpha);
  SGLB_CUDA_CHECK(cudaGetLastError());
}

}  // namespace sglb
