// Shared device helpers of the layer-by-layer decoder kernels (mixers.cu, latent_attn.cu, linear_state.cu).
//
// Those kernels are templates over the model's dtype T.  With T = float the result must be good to 32 bits although the
// extension is compiled with fast math, so exponentials go through double precision and divisions and roots use the
// correctly rounded intrinsics; with T = bf16 the fast forms are used.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "launch.h"
#include "pdl.cuh"

namespace mb {
namespace mx {

using bf16 = __nv_bfloat16;

template <typename T> struct is_exact { static constexpr bool value = false; };
template <> struct is_exact<float> { static constexpr bool value = true; };

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16(v); }

template <typename T> __device__ __forceinline__ float exp_t(float x) {
  if constexpr (is_exact<T>::value) return static_cast<float>(exp(static_cast<double>(x)));
  else return __expf(x);
}
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) {
  if constexpr (is_exact<T>::value) return static_cast<float>(1.0 / (1.0 + exp(-static_cast<double>(x))));
  else return __fdividef(1.f, 1.f + __expf(-x));
}
// __fdividef(1, inf) is 0 and __expf(88.8…) is inf, so sigmoid_t(−large) is 0 as it should be
template <typename T> __device__ __forceinline__ float silu_t(float x) { return x * sigmoid_t<T>(x); }
__device__ __forceinline__ float rsqrt_exact(float x) { return __fdiv_rn(1.f, __fsqrt_rn(x)); }

// N consecutive values ↔ floats (N·sizeof(T) bytes, 16-byte aligned pieces)
template <int N> __device__ __forceinline__ void load_n(const float* p, float (&f)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      const float4 v = *reinterpret_cast<const float4*>(p + i);
      f[i] = v.x; f[i + 1] = v.y; f[i + 2] = v.z; f[i + 3] = v.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = p[i];
  }
}
template <int N> __device__ __forceinline__ void load_n(const bf16* p, float (&f)[N]) {
  if constexpr (N == 8) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(w[i] << 16);
      f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int N> __device__ __forceinline__ void store_n(float* p, const float (&f)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = f[i];
  }
}
template <int N> __device__ __forceinline__ void store_n(bf16* p, const float (&f)[N]) {
  if constexpr (N == 8) {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      __nv_bfloat162 h = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
      w[i] = *reinterpret_cast<uint32_t*>(&h);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = __float2bfloat16(f[i]);
  }
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* sh) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
  __syncthreads();
  float r = 0.f;
#pragma unroll
  for (int w = 0; w < THREADS / 32; ++w) r += sh[w];
  return r;
}

// cs[0 … half) = cosines, cs[half … 2·half) = sines of position · frequency, times `magnitude`; angles in double precision, so that a
// position of any size costs no accuracy.  The caller's CTA barrier comes after.
template <typename T, int THREADS>
__device__ __forceinline__ void rotary_table(float* cs, int position, const double* __restrict__ freq, int half, float magnitude) {
  const double pos = position;
  for (int i = threadIdx.x; i < half; i += THREADS) {
    double a = pos * freq[i];
    a -= rint(a * 0.15915494309189535) * 6.283185307179586;      // one turn off per whole turn: |a| ≤ π
    if constexpr (is_exact<T>::value) {
      double s, c;
      sincos(a, &s, &c);
      cs[i] = static_cast<float>(c * magnitude);
      cs[half + i] = static_cast<float>(s * magnitude);
    } else {
      float s, c;
      __sincosf(static_cast<float>(a), &s, &c);
      cs[i] = c * magnitude;
      cs[half + i] = s * magnitude;
    }
  }
}

// gate · sigmoid(alpha · gate) · (up + 1) with gate ≤ limit and |up| ≤ limit
template <typename T> __device__ __forceinline__ float clamped_glu_t(float gate, float up, float limit, float alpha) {
  const float a = fminf(gate, limit), b = fminf(fmaxf(up, -limit), limit);
  return a * sigmoid_t<T>(alpha * a) * (b + 1.f);
}

// One warp chooses the K largest of E logits (ties: the lower index) and weighs them by a softmax over the chosen ones.  A row of
// NaNs leaves index −1, weight 0.
template <typename T>
__device__ __forceinline__ void topk_softmax_row(const float* __restrict__ z, int E, int K, float* __restrict__ w, int* __restrict__ idx) {
  const int lane = threadIdx.x & 31;
  float last = INFINITY, first = 0.f, sum = 0.f;
  int last_i = -1;
  for (int j = 0; j < K; ++j) {
    float bv = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      const float v = z[e];
      if ((v < last || (v == last && e > last_i)) && (v > bv || (v == bv && e < bi))) { bv = v; bi = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
    if (j == 0) first = bv;
    const bool found = bi != 0x7fffffff;
    const float p = found ? exp_t<T>(bv - first) : 0.f;
    sum += p;
    if (lane == (j & 31)) { idx[j] = found ? bi : -1; w[j] = p; }
    last = bv;
    last_i = bi;
  }
  for (int j = lane; j < K; j += 32) w[j] = sum > 0.f ? __fdiv_rn(w[j], sum) : 0.f;      // every lane reads back what it wrote
}

}  // namespace mx
}  // namespace mb
