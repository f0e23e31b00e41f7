// Row-wise kernels of the layer-by-layer decoders: hashed-bigram embedding, output norm + layer scale + fp32 residual (with the
// model's final norm fused into the last one), sum of fp32 residual and sublayer outputs (experts' rows gathered and weighted on the
// way) with the next norm, clamped gated activation, xIELU, gated token rows, gated norm over all heads of a mixer or each by itself,
// soft cap of logits.
// fp32 math; activations in the model's dtype T (bf16, or float for 32-bit runs).
#include <type_traits>

#include "mixers.cuh"

namespace mb {
namespace mx {

static constexpr int kRow = 256;

// x[t] = embed[tok] + table[(prev·mul_prev + tok·mul_cur) mod buckets] (the last row of the table for a sequence's first token) + sines and
// cosines of position · freq (pairs of neighbours share a frequency; angles in double precision, reduced by whole turns)
template <typename T, int V>
__global__ void __launch_bounds__(128) bigram_embed_kernel(const int* __restrict__ tok, const int* __restrict__ prev,
                                                           const T* __restrict__ embed, const T* __restrict__ table, long long buckets,
                                                           long long mul_prev, long long mul_cur, const int* __restrict__ positions,
                                                           const double* __restrict__ freq, float* __restrict__ x, T* __restrict__ xb, int D) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const long long id = tok[t];
  long long row = 0;
  if (table != nullptr) {
    const long long p = prev[t];
    row = p < 0 ? buckets : (p * mul_prev + id * mul_cur) % buckets;
  }
  for (int i = threadIdx.x * V; i < D; i += 128 * V) {
    float a[V];
    load_n<V>(embed + id * D + i, a);
    if (table != nullptr) {
      float b[V];
      load_n<V>(table + row * D + i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] += b[j];
    }
    if (freq != nullptr) {
      const double pos = positions[t];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        double ang = pos * freq[(i + j) >> 1];
        ang -= rint(ang * 0.15915494309189535) * 6.283185307179586;
        if constexpr (is_exact<T>::value) a[j] += static_cast<float>(((i + j) & 1) ? cos(ang) : sin(ang));
        else a[j] += ((i + j) & 1) ? __cosf(static_cast<float>(ang)) : __sinf(static_cast<float>(ang));
      }
    }
    store_n<V>(x + t * D + i, a);
    if (xb != nullptr) store_n<V>(xb + t * D + i, a);
  }
}

// x += mult · y / rms(y) · nw · ls (ls null: 1);  xb = x, or x / rms(x) · fw · gain (the next norm, or the model's final one)
template <typename T, int V>
__global__ void __launch_bounds__(kRow) output_norm_kernel(float* __restrict__ x, const T* __restrict__ y, const T* __restrict__ nw,
                                                           const T* __restrict__ ls, float mult, const T* __restrict__ fw, float gain,
                                                           T* __restrict__ xb, int D, float eps) {
  __shared__ float sh[kRow / 32];
  pdl_trigger();
  pdl_wait();
  const long long base = static_cast<long long>(blockIdx.x) * D;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < D; i += kRow * V) {
    float a[V];
    load_n<V>(y + base + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += a[j] * a[j];
  }
  const float rstd = mult * rsqrt_exact(__fdiv_rn(block_sum<kRow>(ss, sh), static_cast<float>(D)) + eps);
  ss = 0.f;
  for (int i = threadIdx.x * V; i < D; i += kRow * V) {
    float a[V], w[V], l[V], r[V];
#pragma unroll
    for (int j = 0; j < V; ++j) l[j] = 1.f;
    load_n<V>(y + base + i, a);
    load_n<V>(nw + i, w);
    if (ls != nullptr) load_n<V>(ls + i, l);
    load_n<V>(x + base + i, r);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      r[j] += a[j] * rstd * w[j] * l[j];
      ss += r[j] * r[j];
    }
    store_n<V>(x + base + i, r);
    if (fw == nullptr) store_n<V>(xb + base + i, r);
  }
  if (fw == nullptr) return;
  const float rs2 = rsqrt_exact(__fdiv_rn(block_sum<kRow>(ss, sh), static_cast<float>(D)) + eps);
  for (int i = threadIdx.x * V; i < D; i += kRow * V) {      // every thread reads back what it wrote itself
    float w[V], r[V];
    load_n<V>(fw + i, w);
    load_n<V>(x + base + i, r);
#pragma unroll
    for (int j = 0; j < V; ++j) r[j] = r[j] * rs2 * w[j] * gain;
    store_n<V>(xb + base + i, r);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const T* __restrict__ in, long long ld_in, T* __restrict__ out, long long ld_out,
                                                          long long n, int F, float limit, float alpha, float shift,
                                                          const int* __restrict__ rows) {
  pdl_trigger();
  pdl_wait();
  const int per = F / V;
  if (rows != nullptr) n = min(n, static_cast<long long>(*rows));
  for (long long v = blockIdx.x * 256ll + threadIdx.x; v < n * per; v += gridDim.x * 256ll) {
    const long long t = v / per;
    const int i = static_cast<int>(v - t * per) * V;
    float g[V], u[V];
    load_n<V>(in + t * ld_in + i, g);
    load_n<V>(in + t * ld_in + F + i, u);
#pragma unroll
    for (int j = 0; j < V; ++j) g[j] = clamped_glu_t<T>(g[j], u[j], limit, alpha, shift);
    store_n<V>(out + t * ld_out + i, g);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) relu_square_kernel(T* __restrict__ x, long long T_, int n, const int* __restrict__ rows) {
  pdl_trigger();
  pdl_wait();
  if (rows != nullptr) T_ = min(T_, static_cast<long long>(*rows));
  const long long total = T_ * n;
  for (long long i = (blockIdx.x * 256ll + threadIdx.x) * V; i < total; i += gridDim.x * 256ll * V) {
    float a[V];
    load_n<V>(x + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = relu_square(a[j]);
    store_n<V>(x + i, a);
  }
}

// One CTA per token; the sum waits in shared memory for its norm.  Addends: see MbSumNorm.
static constexpr int kMaxTop = 64;
// SCALED: with scales of the addends, or a second norm.
template <typename T, int V, bool SCALED>
__global__ void __launch_bounds__(kRow) sum_norm_kernel(MbSumNorm p) {
  extern __shared__ __align__(16) float row[];
  __shared__ float sh[kRow / 32], s_w[kMaxTop];
  __shared__ int s_dst[kMaxTop];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x, base = t * p.D;
  const T* y1 = reinterpret_cast<const T*>(p.y1);
  const T* y2 = reinterpret_cast<const T*>(p.y2);
  const T* rows = reinterpret_cast<const T*>(p.rows);
  const T* s1 = reinterpret_cast<const T*>(p.s1);
  const T* s2 = reinterpret_cast<const T*>(p.s2);
  const T* nw = reinterpret_cast<const T*>(p.nw);
  const T* nw2 = reinterpret_cast<const T*>(p.nw2);
  T* h = reinterpret_cast<T*>(p.h);
  T* h2 = reinterpret_cast<T*>(p.h2);
  const int k = rows != nullptr ? p.k : 0;
  for (int j = threadIdx.x; j < k; j += kRow) {
    const int d = p.dst[t * p.k + j];
    s_dst[j] = d;
    s_w[j] = d >= 0 ? p.weights[t * p.k + j] : 0.f;
  }
  if (k > 0) __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < p.D; i += kRow * V) {
    float r[V], a[V], c1[V], c2[V];
#pragma unroll
    for (int j = 0; j < V; ++j) c1[j] = c2[j] = 1.f;
    if (SCALED && s1 != nullptr) load_n<V>(s1 + i, c1);
    if (SCALED && s2 != nullptr) load_n<V>(s2 + i, c2);
#pragma unroll
    for (int j = 0; j < V; ++j) { c1[j] *= p.mult; c2[j] *= p.mult; }
    load_n<V>(p.x + base + i, r);
    if (y1 != nullptr) {
      load_n<V>(y1 + base + i, a);
#pragma unroll
      for (int j = 0; j < V; ++j) r[j] += a[j] * c1[j];
    }
    if (y2 != nullptr) {
      load_n<V>(y2 + base + i, a);
#pragma unroll
      for (int j = 0; j < V; ++j) r[j] += a[j] * c2[j];
    }
    if (k > 0) {
      float m[V];
#pragma unroll
      for (int j = 0; j < V; ++j) m[j] = 0.f;
#pragma unroll 4
      for (int c = 0; c < k; ++c) {
        const int d = s_dst[c];
        if (d < 0) continue;
        load_n<V>(rows + static_cast<long long>(d) * p.D + i, a);
        const float w = s_w[c];
#pragma unroll
        for (int j = 0; j < V; ++j) m[j] = fmaf(w, a[j], m[j]);
      }
#pragma unroll
      for (int j = 0; j < V; ++j) r[j] += m[j] * c2[j];
    }
    if (p.extra != nullptr) {
      load_n<V>(p.extra + base + i, a);
#pragma unroll
      for (int j = 0; j < V; ++j) r[j] += a[j];
    }
    if (p.to != nullptr) store_n<V>(p.to + base + i, r);
    if (nw == nullptr) {
      if (h != nullptr) store_n<V>(h + base + i, r);
      continue;
    }
#pragma unroll
    for (int j = 0; j < V; ++j) ss += r[j] * r[j];
    store_n<V>(row + i, r);
  }
  if (nw == nullptr) return;
  const float rstd = rsqrt_exact(__fdiv_rn(block_sum<kRow>(ss, sh), static_cast<float>(p.D)) + p.eps);
  for (int i = threadIdx.x * V; i < p.D; i += kRow * V) {      // every thread reads back what it wrote itself
    float r[V], w[V];
    load_n<V>(row + i, r);
    load_n<V>(nw + i, w);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      r[j] *= rstd;
      w[j] = r[j] * (w[j] + p.shift) * p.gain;
    }
    store_n<V>(h + base + i, w);
    if (!SCALED || nw2 == nullptr) continue;
    load_n<V>(nw2 + i, w);
#pragma unroll
    for (int j = 0; j < V; ++j) w[j] = r[j] * (w[j] + p.shift) * p.gain;
    store_n<V>(h2 + base + i, w);
  }
}

// out = x / rms(x) · w for every one of `parts` equal parts of a row (of x: ld elements apart); grid (rows, parts)
template <typename T, int V>
__global__ void __launch_bounds__(kRow) part_norm_kernel(const T* __restrict__ xs, long long ld, const T* __restrict__ w, T* __restrict__ out, int n,
                                                         int parts, float eps) {
  __shared__ float sh[kRow / 32];
  constexpr int kHold = 4;                 // vectors per thread that stay in registers between the two passes
  pdl_trigger();
  pdl_wait();
  const long long base = (static_cast<long long>(blockIdx.x) * parts + blockIdx.y) * n;
  const T* pw = w + static_cast<long long>(blockIdx.y) * n;
  const T* x = xs + blockIdx.x * ld + static_cast<long long>(blockIdx.y) * n - base;
  float a[kHold][V], ss = 0.f;
#pragma unroll
  for (int u = 0; u < kHold; ++u) {
    const int i = (threadIdx.x + u * kRow) * V;
    if (i < n) {
      load_n<V>(x + base + i, a[u]);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += a[u][j] * a[u][j];
    }
  }
  for (int i = (threadIdx.x + kHold * kRow) * V; i < n; i += kRow * V) {
    float b[V];
    load_n<V>(x + base + i, b);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += b[j] * b[j];
  }
  const float rstd = rsqrt_exact(__fdiv_rn(block_sum<kRow>(ss, sh), static_cast<float>(n)) + eps);
#pragma unroll
  for (int u = 0; u < kHold; ++u) {
    const int i = (threadIdx.x + u * kRow) * V;
    if (i < n) {
      float b[V];
      load_n<V>(pw + i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) b[j] *= a[u][j] * rstd;
      store_n<V>(out + base + i, b);
    }
  }
  for (int i = (threadIdx.x + kHold * kRow) * V; i < n; i += kRow * V) {
    float b[V], c[V];
    load_n<V>(x + base + i, b);
    load_n<V>(pw + i, c);
#pragma unroll
    for (int j = 0; j < V; ++j) b[j] *= rstd * c[j];
    store_n<V>(out + base + i, b);
  }
}

// out = o / rms(o) · w · sigmoid(gate) over all C = heads · vdim channels of a token
template <typename T, int V>
__global__ void __launch_bounds__(kRow) gated_norm_kernel(const T* __restrict__ o, const T* __restrict__ w, const T* __restrict__ gate,
                                                          long long gate_ld, T* __restrict__ out, int C, float eps) {
  __shared__ float sh[kRow / 32];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < C; i += kRow * V) {
    float a[V];
    load_n<V>(o + t * C + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += a[j] * a[j];
  }
  const float rstd = rsqrt_exact(__fdiv_rn(block_sum<kRow>(ss, sh), static_cast<float>(C)) + eps);
  for (int i = threadIdx.x * V; i < C; i += kRow * V) {
    float a[V], b[V], g[V];
    load_n<V>(o + t * C + i, a);
    load_n<V>(w + i, b);
    load_n<V>(gate + t * gate_ld + i, g);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = a[j] * rstd * b[j] * sigmoid_t<T>(g[j]);
    store_n<V>(out + t * C + i, a);
  }
}

// out = o / rms(o) · w · sigmoid(gate), every head's V channels by themselves: `lanes` (a power of two up to 32) threads a head
template <typename T, int N>
__global__ void __launch_bounds__(256) head_gated_norm_kernel(const T* __restrict__ o, const T* __restrict__ w, const T* __restrict__ gate,
                                                              long long gate_ld, T* __restrict__ out, long long heads, int H, int V, int lanes,
                                                              float eps) {
  pdl_trigger();
  pdl_wait();
  const long long hd = (blockIdx.x * 256ll + threadIdx.x) / lanes;      // head of all tokens
  const int l = threadIdx.x & (lanes - 1);
  const bool on = hd < heads;
  const long long base = hd * V;
  const T* g = gate + (hd / H) * gate_ld + (hd % H) * V;
  float ss = 0.f, a[N], first[N];
  for (int i = l * N; on && i < V; i += lanes * N) {
    load_n<N>(o + base + i, a);
#pragma unroll
    for (int j = 0; j < N; ++j) {
      ss += a[j] * a[j];
      if (i == l * N) first[j] = a[j];
    }
  }
  for (int x = lanes / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
  if (!on) return;
  const float rstd = rsqrt_exact(__fdiv_rn(ss, static_cast<float>(V)) + eps);
  for (int i = l * N; i < V; i += lanes * N) {
    float b[N], c[N];
    if (i == l * N) {
#pragma unroll
      for (int j = 0; j < N; ++j) a[j] = first[j];
    } else {
      load_n<N>(o + base + i, a);
    }
    load_n<N>(w + i, b);
    load_n<N>(g + i, c);
#pragma unroll
    for (int j = 0; j < N; ++j) a[j] = a[j] * rstd * b[j] * sigmoid_t<T>(c[j]);
    store_n<N>(out + base + i, a);
  }
}

// exp(z) − 1 − z for z ≤ 0; in bf16 models by its series near zero, where the difference would lose what matters
template <typename T> __device__ __forceinline__ float exp_rest(float z) {
  if constexpr (is_exact<T>::value) return expm1f(z) - z;
  const float series = z * z * fmaf(z, fmaf(z, fmaf(z, 8.3333333e-3f, 4.1666667e-2f), 0.16666667f), 0.5f);
  return z > -0.25f ? series : __expf(z) - 1.f - z;
}

template <typename T, int V>
__global__ void __launch_bounds__(256) xielu_kernel(const T* __restrict__ z, const T* __restrict__ act, T* __restrict__ out, long long n) {
  pdl_trigger();
  pdl_wait();
  const float pos = softplus_t<T>(to_f(act[0])), neg = 0.5f + softplus_t<T>(to_f(act[1]));
  for (long long i = (blockIdx.x * 256ll + threadIdx.x) * V; i < n; i += gridDim.x * 256ll * V) {
    float a[V];
    load_n<V>(z + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = fmaf(0.5f, a[j], a[j] > 0.f ? pos * a[j] * a[j] : neg * exp_rest<T>(a[j]));
    store_n<V>(out + i, a);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) gelu_rows_kernel(const T* __restrict__ z, long long ld, const int* __restrict__ tok, const T* __restrict__ table,
                                                        long long table_ld, int col, T* __restrict__ out, long long rows, int n) {
  pdl_trigger();
  pdl_wait();
  const int per = n / V;
  for (long long v = blockIdx.x * 256ll + threadIdx.x; v < rows * per; v += gridDim.x * 256ll) {
    const long long t = v / per;
    const int i = static_cast<int>(v - t * per) * V;
    float a[V], e[V];
    load_n<V>(z + t * ld + i, a);
    load_n<V>(table + tok[t] * table_ld + col + i, e);
#pragma unroll
    for (int j = 0; j < V; ++j) {      // ½ (1 + tanh u) = sigmoid(2u)
      const float u = 0.7978845608028654f * (a[j] + 0.044715f * a[j] * a[j] * a[j]);
      a[j] = a[j] * sigmoid_t<T>(2.f * u) * e[j];
    }
    store_n<V>(out + t * n + i, a);
  }
}

template <bool EXACT, int V>
__global__ void __launch_bounds__(256) softcap_kernel(float* __restrict__ x, long long n, float cap) {
  pdl_trigger();
  pdl_wait();
  const float inv = __fdiv_rn(1.f, cap);
#pragma unroll 2
  for (long long i = (blockIdx.x * 256ll + threadIdx.x) * V; i < n; i += gridDim.x * 256ll * V) {
    float a[V];
    load_n<V>(x + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      if (EXACT) {
        a[j] = static_cast<float>(cap * tanh(static_cast<double>(a[j]) / cap));
      } else {                         // tanh u = (1 − e) / (1 + e) with e = exp(−2|u|), odd: nothing overflows
        const float u = a[j] * inv, e = __expf(-2.f * fabsf(u));
        a[j] = copysignf(cap * __fdividef(1.f - e, 1.f + e), u);
      }
    }
    store_n<V>(x + i, a);
  }
}

// 16-byte accesses need element counts (and strides) that are whole vectors
template <typename F>
static int dispatch(int f32, bool vec, F&& f) {
  if (f32) return vec ? f(float{}, std::integral_constant<int, 4>{}) : f(float{}, std::integral_constant<int, 1>{});
  return vec ? f(bf16{}, std::integral_constant<int, 8>{}) : f(bf16{}, std::integral_constant<int, 1>{});
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

extern "C" int mb_bigram_embedding(const int* tok, const int* prev, const void* embed, const void* table, long long buckets,
                                   long long mul_prev, long long mul_cur, const int* positions, const double* freq, float* x, void* xb, int T, int D,
                                   int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  return dispatch(f32, D % 8 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    return static_cast<int>(launch_pdl(bigram_embed_kernel<E, decltype(v)::value>, dim3(T), dim3(128), 0, s, tok, prev,
                                       reinterpret_cast<const E*>(embed), reinterpret_cast<const E*>(table), buckets, mul_prev, mul_cur,
                                       positions, freq, x, reinterpret_cast<E*>(xb), D));
  });
}

extern "C" int mb_output_norm(float* x, const void* y, const void* nw, const void* ls, float mult, const void* fw, float gain, void* xb, int T,
                              int D, float eps, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  return dispatch(f32, D % 8 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    return static_cast<int>(launch_pdl(output_norm_kernel<E, decltype(v)::value>, dim3(T), dim3(kRow), 0, s, x, reinterpret_cast<const E*>(y),
                                       reinterpret_cast<const E*>(nw), reinterpret_cast<const E*>(ls), mult, reinterpret_cast<const E*>(fw), gain,
                                       reinterpret_cast<E*>(xb), D, eps));
  });
}

extern "C" int mb_clamped_glu(const void* in, long long ld_in, void* out, long long ld_out, long long T, int F, float limit, float alpha,
                              float shift, const int* rows, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  const bool vec = F % 8 == 0 && ld_in % 8 == 0 && ld_out % 8 == 0 && (reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out)) % 16 == 0;
  return dispatch(f32, vec, [&](auto ty, auto v) {
    using E = decltype(ty);
    constexpr int V = decltype(v)::value;
    const long long blocks = (T * (F / V) + 255) / 256;
    return static_cast<int>(launch_pdl(clamped_glu_kernel<E, V>, dim3(static_cast<unsigned>(blocks < 148 * 16 ? blocks : 148 * 16)), dim3(256), 0,
                                       s, reinterpret_cast<const E*>(in), ld_in, reinterpret_cast<E*>(out), ld_out, T, F, limit, alpha, shift, rows));
  });
}

extern "C" int mb_relu_square(void* x, long long T, int n, const int* rows, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  return dispatch(f32, n % 8 == 0 && reinterpret_cast<uintptr_t>(x) % 16 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    constexpr int V = decltype(v)::value;
    const long long blocks = (T * n / V + 255) / 256;
    return static_cast<int>(launch_pdl(relu_square_kernel<E, V>, dim3(static_cast<unsigned>(blocks < 148 * 16 ? blocks + 1 : 148 * 16)), dim3(256), 0, s,
                                       reinterpret_cast<E*>(x), T, n, rows));
  });
}

static unsigned elementwise_blocks(long long pieces) {
  const long long blocks = (pieces + 255) / 256;
  return static_cast<unsigned>(blocks < 148 * 16 ? (blocks > 0 ? blocks : 1) : 148 * 16);
}

extern "C" int mb_xielu(const void* z, const void* act, void* out, long long n, int f32, cudaStream_t s) {
  if (n <= 0) return 0;
  return dispatch(f32, n % 8 == 0 && (reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) % 16 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    constexpr int V = decltype(v)::value;
    return static_cast<int>(launch_pdl(xielu_kernel<E, V>, dim3(elementwise_blocks(n / V)), dim3(256), 0, s, reinterpret_cast<const E*>(z),
                                       reinterpret_cast<const E*>(act), reinterpret_cast<E*>(out), n));
  });
}

extern "C" int mb_gelu_rows(const void* z, long long ld, const int* tok, const void* table, long long table_ld, int col, void* out, int T, int n, int f32,
                            cudaStream_t s) {
  if (T <= 0 || n <= 0) return 0;
  const bool vec = n % 8 == 0 && ld % 8 == 0 && table_ld % 8 == 0 && col % 8 == 0 &&
                   (reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(table)) % 16 == 0;
  return dispatch(f32, vec, [&](auto ty, auto v) {
    using E = decltype(ty);
    constexpr int V = decltype(v)::value;
    return static_cast<int>(launch_pdl(gelu_rows_kernel<E, V>, dim3(elementwise_blocks(static_cast<long long>(T) * (n / V))), dim3(256), 0, s,
                                       reinterpret_cast<const E*>(z), ld, tok, reinterpret_cast<const E*>(table), table_ld, col,
                                       reinterpret_cast<E*>(out), static_cast<long long>(T), n));
  });
}

extern "C" int mb_softcap(float* x, long long n, float cap, int exact, cudaStream_t s) {
  if (n <= 0) return 0;
  if (!(cap > 0.f)) return -3;
  const bool vec = n % 4 == 0 && reinterpret_cast<uintptr_t>(x) % 16 == 0;
  auto kern = exact ? (vec ? softcap_kernel<true, 4> : softcap_kernel<true, 1>) : (vec ? softcap_kernel<false, 4> : softcap_kernel<false, 1>);
  return static_cast<int>(launch_pdl(kern, dim3(elementwise_blocks(vec ? n / 4 : n)), dim3(256), 0, s, x, n, cap));
}

extern "C" int mb_head_gated_norm(const void* o, const void* w, const void* gate, long long gate_ld, void* out, long long T, int H, int V, float eps, int f32,
                                  cudaStream_t s) {
  if (T <= 0) return 0;
  const bool vec = V % 8 == 0 && gate_ld % 8 == 0 && (reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(out)) % 16 == 0;
  return dispatch(f32, vec, [&](auto ty, auto v) {
    using E = decltype(ty);
    constexpr int N = decltype(v)::value;
    int lanes = 1;
    while (lanes < 32 && lanes * N < V) lanes *= 2;
    const long long threads = T * H * lanes;
    return static_cast<int>(launch_pdl(head_gated_norm_kernel<E, N>, dim3(static_cast<unsigned>((threads + 255) / 256)), dim3(256), 0, s,
                                       reinterpret_cast<const E*>(o), reinterpret_cast<const E*>(w), reinterpret_cast<const E*>(gate), gate_ld,
                                       reinterpret_cast<E*>(out), T * H, H, V, lanes, eps));
  });
}

extern "C" int mb_part_norm(const void* x, long long ld, const void* w, void* out, int T, int C, int parts, float eps, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  if (parts <= 0 || C % parts || parts > 65535) return -3;
  const int n = C / parts;
  return dispatch(f32, n % 8 == 0 && ld % 8 == 0 && reinterpret_cast<uintptr_t>(x) % 16 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    return static_cast<int>(launch_pdl(part_norm_kernel<E, decltype(v)::value>, dim3(T, parts), dim3(kRow), 0, s, reinterpret_cast<const E*>(x),
                                       ld, reinterpret_cast<const E*>(w), reinterpret_cast<E*>(out), n, parts, eps));
  });
}

extern "C" int mb_sum_norm(MbSumNorm p, int f32, cudaStream_t s) {
  if (p.T <= 0) return 0;
  if (p.rows != nullptr && p.k > kMaxTop) return -3;
  const int bytes = p.D * static_cast<int>(sizeof(float));
  if (bytes > 200 * 1024) return -3;
  return dispatch(f32, p.D % 8 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    constexpr int V = decltype(v)::value;
    const bool scaled = p.s1 != nullptr || p.s2 != nullptr || p.nw2 != nullptr;
    auto kern = scaled ? sum_norm_kernel<E, V, true> : sum_norm_kernel<E, V, false>;
    static int configured = 48 * 1024;                 // one per dtype and vector
    if (bytes > configured) {
      cudaError_t e = cudaFuncSetAttribute(sum_norm_kernel<E, V, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e == cudaSuccess) e = cudaFuncSetAttribute(sum_norm_kernel<E, V, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e != cudaSuccess) return static_cast<int>(e);
      configured = 200 * 1024;
    }
    return static_cast<int>(launch_pdl(kern, dim3(p.T), dim3(kRow), bytes, s, p));
  });
}

extern "C" int mb_gated_norm(const void* o, const void* w, const void* gate, long long gate_ld, void* out, int T, int C, float eps, int f32,
                             cudaStream_t s) {
  if (T <= 0) return 0;
  const bool vec = C % 8 == 0 && gate_ld % 8 == 0 && reinterpret_cast<uintptr_t>(gate) % 16 == 0;
  return dispatch(f32, vec, [&](auto ty, auto v) {
    using E = decltype(ty);
    return static_cast<int>(launch_pdl(gated_norm_kernel<E, decltype(v)::value>, dim3(T), dim3(kRow), 0, s, reinterpret_cast<const E*>(o),
                                       reinterpret_cast<const E*>(w), reinterpret_cast<const E*>(gate), gate_ld, reinterpret_cast<E*>(out), C,
                                       eps));
  });
}
