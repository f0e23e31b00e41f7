// Gated delta rule with a decay per head and key channel:
//     S ← diag(g_t)·S,   u = β_t (v_t − Sᵀk_t),   S ← S + k_t uᵀ,   o_t = Sᵀq_t
// q, k and v come from a causal convolution per channel followed by silu; q and k are unit vectors per head, q over √K on top;
// g = exp(−exp(A_log)·softplus(raw + dt_bias)).  S is fp32, [slots, H, K, V].  A sequence whose first token of the batch is at position 0
// starts from nothing.
//
//   delta_conv_kernel   convolution of any pieces
//   delta_seq_kernel    the recurrence token by token, any sizes and pieces (bf16 or float)
//   delta_step_kernel   one token per sequence (decode), everything in one launch up to the gated norm of the outputs: the state is read once,
//                       stays in registers between the two products with it and is written once
#include "short_conv.cuh"

namespace mb {
namespace mx {

inline __host__ __device__ int channels_of(const MbDelta& m) { return 2 * m.G * m.K + m.H * m.V; }
inline __host__ __device__ MbConv conv_of(const MbDelta& m) {
  return MbConv{0, channels_of(m), m.taps, m.conv_w, nullptr, m.ring, m.slots, m.positions};
}
template <typename T> __device__ __forceinline__ float decay_of(float raw, float bias, float rate) {
  return exp_t<T>(-rate * softplus_t<T>(raw + bias));      // rate = exp(A_log)
}
static constexpr float kUnitEps = 1e-6f;

template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(kConv) delta_conv_kernel(const T* __restrict__ proj, long long ld, MbDelta m, const int* __restrict__ tiles,
                                                           const int* __restrict__ cu_q, int blocks, T* __restrict__ act) {
  pdl_trigger();
  pdl_wait();
  const int tile = blockIdx.x / blocks, cb = blockIdx.x % blocks;
  int t0 = tile, t1 = tile + 1, seq = tile, first = 1;
  if (tiles != nullptr) {
    const int4 v = reinterpret_cast<const int4*>(tiles)[tile];
    t0 = v.x; t1 = v.y; seq = v.z; first = v.w;
  }
  conv_tile<T, V, TAPS>(proj, ld, conv_of(m), tile, cb, tiles != nullptr, t0, t1, seq, first, cu_q, act);
}

static constexpr int kTok = 16;     // tokens staged at a time
static constexpr int kSlice = 32;   // state columns (of V) per CTA

// grid (column slices, heads, sequences), 128 threads: lane = column, warp w owns the rows d ≡ w (mod 4) of the slice
template <typename T>
__global__ void __launch_bounds__(128) delta_seq_kernel(const T* __restrict__ proj, long long ld, const T* __restrict__ act, MbDelta m,
                                                        const int* __restrict__ cu_q, T* __restrict__ out) {
  extern __shared__ __align__(16) float sm[];
  const int K = m.K, V = m.V, H = m.H, CH = channels_of(m);
  float* S = sm;                         // [K][kSlice]
  float* sq = S + K * kSlice;            // [kTok][K]
  float* sk = sq + kTok * K;             // [kTok][K]
  float* sg = sk + kTok * K;             // [kTok][K]
  float* sv = sg + kTok * K;             // [kTok][kSlice]
  float* part = sv + kTok * kSlice;      // [2][4][kSlice]
  float* po = part + 8 * kSlice;         // [kTok][4][kSlice]
  float* sb = po + kTok * 4 * kSlice;    // [kTok]
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kSlice, g = h / (H / m.G);
  const int t0 = cu_q != nullptr ? cu_q[b] : b, t1 = cu_q != nullptr ? cu_q[b + 1] : b + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, col = c0 + lane;
  const int slot = m.slots[b];
  if (t1 <= t0) return;
  if (slot < 0) {                        // padding row of a decode batch
    for (int t = t0 + warp; t < t1; t += 4)
      if (col < V) out[static_cast<long long>(t) * H * V + h * V + col] = from_f<T>(0.f);
    return;
  }
  float* st = m.state + (static_cast<long long>(slot) * H + h) * K * V;
  const bool fresh = m.positions[t0] == 0;
  for (int d = warp; d < K; d += 4) S[d * kSlice + lane] = (!fresh && col < V) ? st[static_cast<long long>(d) * V + col] : 0.f;
  const float rate = exp_t<T>(to_f(reinterpret_cast<const T*>(m.A_log)[h]));
  const T* bias = reinterpret_cast<const T*>(m.dt_bias) + static_cast<long long>(h) * K;
  const T* raw = reinterpret_cast<const T*>(m.raw) + static_cast<long long>(h) * K;
  const float q_scale = __fdiv_rn(1.f, __fsqrt_rn(static_cast<float>(K)));
  for (int tb = t0; tb < t1; tb += kTok) {
    const int n = min(kTok, t1 - tb);
    __syncthreads();
    for (int r = warp; r < 2 * n; r += 4) {              // a warp makes one unit vector
      const int t = r >> 1;
      const T* x = act + static_cast<long long>(tb + t) * CH + ((r & 1) * m.G + g) * K;
      float* y = (r & 1 ? sk : sq) + t * K;
      float ss = 0.f;
      for (int d = lane; d < K; d += 32) {
        const float v = to_f(x[d]);
        ss = fmaf(v, v, ss);
      }
      const float f = rsqrt_exact(warp_sum(ss) + kUnitEps) * (r & 1 ? 1.f : q_scale);
      for (int d = lane; d < K; d += 32) y[d] = to_f(x[d]) * f;
    }
    for (int i = threadIdx.x; i < n * K; i += 128) {
      const int t = i / K, d = i - t * K;
      sg[i] = decay_of<T>(to_f(raw[(tb + t) * m.raw_ld + d]), to_f(bias[d]), rate);
    }
    for (int i = threadIdx.x; i < n * kSlice; i += 128) {
      const int t = i / kSlice, c = i - t * kSlice;
      sv[i] = c0 + c < V ? to_f(act[static_cast<long long>(tb + t) * CH + 2 * m.G * K + h * V + c0 + c]) : 0.f;
    }
    for (int t = threadIdx.x; t < n; t += 128) sb[t] = sigmoid_t<T>(to_f(proj[(tb + t) * ld + m.beta_at + h]));
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float* k = sk + t * K;
      const float* q = sq + t * K;
      const float* dec = sg + t * K;
      float dot = 0.f;
      for (int d = warp; d < K; d += 4) {
        const float s = S[d * kSlice + lane] * dec[d];
        S[d * kSlice + lane] = s;
        dot = fmaf(s, k[d], dot);
      }
      float* p = part + (t & 1) * 4 * kSlice + lane;     // two sets: the next token's sums may come before this one's are read
      p[warp * kSlice] = dot;
      __syncthreads();
      const float u = sb[t] * (sv[t * kSlice + lane] - ((p[0] + p[kSlice]) + (p[2 * kSlice] + p[3 * kSlice])));
      float o = 0.f;
      for (int d = warp; d < K; d += 4) {
        const float s = fmaf(k[d], u, S[d * kSlice + lane]);
        S[d * kSlice + lane] = s;
        o = fmaf(s, q[d], o);
      }
      po[(t * 4 + warp) * kSlice + lane] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * kSlice; i += 128) {
      const int t = i / kSlice, c = i - t * kSlice;
      const float* p = po + t * 4 * kSlice + c;
      if (c0 + c < V) out[static_cast<long long>(tb + t) * H * V + h * V + c0 + c] = from_f<T>((p[0] + p[kSlice]) + (p[2 * kSlice] + p[3 * kSlice]));
    }
  }
  for (int d = warp; d < K; d += 4)
    if (col < V) st[static_cast<long long>(d) * V + col] = S[d * kSlice + lane];
}

static constexpr int kStepRows = 16, kStepThreads = 512;      // state rows of a lane, threads of a CTA at most
// grid (heads, rows of the batch), 32·⌈V/16⌉ threads; V % 4 == 0.  A warp owns 16 state columns: lane = (4 columns lane % 4, rows lane / 4 + 8·u), so
// that both sums over rows are exchanges inside the warp.  THREADS: the most a launch has.
template <typename T, int U, int THREADS>
__global__ void __launch_bounds__(THREADS, 512 / THREADS) delta_step_kernel(const T* __restrict__ proj, long long ld, MbDelta m, const T* __restrict__ norm_w,
                                                                            const T* __restrict__ gate, long long gate_ld, float eps, T* __restrict__ out) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float part[kStepThreads / 32];
  pdl_trigger();
  pdl_wait();
  const int K = m.K, V = m.V, H = m.H, CH = channels_of(m), h = blockIdx.x, b = blockIdx.y, per = H / m.G, g = h / per;
  const int tid = threadIdx.x, threads = blockDim.x, warp = tid >> 5, lane = tid & 31;
  const int slot = m.slots[b], pos = m.positions[b];
  T* o = out + (static_cast<long long>(b) * H + h) * V;
  if (slot < 0) {                        // padding row
    for (int i = tid; i < V; i += threads) o[i] = from_f<T>(0.f);
    return;
  }
  float* sx = sm;                        // [K | K | V]: q, k, v of this token
  float* sg = sx + 2 * K + V;            // [K] decays
  const int row0 = lane >> 2, col = warp * 16 + (lane & 3) * 4;
  const bool on = col < V;
  float* st = m.state + (static_cast<long long>(slot) * H + h) * K * V + col;
  // the state is on its way while the projections of this token are read, convolved and activated
  float4 s[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int d = row0 + u * 8;
    s[u] = (on && pos > 0 && d < K) ? *reinterpret_cast<const float4*>(st + static_cast<long long>(d) * V) : make_float4(0, 0, 0, 0);
  }
  const T* p = proj + b * ld;
  const T* W = reinterpret_cast<const T*>(m.conv_w);
  float* ring = m.ring != nullptr ? m.ring + static_cast<long long>(slot) * m.taps * CH : nullptr;
  const T* gt = gate + b * gate_ld + h * V + col;
  float gv[4], nv[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    gv[j] = on ? to_f(gt[j]) : 0.f;
    nv[j] = on ? to_f(norm_w[col + j]) : 0.f;
  }
  const float beta = sigmoid_t<T>(to_f(p[m.beta_at + h])), rate = exp_t<T>(to_f(reinterpret_cast<const T*>(m.A_log)[h]));
  // everything that is read is on its way before anything is written
  const T* raw = reinterpret_cast<const T*>(m.raw) + b * m.raw_ld + h * K;
  const T* bias = reinterpret_cast<const T*>(m.dt_bias) + h * K;
  const float raw0 = tid < K ? to_f(raw[tid]) : 0.f, bias0 = tid < K ? to_f(bias[tid]) : 0.f;
  const int n = 2 * K + V;
  auto channel = [&](int i) { return i < K ? g * K + i : i < 2 * K ? (m.G + g) * K + i - K : 2 * m.G * K + h * V + i - 2 * K; };
  constexpr int R = 3;                   // channels of a thread at a time
  for (int i0 = tid; i0 < n; i0 += R * threads) {
    float x[R], y[R];
#pragma unroll
    for (int u = 0; u < R; ++u) {
      const int i = i0 + u * threads, c = channel(min(i, n - 1));
      x[u] = to_f(p[c]);
      y[u] = to_f(W[static_cast<long long>(c) * m.taps + m.taps - 1]) * x[u];
    }
    for (int k0 = 1; k0 < m.taps; k0 += 3) {             // three inputs back at a time
      float f[R][3], w[R][3];
#pragma unroll
      for (int u = 0; u < R; ++u) {
        const int c = channel(min(i0 + u * threads, n - 1));
#pragma unroll
        for (int k = 0; k < 3; ++k) {
          const int q = pos - k0 - k;
          const bool ok = k0 + k < m.taps && q >= 0;
          f[u][k] = ok ? ring[static_cast<long long>(q % m.taps) * CH + c] : 0.f;
          w[u][k] = ok ? to_f(W[static_cast<long long>(c) * m.taps + m.taps - 1 - k0 - k]) : 0.f;
        }
      }
#pragma unroll
      for (int u = 0; u < R; ++u)
#pragma unroll
        for (int k = 0; k < 3; ++k) y[u] = fmaf(w[u][k], f[u][k], y[u]);
    }
#pragma unroll
    for (int u = 0; u < R; ++u) {
      const int i = i0 + u * threads;
      if (i >= n) continue;
      sx[i] = to_f(from_f<T>(silu_t<T>(y[u])));          // as the general path stores it
      if (ring != nullptr && (i >= 2 * K || h % per == 0)) ring[static_cast<long long>(pos % m.taps) * CH + channel(i)] = x[u];
    }
  }
  for (int i = tid; i < K; i += threads) {
    const bool first = i == tid;
    sg[i] = decay_of<T>(first ? raw0 : to_f(raw[i]), first ? bias0 : to_f(bias[i]), rate);
  }
  __syncthreads();
  float fq = 0.f, fk = 0.f;              // every warp finds the lengths of q and k
  for (int d = lane; d < K; d += 32) {
    fq = fmaf(sx[d], sx[d], fq);
    fk = fmaf(sx[K + d], sx[K + d], fk);
  }
  fq = rsqrt_exact(warp_sum(fq) + kUnitEps) * __fdiv_rn(1.f, __fsqrt_rn(static_cast<float>(K)));
  fk = rsqrt_exact(warp_sum(fk) + kUnitEps);
  auto over_rows = [&](float (&y)[4]) {
#pragma unroll
    for (int x = 4; x < 32; x <<= 1)
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j] += __shfl_xor_sync(0xffffffffu, y[j], x);
  };
  float y[4] = {0.f, 0.f, 0.f, 0.f}, a[4];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int d = row0 + u * 8;
    if (d < K) {
      const float dec = sg[d], k = sx[K + d] * fk;
      s[u].x *= dec; s[u].y *= dec; s[u].z *= dec; s[u].w *= dec;
      y[0] = fmaf(s[u].x, k, y[0]);
      y[1] = fmaf(s[u].y, k, y[1]);
      y[2] = fmaf(s[u].z, k, y[2]);
      y[3] = fmaf(s[u].w, k, y[3]);
    }
  }
  over_rows(y);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    a[j] = on ? beta * (sx[2 * K + col + j] - y[j]) : 0.f;
    y[j] = 0.f;
  }
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int d = row0 + u * 8;
    if (d < K) {
      const float k = sx[K + d] * fk, q = sx[d] * fq;
      s[u].x = fmaf(k, a[0], s[u].x);
      s[u].y = fmaf(k, a[1], s[u].y);
      s[u].z = fmaf(k, a[2], s[u].z);
      s[u].w = fmaf(k, a[3], s[u].w);
      y[0] = fmaf(s[u].x, q, y[0]);
      y[1] = fmaf(s[u].y, q, y[1]);
      y[2] = fmaf(s[u].z, q, y[2]);
      y[3] = fmaf(s[u].w, q, y[3]);
      if (on) *reinterpret_cast<float4*>(st + static_cast<long long>(d) * V) = s[u];
    }
  }
  over_rows(y);
  const float ss = warp_sum(lane < 4 && on ? y[0] * y[0] + y[1] * y[1] + y[2] * y[2] + y[3] * y[3] : 0.f);
  if (lane == 0) part[warp] = ss;
  __syncthreads();
  if (lane >= 4 || !on) return;
  float sum = 0.f;
  for (int w = 0; w < threads / 32; ++w) sum += part[w];
  const float rstd = rsqrt_exact(__fdiv_rn(sum, static_cast<float>(V)) + eps);
#pragma unroll
  for (int j = 0; j < 4; ++j) o[col + j] = from_f<T>(y[j] * rstd * nv[j] * sigmoid_t<T>(gv[j]));
}

static bool sizes_ok(const MbDelta& m) {
  return m.H > 0 && m.V > 0 && m.K > 0 && m.G > 0 && m.H % m.G == 0 && m.taps >= 1 && m.taps <= kConvTaps && (m.taps == 1 || m.ring != nullptr);
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

extern "C" int mb_delta_conv(const void* proj, long long ld, MbDelta m, const int* tiles, const int* cu_q, int n_tiles, void* act, int f32,
                             cudaStream_t s) {
  if (n_tiles <= 0) return 0;
  if (!sizes_ok(m)) return -3;
  const int CH = channels_of(m);
  auto run = [&](auto ty, auto vec) {
    using E = decltype(ty);
    constexpr int V = decltype(vec)::value;
    const int blocks = (CH + kConv * V - 1) / (kConv * V);
    auto kern = m.taps == 4 ? delta_conv_kernel<E, V, 4> : m.taps == 3 ? delta_conv_kernel<E, V, 3>
              : m.taps == 2 ? delta_conv_kernel<E, V, 2> : delta_conv_kernel<E, V, 0>;
    return static_cast<int>(launch_pdl(kern, dim3(static_cast<unsigned>(n_tiles) * blocks), dim3(kConv), 0, s, reinterpret_cast<const E*>(proj), ld, m,
                                       tiles, cu_q, blocks, reinterpret_cast<E*>(act)));
  };
  auto aligned = [&](int v) { return ld % v == 0 && CH % v == 0 && (reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(m.conv_w)) % 16 == 0; };
  if (f32) return aligned(4) ? run(float{}, std::integral_constant<int, 4>{}) : run(float{}, std::integral_constant<int, 1>{});
  return aligned(8) ? run(bf16{}, std::integral_constant<int, 8>{}) : run(bf16{}, std::integral_constant<int, 1>{});
}

extern "C" int mb_delta_seq(const void* proj, long long ld, const void* act, MbDelta m, const int* cu_q, void* out, int B, int f32, cudaStream_t s) {
  if (B <= 0) return 0;
  if (!sizes_ok(m) || B > 65535) return -3;
  const size_t bytes = (static_cast<size_t>(m.K) * (kSlice + 3 * kTok) + kTok * kSlice * 5 + 8 * kSlice + kTok) * sizeof(float);
  if (bytes > 200 * 1024) return -3;
  auto run = [&](auto ty) {
    using E = decltype(ty);
    static bool once = false;
    if (!once) {
      const cudaError_t e = cudaFuncSetAttribute(delta_seq_kernel<E>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e != cudaSuccess) return static_cast<int>(e);
      once = true;
    }
    return static_cast<int>(launch_pdl(delta_seq_kernel<E>, dim3((m.V + kSlice - 1) / kSlice, m.H, B), dim3(128), bytes, s, reinterpret_cast<const E*>(proj),
                                       ld, reinterpret_cast<const E*>(act), m, cu_q, reinterpret_cast<E*>(out)));
  };
  return f32 ? run(float{}) : run(bf16{});
}

extern "C" int mb_delta_step_ok(int K, int V) { return V % 4 == 0 && (V + 15) / 16 * 32 <= kStepThreads && K <= 8 * kStepRows; }

extern "C" int mb_delta_step(const void* proj, long long ld, MbDelta m, const void* norm_w, const void* gate, long long gate_ld, float eps, void* out, int B,
                             int f32, cudaStream_t s) {
  if (B <= 0) return 0;
  if (!sizes_ok(m) || !mb_delta_step_ok(m.K, m.V) || B > 65535) return -3;
  const int rows = (m.K + 7) / 8, threads = (m.V + 15) / 16 * 32;
  auto run = [&](auto ty) {
    using E = decltype(ty);
    auto kern = threads <= 256 ? (rows <= 4 ? delta_step_kernel<E, 4, 256> : rows <= 8 ? delta_step_kernel<E, 8, 256> : delta_step_kernel<E, kStepRows, 256>)
                               : delta_step_kernel<E, kStepRows, kStepThreads>;
    return static_cast<int>(launch_pdl(kern, dim3(m.H, B), dim3(threads), (3 * m.K + m.V) * sizeof(float), s, reinterpret_cast<const E*>(proj), ld, m,
                                       reinterpret_cast<const E*>(norm_w), reinterpret_cast<const E*>(gate), gate_ld, eps, reinterpret_cast<E*>(out)));
  };
  return f32 ? run(float{}) : run(bf16{});
}
