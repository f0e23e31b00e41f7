// State-space mixer with a scalar decay per head and token (state-space duality):
//     S_t = exp(−exp(A_log)·dt_t)·S_{t−1} + dt_t·B_t x_tᵀ,   y_t = S_tᵀ C_t + D·x_t,   output y_t · silu(z_t)
// x, B and C come from a causal convolution per channel followed by silu, dt from a softplus.  S is fp32, [slots, H, N, V]; the
// convolution's last inputs are kept in a ring per sequence, indexed by position mod taps: a decode step writes the one entry that no
// other CTA of the step reads.  A sequence whose first token of the batch is at position 0 starts from nothing.
//
//   ssm_conv_kernel   convolution, step sizes and log decays of any pieces
//   ssm_seq_kernel    the recurrence token by token, any sizes and pieces (bf16 or float)
//   ssm_step_kernel   one token per sequence (decode), everything in one launch: streams the state once, 16 bytes per thread and access
#include "short_conv.cuh"

namespace mb {
namespace mx {

inline __host__ __device__ MbConv conv_of(const MbSsm& m) {
  return MbConv{m.H * m.V, m.H * m.V + 2 * m.G * m.N, m.taps, m.conv_w, m.conv_b, m.ring, m.slots, m.positions};
}

// 1-D grid: n_tiles · (channel blocks + 1), then one CTA per token for the aside.  TAPS 0: any number, one load per tap and token.
template <typename T, int V, int TAPS, bool GROUPED>
__global__ void __launch_bounds__(kConv) ssm_conv_kernel(const T* __restrict__ proj, long long ld, MbSsm m, const int* __restrict__ tiles,
                                                         const int* __restrict__ cu_q, int n_tiles, int blocks, T* __restrict__ xbc,
                                                         float* __restrict__ dt, float* __restrict__ la, MbAside a) {
  pdl_trigger();
  pdl_wait();
  const int inner = m.H * m.V, CH = inner + 2 * m.G * m.N;
  if (static_cast<int>(blockIdx.x) >= n_tiles * (blocks + 1)) {
    aside_row<T, V != 1, kConv, GROUPED>(a, blockIdx.x - n_tiles * (blocks + 1));
    return;
  }
  const int tile = blockIdx.x / (blocks + 1), cb = blockIdx.x % (blocks + 1);
  int t0 = tile, t1 = tile + 1, seq = tile, first = 1;
  if (tiles != nullptr) {
    const int4 v = reinterpret_cast<const int4*>(tiles)[tile];
    t0 = v.x; t1 = v.y; seq = v.z; first = v.w;
  }
  if (cb == blocks) {
    const T* bias = reinterpret_cast<const T*>(m.dt_bias);
    const T* al = reinterpret_cast<const T*>(m.A_log);
    for (int i = threadIdx.x; i < (t1 - t0) * m.H; i += kConv) {
      const int t = t0 + i / m.H, h = i % m.H;
      const float d = softplus_t<T>(to_f(proj[t * ld + inner + CH + h]) + to_f(bias[h]));
      dt[static_cast<long long>(t) * m.H + h] = d;
      la[static_cast<long long>(t) * m.H + h] = -exp_t<T>(to_f(al[h])) * d;
    }
    return;
  }
  conv_tile<T, V, TAPS>(proj, ld, conv_of(m), tile, cb, tiles != nullptr, t0, t1, seq, first, cu_q, xbc);
}

static constexpr int kTok = 16;     // tokens staged at a time
static constexpr int kSlice = 32;   // state columns (of V) per CTA

// grid (column slices, heads, sequences), 128 threads: lane = column, warp w owns the rows d ≡ w (mod 4) of the slice
template <typename T>
__global__ void __launch_bounds__(128) ssm_seq_kernel(const T* __restrict__ proj, long long ld, const T* __restrict__ xbc, const float* __restrict__ dt,
                                                      const float* __restrict__ la, MbSsm m, const int* __restrict__ cu_q, T* __restrict__ out) {
  extern __shared__ __align__(16) float sm[];
  const int N = m.N, V = m.V, H = m.H, inner = H * V, CH = inner + 2 * m.G * N;
  float* S = sm;                         // [N][kSlice]
  float* sb = S + N * kSlice;            // [kTok][N]
  float* sc = sb + kTok * N;             // [kTok][N]
  float* sx = sc + kTok * N;             // [kTok][kSlice]
  float* part = sx + kTok * kSlice;      // [kTok][4][kSlice]
  float* sd = part + kTok * 4 * kSlice;  // [kTok] step sizes, [kTok] decays
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kSlice;
  const int t0 = cu_q != nullptr ? cu_q[b] : b, t1 = cu_q != nullptr ? cu_q[b + 1] : b + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, col = c0 + lane;
  const int slot = m.slots[b];
  if (t1 <= t0) return;
  if (slot < 0) {                        // padding row of a decode batch
    for (int t = t0 + warp; t < t1; t += 4)
      if (col < V) out[static_cast<long long>(t) * inner + h * V + col] = from_f<T>(0.f);
    return;
  }
  float* st = m.state + (static_cast<long long>(slot) * H + h) * N * V;
  const bool fresh = m.positions[t0] == 0;
  for (int d = warp; d < N; d += 4) S[d * kSlice + lane] = (!fresh && col < V) ? st[static_cast<long long>(d) * V + col] : 0.f;
  const T* px = xbc + h * V;
  const T* pb = xbc + inner + (h / (H / m.G)) * N;
  const T* pc = pb + m.G * N;
  const float D = to_f(reinterpret_cast<const T*>(m.D)[h]);
  for (int tb = t0; tb < t1; tb += kTok) {
    const int n = min(kTok, t1 - tb);
    __syncthreads();
    for (int i = threadIdx.x; i < n * N; i += 128) {
      const int t = i / N, d = i - t * N;
      sb[i] = to_f(pb[static_cast<long long>(tb + t) * CH + d]);
      sc[i] = to_f(pc[static_cast<long long>(tb + t) * CH + d]);
    }
    for (int i = threadIdx.x; i < n * kSlice; i += 128) {
      const int t = i / kSlice, c = i - t * kSlice;
      sx[i] = c0 + c < V ? to_f(px[static_cast<long long>(tb + t) * CH + c0 + c]) : 0.f;
    }
    for (int t = threadIdx.x; t < n; t += 128) {
      sd[t] = dt[static_cast<long long>(tb + t) * H + h];
      sd[kTok + t] = exp_t<T>(la[static_cast<long long>(tb + t) * H + h]);
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float v = sx[t * kSlice + lane] * sd[t], lam = sd[kTok + t];
      float o = 0.f;
      for (int d = warp; d < N; d += 4) {
        const float s = fmaf(lam, S[d * kSlice + lane], sb[t * N + d] * v);
        S[d * kSlice + lane] = s;
        o = fmaf(s, sc[t * N + d], o);
      }
      part[(t * 4 + warp) * kSlice + lane] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * kSlice; i += 128) {
      const int t = i / kSlice, c = i - t * kSlice;
      if (c0 + c >= V) continue;
      const float* p = part + t * 4 * kSlice + c;
      const float y = fmaf(D, sx[i], (p[0] + p[kSlice]) + (p[2 * kSlice] + p[3 * kSlice]));
      out[static_cast<long long>(tb + t) * inner + h * V + c0 + c] = from_f<T>(y * silu_t<T>(to_f(proj[(tb + t) * ld + h * V + c0 + c])));
    }
  }
  for (int d = warp; d < N; d += 4)
    if (col < V) st[static_cast<long long>(d) * V + col] = S[d * kSlice + lane];
}

static constexpr int kStep = 256;
// grid (heads / HP (+ 1 with an aside), rows), 256 threads; V % 4 == 0, HP · V ≤ 1024.  A CTA takes HP neighbouring heads of a group: they share
// the convolution of B and C, and enough of the state is on its way.  A thread owns four columns of a head in every (256 / (HP · V / 4))-th
// state row.
template <typename T, bool GROUPED, int HP>
__global__ void __launch_bounds__(kStep) ssm_step_kernel(const T* __restrict__ proj, long long ld, MbSsm m, T* __restrict__ out, MbAside a,
                                                         int aside_vec_ok) {
  extern __shared__ __align__(16) float sm[];
  pdl_trigger();
  pdl_wait();
  const int N = m.N, V = m.V, H = m.H, inner = H * V, CH = inner + 2 * m.G * N, per = H / m.G;
  const int b = blockIdx.y, h0 = blockIdx.x * HP, W = HP * V;
  if (h0 >= H) {
    if (aside_vec_ok) aside_row<T, true, kStep, GROUPED>(a, b);
    else aside_row<T, false, kStep, GROUPED>(a, b);
    return;
  }
  const int slot = m.slots[b];
  T* o = out + static_cast<long long>(b) * inner + h0 * V;
  if (slot < 0) {                        // padding row
    for (int i = threadIdx.x; i < W; i += kStep) o[i] = from_f<T>(0.f);
    return;
  }
  const int cg = W / 4, rpp = kStep / cg;                // column groups, state rows per pass
  float* red = sm;                       // [rpp][W]
  float* sx = red + rpp * W;             // [W | N | N]: x, B, C of this token
  const int row0 = threadIdx.x / cg, col = (threadIdx.x % cg) * 4, mine = HP == 2 && col >= V;      // column among the CTA's, its head
  const bool on = row0 < rpp;
  float* st = m.state + (static_cast<long long>(slot) * H + h0 + mine) * N * V + (col - mine * V);
  const int pos = m.positions[b];
  // the state is on its way while the projections of this token are read, convolved and activated
  constexpr int U = 8 * HP;
  float4 s[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int d = row0 + u * rpp;
    s[u] = (on && pos > 0 && d < N) ? *reinterpret_cast<const float4*>(st + static_cast<long long>(d) * V) : make_float4(0, 0, 0, 0);
  }
  const T* p = proj + b * ld;
  const int g = h0 / per;
  float* ring = m.ring != nullptr ? m.ring + static_cast<long long>(slot) * m.taps * CH : nullptr;
  const float z0 = threadIdx.x < W ? to_f(p[h0 * V + threadIdx.x]) : 0.f;
  const T raw_dt = p[inner + CH + h0 + mine], raw_bias = reinterpret_cast<const T*>(m.dt_bias)[h0 + mine],
          raw_a = reinterpret_cast<const T*>(m.A_log)[h0 + mine];
  constexpr int R = 2;                                   // channels of a thread that are on their way together
  auto channel = [&](int i) { return i < W ? h0 * V + i : i < W + N ? inner + g * N + i - W : inner + (m.G + g) * N + i - W - N; };
  for (int i0 = threadIdx.x; i0 < W + 2 * N; i0 += R * kStep) {
    float x[R], y[R];
#pragma unroll
    for (int u = 0; u < R; ++u) {
      const int i = i0 + u * kStep;
      x[u] = y[u] = 0.f;
      if (i >= W + 2 * N) continue;
      const int c = channel(i);
      x[u] = to_f(p[inner + c]);
      y[u] = fmaf(to_f(reinterpret_cast<const T*>(m.conv_w)[static_cast<long long>(c) * m.taps + m.taps - 1]), x[u],
                  to_f(reinterpret_cast<const T*>(m.conv_b)[c]));
    }
    for (int k0 = 1; k0 < m.taps; k0 += 3) {             // three inputs back at a time, all on their way together
      float f[R][3], w[R][3];
#pragma unroll
      for (int u = 0; u < R; ++u) {
        const int i = i0 + u * kStep, c = i < W + 2 * N ? channel(i) : 0;
#pragma unroll
        for (int k = 0; k < 3; ++k) {
          const int q = pos - k0 - k;
          const bool ok = i < W + 2 * N && k0 + k < m.taps && q >= 0;
          f[u][k] = ok ? ring[static_cast<long long>(q % m.taps) * CH + c] : 0.f;
          w[u][k] = ok ? to_f(reinterpret_cast<const T*>(m.conv_w)[static_cast<long long>(c) * m.taps + m.taps - 1 - k0 - k]) : 0.f;
        }
      }
#pragma unroll
      for (int u = 0; u < R; ++u)
#pragma unroll
        for (int k = 0; k < 3; ++k) y[u] = fmaf(w[u][k], f[u][k], y[u]);
    }
#pragma unroll
    for (int u = 0; u < R; ++u) {
      const int i = i0 + u * kStep;
      if (i >= W + 2 * N) continue;
      sx[i] = to_f(from_f<T>(silu_t<T>(y[u])));          // as the general path stores it
      if (ring != nullptr && (i < W || h0 % per == 0)) ring[static_cast<long long>(pos % m.taps) * CH + channel(i)] = x[u];
    }
  }
  const float dt = softplus_t<T>(to_f(raw_dt) + to_f(raw_bias)), lam = exp_t<T>(-exp_t<T>(to_f(raw_a)) * dt);
  __syncthreads();
  if (on) {
    const float* sB = sx + W;
    const float* sC = sB + N;
    float v[4], y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = sx[col + j] * dt;
    for (int d0 = row0; d0 < N; d0 += U * rpp) {
      if (d0 != row0)
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int d = d0 + u * rpp;
          s[u] = (pos > 0 && d < N) ? *reinterpret_cast<const float4*>(st + static_cast<long long>(d) * V) : make_float4(0, 0, 0, 0);
        }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int d = d0 + u * rpp;
        if (d >= N) break;
        const float k = sB[d], q = sC[d];
        s[u].x = fmaf(lam, s[u].x, k * v[0]);
        s[u].y = fmaf(lam, s[u].y, k * v[1]);
        s[u].z = fmaf(lam, s[u].z, k * v[2]);
        s[u].w = fmaf(lam, s[u].w, k * v[3]);
        y[0] = fmaf(s[u].x, q, y[0]);
        y[1] = fmaf(s[u].y, q, y[1]);
        y[2] = fmaf(s[u].z, q, y[2]);
        y[3] = fmaf(s[u].w, q, y[3]);
        *reinterpret_cast<float4*>(st + static_cast<long long>(d) * V) = s[u];
      }
    }
    *reinterpret_cast<float4*>(red + row0 * W + col) = make_float4(y[0], y[1], y[2], y[3]);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < W; i += kStep) {
    float r = to_f(reinterpret_cast<const T*>(m.D)[h0 + i / V]) * sx[i];
    for (int w = 0; w < rpp; ++w) r += red[w * W + i];
    o[i] = from_f<T>(r * silu_t<T>(i < kStep ? z0 : to_f(p[h0 * V + i])));
  }
}

template <typename T, int V, bool GROUPED>
static int conv_taps(const T* proj, long long ld, MbSsm m, const int* tiles, const int* cu_q, int n_tiles, T* xbc, float* dt, float* la, int n_aside,
                     MbAside a, cudaStream_t s) {
  const int CH = m.H * m.V + 2 * m.G * m.N, blocks = (CH + kConv * V - 1) / (kConv * V);
  auto kern = m.taps == 4 ? ssm_conv_kernel<T, V, 4, GROUPED> : m.taps == 3 ? ssm_conv_kernel<T, V, 3, GROUPED>
            : m.taps == 2 ? ssm_conv_kernel<T, V, 2, GROUPED> : ssm_conv_kernel<T, V, 0, GROUPED>;
  return static_cast<int>(launch_pdl(kern, dim3(static_cast<unsigned>(n_tiles * (blocks + 1) + n_aside)), dim3(kConv), 0, s, proj, ld, m, tiles, cu_q,
                                     n_tiles, blocks, xbc, dt, la, a));
}

static bool sizes_ok(const MbSsm& m) {
  return m.H > 0 && m.V > 0 && m.N > 0 && m.G > 0 && m.H % m.G == 0 && m.taps >= 1 && m.taps <= kConvTaps && (m.taps == 1 || m.ring != nullptr);
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

extern "C" int mb_ssm_conv(const void* proj, long long ld, MbSsm m, const int* tiles, const int* cu_q, int n_tiles, void* xbc, float* dt, float* la, int T,
                           MbAside a, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  if (!sizes_ok(m) || !aside_ok(a)) return -3;
  auto run = [&](auto ty) {
    using E = decltype(ty);
    constexpr int v = 16 / static_cast<int>(sizeof(E));
    const int n_aside = aside_on(a) ? T : 0;
    const bool vec = ld % v == 0 && (m.H * m.V) % v == 0 && (m.G * m.N) % v == 0 && reinterpret_cast<uintptr_t>(proj) % 16 == 0 && aside_vec<E>(a);
    auto P = reinterpret_cast<const E*>(proj);
    auto X = reinterpret_cast<E*>(xbc);
    auto f = a.grouped ? (vec ? conv_taps<E, v, true> : conv_taps<E, 1, true>) : (vec ? conv_taps<E, v, false> : conv_taps<E, 1, false>);
    return f(P, ld, m, tiles, cu_q, n_tiles, X, dt, la, n_aside, a, s);
  };
  return f32 ? run(float{}) : run(bf16{});
}

extern "C" int mb_ssm_step(const void* proj, long long ld, MbSsm m, void* out, int B, MbAside a, int f32, cudaStream_t s) {
  if (B <= 0) return 0;
  if (!sizes_ok(m) || m.V % 4 || m.V > 4 * kStep || B > 65535 || !aside_ok(a)) return -3;
  // two heads per CTA where that leaves CTAs for every SM
  const int hp = m.V <= 64 && (m.H / m.G) % 2 == 0 && static_cast<long long>(B) * m.H >= 4 * 148 ? 2 : 1, W = hp * m.V;
  const size_t bytes = (static_cast<size_t>(kStep / (W / 4)) * W + W + 2 * m.N) * sizeof(float);
  if (bytes > 48 * 1024) return -3;
  auto run = [&](auto ty) {
    using E = decltype(ty);
    auto kern = hp == 2 ? (a.grouped ? ssm_step_kernel<E, true, 2> : ssm_step_kernel<E, false, 2>)
                        : (a.grouped ? ssm_step_kernel<E, true, 1> : ssm_step_kernel<E, false, 1>);
    return static_cast<int>(launch_pdl(kern, dim3(m.H / hp + aside_on(a), B), dim3(kStep), bytes, s, reinterpret_cast<const E*>(proj), ld, m,
                                       reinterpret_cast<E*>(out), a, aside_vec<E>(a) ? 1 : 0));
  };
  return f32 ? run(float{}) : run(bf16{});
}

extern "C" int mb_ssm_seq(const void* proj, long long ld, const void* xbc, const float* dt, const float* la, MbSsm m, const int* cu_q, void* out, int B,
                          int f32, cudaStream_t s) {
  if (B <= 0) return 0;
  if (!sizes_ok(m) || B > 65535) return -3;
  const size_t bytes = (static_cast<size_t>(m.N) * (kSlice + 2 * kTok) + kTok * kSlice * 5 + 2 * kTok) * sizeof(float);
  if (bytes > 200 * 1024) return -3;
  auto run = [&](auto ty) {
    using E = decltype(ty);
    static bool once = false;
    if (!once) {
      const cudaError_t e = cudaFuncSetAttribute(ssm_seq_kernel<E>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e != cudaSuccess) return static_cast<int>(e);
      once = true;
    }
    return static_cast<int>(launch_pdl(ssm_seq_kernel<E>, dim3((m.V + kSlice - 1) / kSlice, m.H, B), dim3(128), bytes, s, reinterpret_cast<const E*>(proj),
                                       ld, reinterpret_cast<const E*>(xbc), dt, la, m, cu_q, reinterpret_cast<E*>(out)));
  };
  return f32 ? run(float{}) : run(bf16{});
}
