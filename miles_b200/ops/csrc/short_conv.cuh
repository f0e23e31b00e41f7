// Short causal convolution per channel followed by silu, over the packed pieces of a batch (ssm_state.cu, delta_state.cu).
//
// A sequence's last inputs are kept in a ring, indexed by position mod taps, with one entry more than the convolution looks back: a
// decode step writes the one entry that no other CTA of the step reads.  A sequence whose first token of the batch is at position 0 starts
// from nothing.
#pragma once
#include "mixers.cuh"

namespace mb {
namespace mx {

static constexpr int kConv = 128, kConvTaps = 33;      // threads, most taps (a tile has at least taps − 1 tokens)

// silu of neighbours; in bf16 two share one reciprocal: 1/a = b · 1/(ab).  Arguments below −40 count as −40 in the exponential (the result
// is zero to 15 digits either way), which keeps the product finite.
template <typename T, int V> __device__ __forceinline__ void silu_n(float (&y)[V]) {
  if constexpr (is_exact<T>::value || V % 2) {
#pragma unroll
    for (int j = 0; j < V; ++j) y[j] = silu_t<T>(y[j]);
  } else {
#pragma unroll
    for (int j = 0; j < V; j += 2) {
      const float a = 1.f + __expf(fminf(-y[j], 40.f)), b = 1.f + __expf(fminf(-y[j + 1], 40.f));
      const float r = __fdividef(1.f, a * b);
      y[j] *= r * b;
      y[j + 1] *= r * a;
    }
  }
}

// V values as they lie in memory (16 bytes, or one value), and as floats
template <typename T, int V> struct Raw {
  uint4 v;
  __device__ __forceinline__ void load(const T* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float (&f)[V]) const {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int j = 0; j < V; ++j)
      f[j] = sizeof(T) == 4 ? __uint_as_float(w[j % 4]) : __uint_as_float((j & 1) ? w[j / 2 % 4] & 0xffff0000u : w[j / 2 % 4] << 16);
  }
};
template <typename T> struct Raw<T, 1> {
  T v;
  __device__ __forceinline__ void load(const T* p) { v = *p; }
  __device__ __forceinline__ void get(float (&f)[1]) const { f[0] = to_f(v); }
};

// Channel block `cb` of one tile: the tokens [t0, t1) of sequence `seq`, `first` for a piece's first tile (see mb_ssm_conv), or token t0 of row
// `seq` in a decode step (packed_pieces false).  TAPS 0: any number, one load per tap and token.
template <typename T, int V, int TAPS>
__device__ __forceinline__ void conv_tile(const T* __restrict__ proj, long long ld, const MbConv& m, int tile, int cb, bool packed_pieces, int t0, int t1,
                                          int seq, int first, const int* __restrict__ cu_q, T* __restrict__ xbc) {
  const int CH = m.channels;
  const int c = (cb * kConv + threadIdx.x) * V;
  if (c >= CH) return;
  const T* in = proj + m.at + c;
  const T* W = reinterpret_cast<const T*>(m.w) + static_cast<long long>(c) * m.taps;
  // weights and the first tokens are on their way before anything is known of the sequence
  constexpr int U = 4;
  Raw<T, V> packed[TAPS > 0 ? TAPS : 1], cur[U];         // V · TAPS weights side by side
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int k = 0; k < TAPS; ++k) packed[k].load(W + k * V);
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (t0 + u < t1) cur[u].load(in + (t0 + u) * ld);
  }
  float b[V];
#pragma unroll
  for (int j = 0; j < V; ++j) b[j] = 0.f;
  if (m.b != nullptr) load_n<V>(reinterpret_cast<const T*>(m.b) + c, b);
  const int slot = m.slots[seq], pos0 = m.positions[t0];
  const int begin = packed_pieces ? cu_q[seq] : tile, end = packed_pieces ? cu_q[seq + 1] : tile + 1;
  if (slot < 0) return;                                  // padding row of a decode batch
  float* ring = m.ring != nullptr ? m.ring + static_cast<long long>(slot) * m.taps * CH + c : nullptr;
  const int taps = TAPS ? TAPS : m.taps;
  // the input `back` places before token t (t − back ≥ t0 − taps + 1)
  auto before = [&](int t, int back, float (&f)[V]) {
    if (t - back >= begin) {
      load_n<V>(in + (t - back) * ld, f);
      return;
    }
    const int p = pos0 + (t - t0) - back;
    if (p >= 0) load_n<V>(ring + static_cast<long long>(p % taps) * CH, f);
    else
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] = 0.f;
  };
  auto finish = [&](int t, float (&y)[V]) {
    silu_n<T, V>(y);
    store_n<V>(xbc + static_cast<long long>(t) * CH + c, y);
  };
  if constexpr (TAPS > 0) {
    float w[TAPS][V], x[TAPS][V];                        // x[k]: the input taps − 1 − k places back
#pragma unroll
    for (int k = 0; k < TAPS - 1; ++k) before(t0, TAPS - 1 - k, x[k]);
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      float f[V];
      packed[k].get(f);
#pragma unroll
      for (int j = 0; j < V; ++j) w[(k * V + j) % TAPS][(k * V + j) / TAPS] = f[j];
    }
    for (int tb = t0; tb < t1; tb += U) {
      Raw<T, V> next[U];
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (tb + U + u < t1) next[u].load(in + (tb + U + u) * ld);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (tb + u < t1) {
          float y[V];
          cur[u].get(x[TAPS - 1]);
#pragma unroll
          for (int j = 0; j < V; ++j) {
            y[j] = b[j];
#pragma unroll
            for (int k = 0; k < TAPS; ++k) y[j] = fmaf(w[k][j], x[k][j], y[j]);
          }
          finish(tb + u, y);
#pragma unroll
          for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
            for (int j = 0; j < V; ++j) x[k][j] = x[k + 1][j];
        }
        cur[u] = next[u];
      }
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float y[V];
#pragma unroll
      for (int j = 0; j < V; ++j) y[j] = b[j];
      for (int k = 0; k < taps; ++k) {
        float x[V];
        before(t, taps - 1 - k, x);
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] = fmaf(to_f(W[j * taps + k]), x[j], y[j]);
      }
      finish(t, y);
    }
  }
  // the tile that starts a piece is the only one that reads the ring (a tile has more tokens than the convolution looks back), and every
  // thread its own channels: it writes the piece's last inputs when it is done
  if (!first || ring == nullptr) return;
  for (int back = min(end - begin, taps - 1); back > 0; --back) {
    float f[V];
    load_n<V>(in + (end - back) * ld, f);
    store_n<V>(ring + static_cast<long long>(m.positions[end - back] % taps) * CH, f);
  }
}

}  // namespace mx
}  // namespace mb
