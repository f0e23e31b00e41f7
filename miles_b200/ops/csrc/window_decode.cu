// Decode attention over a paged cache of keys and values with a sliding window that keeps the first tokens, and a softmax sink.
//
// One cluster = (token, key head, up to R = 8 or 16 query heads of its group); its CTAs split the keys the token sees, which are numbered
// without a gap: first the kept ones, then those of the window.  As in paged_decode.cu the heads of the group are rows of
// mma.sync.m16n8k16 and tiles of 64 keys are gathered from their pages with cp.async, double buffered, 16 keys per warp.  What differs:
//   * the softmax weights enter P·V as two bf16 parts, 16 bits of mantissa.  R = 8: the eight rows that pad the tile carry the second
//     part for no extra instruction, and the two halves of the accumulator are added at the end.  R = 16: two products;
//   * the splits are joined through distributed shared memory, the sink enters there: one launch, no partial results in HBM;
//   * a token may see its own chunk instead of a window; BIAS: r1 · ln(1 + r2 · distance) comes off the scores; outputs may pass a gate
//     (MbScores);
//   * differential attention (MbDiff): heads 2h and 2h + 1 are neighbours among the rows; a warp joins both, subtracts, norms and gates.
// Heads narrower than DK / DV are padded with zeros in shared memory.
#include <cooperative_groups.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "launch.h"
#include "mma_sync.cuh"
#include "pdl.cuh"

namespace mb {
namespace wd {

namespace cg = cooperative_groups;
using namespace mb::ms;
using bf16 = __nv_bfloat16;
static constexpr float kLog2e = 1.4426950408889634f;
static constexpr int TK = 64;

template <int D>
__device__ __forceinline__ int toff(int row, int chunk) { return row * D + ((chunk ^ (row & 7)) << 3); }

template <int DK, int DV, int R>
struct Smem {
  // the warps' outputs take the place of the key tiles where they fit, the split's output that of the value tiles
  static constexpr int q = 0, k = 16 * DK * 2, v = k + 2 * TK * DK * 2, ml = v + 2 * TK * DV * 2, fml = ml + 8 * R * 4, total = fml + 2 * R * 4;
  static constexpr int o = 4 * R * DV * 4 <= 2 * TK * DK * 2 ? k : v + 2 * TK * DV * 2 + 10 * R * 4, f = v;
  static constexpr int bytes = o == k ? total : o + 4 * R * DV * 4;
};

template <int DK, int DV, int R, bool BIAS>
__global__ void __launch_bounds__(128) window_decode_kernel(const bf16* __restrict__ q, const bf16* __restrict__ kc, const bf16* __restrict__ vc,
                                                            const int* __restrict__ block_table, int max_blocks, int block_size,
                                                            const int* __restrict__ token_seq, const int* __restrict__ positions,
                                                            const long long* __restrict__ slots, const bf16* __restrict__ sink,
                                                            bf16* __restrict__ out, long long o_row, float scale, MbWindow L, MbDiff D, MbScores X) {
  using S = Smem<DK, DV, R>;
  extern __shared__ __align__(128) uint8_t smem[];
  bf16* sQ = reinterpret_cast<bf16*>(smem + S::q);
  bf16* sK = reinterpret_cast<bf16*>(smem + S::k);
  bf16* sV = reinterpret_cast<bf16*>(smem + S::v);
  float* sM = reinterpret_cast<float*>(smem + S::ml);      // [4][R] maxima, then [4][R] sums
  float* sL = sM + 4 * R;
  float* sO = reinterpret_cast<float*>(smem + S::o);       // [4][R][DV]
  float* fO = reinterpret_cast<float*>(smem + S::f);       // [R][DV]: this split's output …
  float* fM = reinterpret_cast<float*>(smem + S::fml);     // [R] maxima (times scale·log2 e), [R] sums
  constexpr int RS = R / 8;                                // rows of a thread: lane / 4 (+ 8)
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.z, split = blockIdx.x, splits = gridDim.x;
  const int group = L.heads / L.kv_heads, chunks = (group + R - 1) / R;
  const int hk = blockIdx.y / chunks, h0 = hk * group + (blockIdx.y % chunks) * R;
  const int rows = min(R, group - (blockIdx.y % chunks) * R);
  const bool diff = D.lam != nullptr;
  if (slots[t] < 0) {                    // padding row of a decode batch (the whole cluster leaves)
    const int heads = diff ? rows / 2 : rows, first = diff ? h0 / 2 : h0;
    for (int i = split * 128 + threadIdx.x; i < heads * L.vdim; i += splits * 128)
      out[t * o_row + static_cast<long long>(first + i / L.vdim) * L.vdim + i % L.vdim] = __float2bfloat16(0.f);
    return;
  }
  const int pos = positions[t];
  const int lo = L.window > 0 ? max(0, pos - L.window + 1) : L.chunk > 0 ? pos - pos % L.chunk : 0, kept = L.window > 0 ? min(L.keep, lo) : 0;
  const int n_keys = kept + pos + 1 - lo;
  const int per = ((n_keys + splits - 1) / splits + TK - 1) / TK * TK;   // keys per split, whole tiles
  const int k_begin = min(split * per, n_keys), k_end = min(n_keys, k_begin + per);
  const int n_tiles = (k_end - k_begin + TK - 1) / TK;
  const int* bt = block_table + static_cast<long long>(token_seq != nullptr ? token_seq[t] : t) * max_blocks;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int kq = DK / 8, kv = DV / 8;

  for (int i = threadIdx.x; i < 16 * kq; i += 128) {
    const int r = i / kq, c = i % kq;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < rows && c * 8 < L.dim) v = *reinterpret_cast<const uint4*>(q + (static_cast<long long>(t) * L.heads + h0 + r) * L.q_pitch + c * 8);
    *reinterpret_cast<uint4*>(sQ + toff<DK>(r, c)) = v;
  }
  // a thread copies one 16-byte column of every (128 / columns)-th row: K and V rows of equal width share the page look-up
  auto load_tile = [&](int tile, int st) {
    const int i0 = k_begin + tile * TK;
    auto slot_of = [&](int r, bool& ok) -> long long {
      const int i = i0 + r;
      ok = i < k_end;
      const int ii = ok ? i : k_begin;
      const int key = ii < kept ? ii : lo + ii - kept;
      return static_cast<long long>(bt[key / block_size]) * block_size + key % block_size;
    };
    if constexpr (DK == DV) {
#pragma unroll
      for (int j = 0; j < TK * kq / 128; ++j) {
        const int r = (threadIdx.x + j * 128) / kq, c = (threadIdx.x + j * 128) % kq;
        bool ok;
        const long long slot = slot_of(r, ok);
        const bool okk = ok && c * 8 < L.dim, okv = ok && c * 8 < L.vdim;
        cp_async16(sK + st * TK * DK + toff<DK>(r, c), kc + (slot * L.kv_heads + hk) * L.dim + (okk ? c * 8 : 0), okk);
        cp_async16(sV + st * TK * DV + toff<DV>(r, c), vc + (slot * L.kv_heads + hk) * L.vdim + (okv ? c * 8 : 0), okv);
      }
    } else {
      for (int i = threadIdx.x; i < TK * kq; i += 128) {
        const int r = i / kq, c = i % kq;
        bool ok;
        const long long slot = slot_of(r, ok);
        ok = ok && c * 8 < L.dim;
        cp_async16(sK + st * TK * DK + toff<DK>(r, c), kc + (slot * L.kv_heads + hk) * L.dim + (ok ? c * 8 : 0), ok);
      }
      for (int i = threadIdx.x; i < TK * kv; i += 128) {
        const int r = i / kv, c = i % kv;
        bool ok;
        const long long slot = slot_of(r, ok);
        ok = ok && c * 8 < L.vdim;
        cp_async16(sV + st * TK * DV + toff<DV>(r, c), vc + (slot * L.kv_heads + hk) * L.vdim + (ok ? c * 8 : 0), ok);
      }
    }
    cp_async_commit();
  };
  if (n_tiles > 0) load_tile(0, 0);
  __syncthreads();
  uint32_t qa[DK / 16][4];               // query fragments stay in registers
#pragma unroll
  for (int ks = 0; ks < DK / 16; ++ks) ldsm_x4(s_addr(sQ + toff<DK>(lane & 15, ks * 2 + (lane >> 4))), qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3]);
  float o_acc[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o_acc[i][0] = o_acc[i][1] = o_acc[i][2] = o_acc[i][3] = 0.f;
  float m_i[RS], l_i[RS];                // of rows lane / 4 (and 8 more)
#pragma unroll
  for (int r = 0; r < RS; ++r) { m_i[r] = -INFINITY; l_i[r] = 0.f; }
  const float sl2 = scale * kLog2e;
  float r1[RS], r2[RS];
#pragma unroll
  for (int r = 0; r < RS; ++r) {
    const int row = (lane >> 2) + 8 * r;
    r1[r] = BIAS && row < rows ? __bfloat162float(reinterpret_cast<const bf16*>(X.r1)[h0 + row]) : 0.f;
    r2[r] = BIAS && row < rows ? __bfloat162float(reinterpret_cast<const bf16*>(X.r2)[h0 + row]) : 0.f;
  }

  for (int tile = 0; tile < n_tiles; ++tile) {
    const int st = tile & 1;
    if (tile + 1 < n_tiles) {
      load_tile(tile + 1, st ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const bf16* tK = sK + st * TK * DK;
    const bf16* tV = sV + st * TK * DV;
    const int key0 = k_begin + tile * TK + warp * 16;
    if (key0 < k_end) {
      float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        uint32_t b[4];
        ldsm_x4(s_addr(tK + toff<DK>(warp * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1))), b[0], b[1], b[2], b[3]);
        mma16816(s[0], qa[ks], b[0], b[1]);
        mma16816(s[1], qa[ks], b[2], b[3]);
      }
      float alpha[RS];
      uint32_t pa[RS][4];                               // R = 8: rows 0–7 the weights' first part, rows 8–15 what rounding took off it
#pragma unroll
      for (int r = 0; r < RS; ++r) {
        float mx = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int i = key0 + nt * 8 + (lane & 3) * 2 + e;
            s[nt][2 * r + e] = i < k_end ? s[nt][2 * r + e] * sl2 : -INFINITY;
            if (BIAS) s[nt][2 * r + e] -= r1[r] * __log2f(fmaf(r2[r], static_cast<float>(max(pos - (i < kept ? i : lo + i - kept), 0)), 1.f));
            mx = fmaxf(mx, s[nt][2 * r + e]);
          }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(m_i[r], fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2)));
        alpha[r] = exp2f(m_i[r] - mx);                  // the first key of the tile is seen: mx is finite
        m_i[r] = mx;
        float rs = 0.f;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const float a = exp2f(s[nt][2 * r] - mx), b = exp2f(s[nt][2 * r + 1] - mx);
          rs += a + b;
          const uint32_t hi = pack2(a, b), lo = pack2(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
          if (R == 8) {
            pa[0][2 * nt] = hi;
            pa[0][2 * nt + 1] = lo;
          } else {                                      // pa[0]: first parts of rows lane / 4 and lane / 4 + 8, pa[1]: second parts
            pa[0][2 * nt + r] = hi;
            pa[RS - 1][2 * nt + r] = lo;
          }
        }
        l_i[r] = l_i[r] * alpha[r] + rs;
      }
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) { o_acc[i][0] *= alpha[0]; o_acc[i][1] *= alpha[0]; o_acc[i][2] *= alpha[RS - 1]; o_acc[i][3] *= alpha[RS - 1]; }
#pragma unroll
      for (int nc = 0; nc < DV / 16; ++nc) {
        uint32_t b[4];
        ldsm_x4_t(s_addr(tV + toff<DV>(warp * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), nc * 2 + (lane >> 4))), b[0], b[1], b[2], b[3]);
#pragma unroll
        for (int part = 0; part < RS; ++part) {
          mma16816(o_acc[2 * nc], pa[part], b[0], b[1]);
          mma16816(o_acc[2 * nc + 1], pa[part], b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int k = 0; k < RS; ++k) {
    l_i[k] += __shfl_xor_sync(0xffffffffu, l_i[k], 1);
    l_i[k] += __shfl_xor_sync(0xffffffffu, l_i[k], 2);
    const int r = (lane >> 2) + 8 * k;
    if ((lane & 3) == 0) { sM[warp * R + r] = m_i[k]; sL[warp * R + r] = l_i[k]; }
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
      *reinterpret_cast<float2*>(sO + (warp * R + r) * DV + i * 8 + (lane & 3) * 2) =
          R == 8 ? make_float2(o_acc[i][0] + o_acc[i][2], o_acc[i][1] + o_acc[i][3]) : make_float2(o_acc[i][2 * k], o_acc[i][2 * k + 1]);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < rows * DV; i += 128) {
    const int g = i / DV, d = i % DV;
    float mm = -INFINITY, ll = 0.f, oo = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, sM[w * R + g]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float a = sM[w * R + g] == -INFINITY ? 0.f : exp2f(sM[w * R + g] - mm);
      ll += sL[w * R + g] * a;
      oo += sO[(w * R + g) * DV + d] * a;
    }
    fO[g * DV + d] = oo;
    if (d == 0) { fM[g] = mm; fM[R + g] = ll; }
  }
  // join the splits: every CTA of the cluster finishes its share of the outputs
  cg::cluster_group cluster = cg::this_cluster();
  if (splits > 1) cluster.sync();
  else __syncthreads();
  if (diff) {                            // a warp per head: both maps, their difference, its norm and gate
    const float lam = *D.lam;
    for (int hp = split * 4 + warp; hp < rows / 2; hp += splits * 4) {
      const int head = h0 / 2 + hp;
      const float gate = __bfloat162float(reinterpret_cast<const bf16*>(D.gate)[t * D.gate_ld + head]);
      float v[DV / 32], ss = 0.f;
#pragma unroll
      for (int j = 0; j < DV / 32; ++j) v[j] = 0.f;
#pragma unroll
      for (int map = 0; map < 2; ++map) {
        const int g = 2 * hp + map;
        float mm = -INFINITY, ms[8], den = 0.f, w[8];
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          ms[c] = c < splits ? cluster.map_shared_rank(fM, c)[g] : -INFINITY;
          mm = fmaxf(mm, ms[c]);
        }
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          w[c] = 0.f;
          if (ms[c] == -INFINITY) continue;
          w[c] = exp2f(ms[c] - mm);
          den = fmaf(cluster.map_shared_rank(fM, c)[R + g], w[c], den);
        }
        const float f = __fdiv_rn(map ? -lam : 1.f, den);
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          if (w[c] == 0.f) continue;
          const float* o = cluster.map_shared_rank(fO, c) + g * DV;
#pragma unroll
          for (int j = 0; j < DV / 32; ++j) v[j] = fmaf(o[lane + 32 * j], w[c] * f, v[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < DV / 32; ++j)
        if (lane + 32 * j < L.vdim) ss = fmaf(v[j], v[j], ss);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float rstd = __fdiv_rn(1.f, __fsqrt_rn(__fdiv_rn(ss, static_cast<float>(L.vdim)) + D.eps));
      const float f = rstd * D.gain * __fdividef(1.f, 1.f + __expf(-gate));
#pragma unroll
      for (int j = 0; j < DV / 32; ++j)
        if (lane + 32 * j < L.vdim) out[t * o_row + static_cast<long long>(head) * L.vdim + lane + 32 * j] = __float2bfloat16(v[j] * f);
    }
  }
  for (int i = split * 128 + threadIdx.x; !diff && i < rows * DV; i += splits * 128) {
    const int g = i / DV, d = i % DV;
    const float sk = sink != nullptr ? __bfloat162float(sink[h0 + g]) * kLog2e : -INFINITY;
    float mm = sk, ms[8];
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      ms[c] = c < splits ? cluster.map_shared_rank(fM, c)[g] : -INFINITY;
      mm = fmaxf(mm, ms[c]);
    }
    float den = sink != nullptr ? exp2f(sk - mm) : 0.f, oo = 0.f;
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      if (ms[c] == -INFINITY) continue;
      const float a = exp2f(ms[c] - mm);
      den = fmaf(cluster.map_shared_rank(fM, c)[R + g], a, den);
      oo = fmaf(cluster.map_shared_rank(fO, c)[g * DV + d], a, oo);
    }
    if (d < L.vdim) {
      const long long at = static_cast<long long>(h0 + g) * L.vdim + d;
      float r = __fdiv_rn(oo, den);
      if (X.gate != nullptr) r *= __fdividef(1.f, 1.f + __expf(-__bfloat162float(reinterpret_cast<const bf16*>(X.gate)[t * X.gate_ld + at])));
      out[t * o_row + at] = __float2bfloat16(r);
    }
  }
  if (splits > 1) cluster.sync();        // the shared memory stays until the others have read it
}

template <int DK, int DV, int R, bool BIAS>
static int launch_rows(const bf16* q, const bf16* kc, const bf16* vc, const int* bt, int max_blocks, int bs, const int* seq, const int* pos,
                  const long long* slots, const bf16* sink, bf16* out, long long o_row, int T, float scale, int splits, MbWindow L, MbDiff d,
                  MbScores x, cudaStream_t s) {
  static bool once = false;
  if (!once) {
    const cudaError_t e = cudaFuncSetAttribute(window_decode_kernel<DK, DV, R, BIAS>, cudaFuncAttributeMaxDynamicSharedMemorySize, Smem<DK, DV, R>::bytes);
    if (e != cudaSuccess) return static_cast<int>(e);
    once = true;
  }
  const int chunks = (L.heads / L.kv_heads + R - 1) / R;
  return static_cast<int>(launch_pdl_cluster(window_decode_kernel<DK, DV, R, BIAS>, dim3(splits, L.kv_heads * chunks, T), dim3(128), splits,
                                             Smem<DK, DV, R>::bytes, s, q, kc, vc, bt, max_blocks, bs, seq, pos, slots, sink, out, o_row, scale, L, d, x));
}

// groups of more than 8 heads are read once for 16 of them
template <int DK, int DV>
static int launch(const bf16* q, const bf16* kc, const bf16* vc, const int* bt, int max_blocks, int bs, const int* seq, const int* pos,
                  const long long* slots, const bf16* sink, bf16* out, long long o_row, int T, float scale, int splits, MbWindow L, MbDiff d,
                  MbScores x, cudaStream_t s) {
  auto f = x.r1 != nullptr ? (L.heads / L.kv_heads > 8 ? launch_rows<DK, DV, 16, true> : launch_rows<DK, DV, 8, true>)
                           : (L.heads / L.kv_heads > 8 ? launch_rows<DK, DV, 16, false> : launch_rows<DK, DV, 8, false>);
  return f(q, kc, vc, bt, max_blocks, bs, seq, pos, slots, sink, out, o_row, T, scale, splits, L, d, x, s);
}

}  // namespace wd
}  // namespace mb

using namespace mb;

// q [T, heads, q_pitch], kc [pages·block_size, kv_heads, dim], vc [.., kv_heads, vdim], out rows of o_row elements.  dim, vdim multiples of
// 8 up to 128, splits ∈ 1 … 8, T ≤ 65535.
extern "C" int mb_window_decode(const void* q, const void* kc, const void* vc, const int* block_table, int max_blocks, int block_size, const int* token_seq,
                                const int* positions, const long long* slots, const void* sink, void* out, long long o_row, int T, float scale,
                                int splits, MbWindow L, MbDiff d, MbScores x, cudaStream_t s) {
  if (T <= 0) return 0;
  if (L.dim % 8 || L.vdim % 8 || L.q_pitch % 8 || L.dim > 128 || L.vdim > 128 || L.heads % L.kv_heads || splits < 1 || splits > 8 || T > 65535) return -3;
  if (d.lam != nullptr && (sink != nullptr || (L.heads / L.kv_heads) % 2 || x.gate != nullptr)) return -3;
  if ((L.chunk > 0 && L.window > 0) || (x.r1 != nullptr && sink != nullptr)) return -3;
  using wd::bf16;
  auto Q = reinterpret_cast<const bf16*>(q), K = reinterpret_cast<const bf16*>(kc), V = reinterpret_cast<const bf16*>(vc), SK = reinterpret_cast<const bf16*>(sink);
  auto O = reinterpret_cast<bf16*>(out);
  auto f = L.dim <= 64 ? (L.vdim <= 64 ? wd::launch<64, 64> : wd::launch<64, 128>) : (L.vdim <= 64 ? wd::launch<128, 64> : wd::launch<128, 128>);
  return f(Q, K, V, block_table, max_blocks, block_size, token_seq, positions, slots, SK, O, o_row, T, scale, splits, L, d, x, s);
}
