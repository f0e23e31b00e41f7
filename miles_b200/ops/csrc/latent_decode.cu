// Tensor-core kernels of latent attention for a few new tokens per sequence (bf16), and the gather that feeds the prefill form.
//
//   latent_gather_kernel    cached rows of every sequence's key range → packed rows
//   head_linear_mma_kernel  y[t, h, :] = w[h] · x[t, h, :] for a handful of tokens (key up-projection into the query, value
//                           up-projection of the attended latent): weights streamed once per 64 tokens
//   latent_decode_kernel    attention of absorbed queries over the cached latents (mma.sync m16n8k16): 16 or 32 heads of one
//                           token are the M dimension, so a latent row fetched from the cache serves them all, as key and as value;
//                           split keys + merge (latent_merge_kernel adds the softmax sink)
#include "debug.cuh"
#include "mixers.cuh"

namespace mb {
namespace ld {

using mx::bf16;
static constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ uint32_t s_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void cp16(void* dst, const void* src, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s_addr(dst)), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm4(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}

// one warp per packed row: row i of sequence b is position base[b] + (i − cu_k[b])
__global__ void __launch_bounds__(256) latent_gather_kernel(const bf16* __restrict__ cache, const int* __restrict__ block_table, int max_blocks,
                                                            int block_size, const int* __restrict__ cu_k, const int* __restrict__ base,
                                                            bf16* __restrict__ out, int n_seq, int total, int pitch) {
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= total) return;
  int lo = 0, hi = n_seq - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_k[mid] <= i) lo = mid; else hi = mid - 1;
  }
  const int pos = base[lo] + i - cu_k[lo];
  const long long slot = static_cast<long long>(block_table[static_cast<long long>(lo) * max_blocks + pos / block_size]) * block_size + pos % block_size;
  const uint4* src = reinterpret_cast<const uint4*>(cache + slot * pitch);
  uint4* dst = reinterpret_cast<uint4*>(out + static_cast<long long>(i) * pitch);
  for (int c = lane; c < pitch / 8; c += 32) dst[c] = src[c];
}

// grid (N / (32·NW), H, ceil(T / 64)), 128 threads; warp = 8·NW output columns, all token tiles.  NK: w [H, N, K], else [H, K, N].
template <bool NK, int NW>
__global__ void __launch_bounds__(128) head_linear_mma_kernel(const bf16* __restrict__ x, long long x_t, long long x_h,
                                                              const bf16* __restrict__ w, bf16* __restrict__ y, long long y_t, long long y_h,
                                                              int T, int N, int K, const bf16* __restrict__ gate, long long gate_ld) {
  constexpr int TN = 32 * NW, S = NW == 2 ? 2 : 3, XP = 72, WP = NK ? 72 : TN + 8, WR = NK ? TN : 64;
  __shared__ __align__(16) bf16 sx[S][64 * XP];
  __shared__ __align__(16) bf16 sw[S][WR * WP];
  pdl_trigger();
  const int h = blockIdx.y, n0 = blockIdx.x * TN, t0 = blockIdx.z * 64;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nt = min(64, T - t0), mt = (nt + 15) / 16;
  const bf16* wh = w + static_cast<long long>(h) * N * K;
  const bf16* xh = x + t0 * x_t + h * x_h;
  const int chunks = (K + 63) / 64;
  auto load = [&](int c) {
    if (c < chunks) {
      const int st = c % S, k0 = c * 64;
      for (int i = threadIdx.x; i < mt * 16 * 8; i += 128) {
        const int r = i >> 3, cc = (i & 7) * 8;
        const bool ok = r < nt && k0 + cc < K;
        cp16(&sx[st][r * XP + cc], ok ? xh + r * x_t + k0 + cc : xh, ok);
      }
      if (NK) {
        for (int i = threadIdx.x; i < TN * 8; i += 128) {
          const int r = i >> 3, cc = (i & 7) * 8;
          const bool ok = n0 + r < N && k0 + cc < K;
          cp16(&sw[st][r * WP + cc], ok ? wh + static_cast<long long>(n0 + r) * K + k0 + cc : wh, ok);
        }
      } else {
        for (int i = threadIdx.x; i < 64 * (TN / 8); i += 128) {
          const int r = i / (TN / 8), cc = (i % (TN / 8)) * 8;
          const bool ok = k0 + r < K && n0 + cc < N;
          cp16(&sw[st][r * WP + cc], ok ? wh + static_cast<long long>(k0 + r) * N + n0 + cc : wh, ok);
        }
      }
    }
    cp_commit();
  };
  pdl_wait();
  for (int c = 0; c < S - 1; ++c) load(c);
  float acc[4][NW][4] = {};
  for (int c = 0; c < chunks; ++c) {
    cp_wait<S - 2>();
    __syncthreads();
    load(c + S - 1);
    const bf16* tx = sx[c % S];
    const bf16* tw = sw[c % S];
#pragma unroll
    for (int kk = 0; kk < 64; kk += 32) {
      // B fragments of two k steps: b[step][tile] pairs
      uint32_t b[2][NW][2];
#pragma unroll
      for (int nw = 0; nw < NW; ++nw) {
        const int n = warp * 8 * NW + nw * 8;
        uint32_t r[4];
        if (NK) ldsm4(s_addr(tw + (n + (lane & 7)) * WP + kk + (lane >> 3) * 8), r);
        else ldsm4t(s_addr(tw + (kk + lane) * WP + n), r);
        b[0][nw][0] = r[0]; b[0][nw][1] = r[1]; b[1][nw][0] = r[2]; b[1][nw][1] = r[3];
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        if (m < mt) {
#pragma unroll
          for (int st = 0; st < 2; ++st) {
            uint32_t a[4];
            ldsm4(s_addr(tx + (m * 16 + (lane & 15)) * XP + kk + st * 16 + (lane >> 4) * 8), a);
#pragma unroll
            for (int nw = 0; nw < NW; ++nw) mma(acc[m][nw], a, b[st][nw][0], b[st][nw][1]);
          }
        }
      }
    }
  }
  cp_wait<0>();
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int nw = 0; nw < NW; ++nw)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = m * 16 + half * 8 + (lane >> 2), n = n0 + warp * 8 * NW + nw * 8 + (lane & 3) * 2;
        if (t < nt && n < N) {                  // N is even
          bf16* dst = y + (t0 + t) * y_t + h * y_h + n;
          if (gate != nullptr) {
            const bf16* g = gate + (t0 + t) * gate_ld + h * N + n;
            acc[m][nw][half * 2] *= mx::sigmoid_t<bf16>(__bfloat162float(g[0]));
            acc[m][nw][half * 2 + 1] *= mx::sigmoid_t<bf16>(__bfloat162float(g[1]));
          }
          *reinterpret_cast<uint32_t*>(dst) = pack2(acc[m][nw][half * 2], acc[m][nw][half * 2 + 1]);
        }
      }
}

// grid (splits, head groups of 16·MT, tokens), 512 threads.  Warp = (head tile, column group): scores of its head tile for its share
// of the 64 keys of a tile, then its share of the latent columns of P·C.
template <int MT>
struct Dec {
  static constexpr int TK = 64, NG = 16 / MT, HT = 16 * MT, KH = NG / 4;      // 4 groups of 16 keys × KH row parts
  static constexpr int NT16 = (32 + NG - 1) / NG;                       // latent columns per warp in 16s (rank ≤ 512)
  static constexpr int SP = TK + 4, PP = TK + 8;
  static size_t bytes(int pitch) {
    return static_cast<size_t>(HT + 2 * TK) * (pitch + 8) * 2 + KH * HT * SP * 4 + 2 * HT * PP * 2 + HT * 4;
  }
};

template <int MT>
__global__ void __launch_bounds__(512) latent_decode_kernel(const bf16* __restrict__ q, const bf16* __restrict__ cache,
                                                            const int* __restrict__ block_table, int max_blocks, int block_size,
                                                            const int* __restrict__ token_seq, const int* __restrict__ positions,
                                                            const long long* __restrict__ slots, float* __restrict__ part_o,
                                                            float* __restrict__ part_ml, float scale, int window, int num_splits,
                                                            int num_blocks, MbLatent L) {
  using G = Dec<MT>;
  constexpr int TK = G::TK, NG = G::NG, HT = G::HT;
  extern __shared__ __align__(128) uint8_t smem[];
  const int rp = L.pitch + 8;                                           // shared row length: an odd number of 16-byte pieces
  bf16* sq = reinterpret_cast<bf16*>(smem);                             // [HT][rp]
  bf16* sk = sq + HT * rp;                                              // [2][TK][rp]
  float* ss = reinterpret_cast<float*>(sk + 2 * TK * rp);               // [HT][SP] scores
  bf16* sph = reinterpret_cast<bf16*>(ss + G::KH * HT * G::SP);                 // [HT][PP] P_hi, then P_lo
  bf16* spl = sph + HT * G::PP;
  float* sa = reinterpret_cast<float*>(spl + HT * G::PP);               // [HT] rescale factors of the current tile
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.z;
  const int split = blockIdx.x, h0 = blockIdx.y * HT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int mt = warp / NG, ng = warp % NG;
  const bool pad = slots[t] < 0;
  const int pos = pad ? -1 : positions[t];
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int n_keys = pos + 1 - lo;
  const int per = ((n_keys + num_splits - 1) / num_splits + TK - 1) / TK * TK;      // keys per split, whole tiles
  const int k_begin = lo + split * per, k_end = min(pos + 1, k_begin + per);
  const int n_tiles = k_end > k_begin ? (k_end - k_begin + TK - 1) / TK : 0;
  const int* bt = block_table + static_cast<long long>(token_seq != nullptr ? token_seq[t] : t) * max_blocks;
  const int pieces = L.pitch / 8;
  // lane j < 4 of a warp looks up the page of its j-th row of a tile, one tile before the tile is copied
  auto lookup = [&](int i) -> long long {
    if (lane >= TK / 16) return -1;
    const int key = k_begin + i * TK + warp + lane * 16;
    if (key >= k_end) return -1;
    const long long blk = bt[key / block_size];
    return blk >= 0 && blk < num_blocks ? blk * block_size + key % block_size : -1;      // an entry outside the pool reads as zeros
  };
  long long next = n_tiles > 0 ? lookup(0) : -1;
  auto load_tile = [&](int i, int st) {
#pragma unroll
    for (int j = 0; j < TK / 16; ++j) {
      const long long slot = __shfl_sync(0xffffffffu, next, j);
      const bf16* src = cache + (slot >= 0 ? slot : 0) * L.pitch;
      bf16* dst = sk + (st * TK + warp + j * 16) * rp;
      for (int c = lane; c < pieces; c += 32) cp16(dst + c * 8, src + c * 8, slot >= 0);
    }
    cp_commit();
    if (i + 1 < n_tiles) next = lookup(i + 1);
  };
  if (n_tiles > 0) {
    for (int i = threadIdx.x; i < HT * pieces; i += 512) {
      const int r = i / pieces, c = i - r * pieces;
      const bool ok = h0 + r < L.heads;
      cp16(sq + r * rp + c * 8, ok ? q + (t * L.heads + h0 + r) * L.pitch + c * 8 : q, ok);
    }
    load_tile(0, 0);                                                    // queries and first tile in one group
  }
  const int n16 = L.rank_p / 16;                                        // 16-column tiles of the latent
  float o[G::NT16][2][4];
#pragma unroll
  for (int i = 0; i < G::NT16; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
  // softmax state of row `srow`, held by its 32 (MT 2: 16) consecutive threads
  constexpr int TPR = 512 / HT, KPT = TK / TPR;
  const int srow = threadIdx.x / TPR, sub = threadIdx.x % TPR;
  float m_run = -INFINITY, l_run = 0.f;
  const float sl2 = scale * kLog2e;
  for (int i = 0; i < n_tiles; ++i) {
    const int st = i & 1;
    if (i + 1 < n_tiles) {
      load_tile(i + 1, st ^ 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const bf16* tk = sk + st * TK * rp;
    // scores: head tile mt × keys [ng·TK/NG, …)
    // scores: 16 keys and a part (1/KH) of the row per warp — query fragments are the larger half of the shared-memory reads, and wide
    // key groups re-read them less often; the parts are added up in the softmax
    constexpr int KH = G::KH;
    const int kg = ng / KH, kh = ng % KH;
    float s[2][4] = {};
    const int steps = L.pitch / 16, per_h = (steps + KH - 1) / KH;
#pragma unroll 6
    for (int ks = kh * per_h; ks < min(steps, (kh + 1) * per_h); ++ks) {
      uint32_t a[4], b[4];
      ldsm4(s_addr(sq + (mt * 16 + (lane & 15)) * rp + ks * 16 + (lane >> 4) * 8), a);
      ldsm4(s_addr(tk + (kg * 16 + (lane & 7) + ((lane >> 4) << 3)) * rp + ks * 16 + ((lane >> 3) & 1) * 8), b);
      mma(s[0], a, b[0], b[1]);
      mma(s[1], a, b[2], b[3]);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      float* dst = ss + kh * HT * G::SP + (mt * 16 + (lane >> 2)) * G::SP + kg * 16 + n * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(dst) = make_float2(s[n][0], s[n][1]);
      *reinterpret_cast<float2*>(dst + 8 * G::SP) = make_float2(s[n][2], s[n][3]);
    }
    __syncthreads();
    {
      const int key0 = k_begin + i * TK;
      float v[KPT], mx = m_run;
#pragma unroll
      for (int j = 0; j < KPT; ++j) {
        const int c = j * TPR + sub;
        float x = ss[srow * G::SP + c];
#pragma unroll
        for (int k = 1; k < KH; ++k) x += ss[(k * HT + srow) * G::SP + c];
        v[j] = key0 + c < k_end ? x * sl2 : -INFINITY;
        mx = fmaxf(mx, v[j]);
      }
#pragma unroll
      for (int d = 1; d < TPR; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - mx);
      m_run = mx;                                                       // finite: every tile of a split has a key
      float rs = 0.f;
#pragma unroll
      for (int j = 0; j < KPT; ++j) {
        const float p = exp2f(v[j] - mx);
        rs += p;
        const bf16 hi = __float2bfloat16(p);
        sph[srow * G::PP + j * TPR + sub] = hi;
        spl[srow * G::PP + j * TPR + sub] = __float2bfloat16(p - __bfloat162float(hi));
      }
#pragma unroll
      for (int d = 1; d < TPR; d <<= 1) rs += __shfl_xor_sync(0xffffffffu, rs, d);
      l_run = l_run * alpha + rs;
      if (sub == 0) sa[srow] = alpha;
    }
    __syncthreads();
    const float a0 = sa[mt * 16 + (lane >> 2)], a1 = sa[mt * 16 + (lane >> 2) + 8];
    if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
      for (int n = 0; n < G::NT16; ++n)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          o[n][j][0] *= a0; o[n][j][1] *= a0;
          o[n][j][2] *= a1; o[n][j][3] *= a1;
        }
    }
#pragma unroll
    for (int ks = 0; ks < TK / 16; ++ks) {
      uint32_t ph[4], pl[4];
      ldsm4(s_addr(sph + (mt * 16 + (lane & 15)) * G::PP + ks * 16 + (lane >> 4) * 8), ph);
      ldsm4(s_addr(spl + (mt * 16 + (lane & 15)) * G::PP + ks * 16 + (lane >> 4) * 8), pl);
#pragma unroll
      for (int n = 0; n < G::NT16; ++n) {
        const int c16 = n * NG + ng;
        if (c16 < n16) {
          uint32_t b[4];
          ldsm4t(s_addr(tk + (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * rp + c16 * 16 + (lane >> 4) * 8), b);
          mma(o[n][0], ph, b[0], b[1]);
          mma(o[n][1], ph, b[2], b[3]);
          mma(o[n][0], pl, b[0], b[1]);
          mma(o[n][1], pl, b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
  // unnormalised partials and (maximum in log2 units, sum) per head and split
  if (sub == 0 && h0 + srow < L.heads) {
    float* ml = part_ml + ((t * L.heads + h0 + srow) * num_splits + split) * 2;
    ml[0] = m_run;
    ml[1] = l_run;
  }
  if (n_tiles == 0) return;
#pragma unroll
  for (int n = 0; n < G::NT16; ++n) {
    const int c16 = n * NG + ng;
    if (c16 >= n16) continue;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int head = h0 + mt * 16 + half * 8 + (lane >> 2), c = c16 * 16 + j * 8 + (lane & 3) * 2;
        if (head < L.heads)
          *reinterpret_cast<float2*>(part_o + ((t * L.heads + head) * num_splits + split) * L.rank_p + c) =
              make_float2(o[n][j][half * 2], o[n][j][half * 2 + 1]);
      }
  }
}

// grid (heads, tokens), 128 threads: combine the splits, add the sink to the denominator, write [rank] bf16
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                           const bf16* __restrict__ sink, bf16* __restrict__ out, int num_splits, MbLatent L) {
  pdl_trigger();
  pdl_wait();
  const long long th = static_cast<long long>(blockIdx.y) * L.heads + blockIdx.x;
  const int lane = threadIdx.x & 31;
  // lane = split: maximum, weight and denominator by warp reductions (every warp the same)
  const float2 ml = lane < num_splits ? *reinterpret_cast<const float2*>(part_ml + (th * num_splits + lane) * 2) : make_float2(-INFINITY, 0.f);
  const float sk = sink != nullptr ? __bfloat162float(sink[blockIdx.x]) * kLog2e : -INFINITY;
  float mm = fmaxf(ml.x, sk);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffffu, mm, o));
  const float w = ml.x == -INFINITY ? 0.f : exp2f(ml.x - mm);
  const float den = mx::warp_sum(ml.y * w) + (sink != nullptr ? exp2f(sk - mm) : 0.f);
  const float f = den > 0.f ? __fdiv_rn(w, den) : 0.f;
  // four columns per thread (rank_p is a multiple of 16): one round for 512
  const float* po = part_o + th * num_splits * L.rank_p;
  for (int c = threadIdx.x * 4; c - threadIdx.x * 4 < L.rank; c += 512) {
    float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < num_splits; ++s) {
      const float fs = __shfl_sync(0xffffffffu, f, s);
      if (fs > 0.f && c < L.rank_p) {               // an empty split wrote nothing
        const float4 v = *reinterpret_cast<const float4*>(po + s * L.rank_p + c);
        r.x = fmaf(fs, v.x, r.x);
        r.y = fmaf(fs, v.y, r.y);
        r.z = fmaf(fs, v.z, r.z);
        r.w = fmaf(fs, v.w, r.w);
      }
    }
    const float o[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (c + j < L.rank) out[th * L.rank + c + j] = __float2bfloat16(o[j]);
  }
}

template <int MT>
static cudaError_t decode(dim3 grid, cudaStream_t s, const bf16* q, const bf16* cache, const int* bt, int mbk, int bs, const int* seq, const int* pos,
                          const long long* slots, float* po, float* pml, float scale, int window, int splits, int nb, MbLatent L) {
  static bool once = false;
  if (!once) {
    const cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return e;
    once = true;
  }
  return launch_pdl(latent_decode_kernel<MT>, grid, dim3(512), Dec<MT>::bytes(L.pitch), s, q, cache, bt, mbk, bs, seq, pos, slots, po, pml, scale,
                    window, splits, nb, L);
}

}  // namespace ld
}  // namespace mb

using namespace mb;
using namespace mb::ld;

extern "C" int mb_latent_gather(const void* cache, const int* block_table, int max_blocks, int block_size, const int* cu_k, const int* base,
                                void* out, int n_seq, int total, int pitch, cudaStream_t s) {
  if (total <= 0) return 0;
  return static_cast<int>(launch_pdl(latent_gather_kernel, dim3((total + 7) / 8), dim3(256), 0, s, reinterpret_cast<const bf16*>(cache), block_table,
                                     max_blocks, block_size, cu_k, base, reinterpret_cast<bf16*>(out), n_seq, total, pitch));
}

// bf16, K % 8 == 0, N % 8 == 0, 16-byte aligned rows of x
extern "C" int mb_head_linear_mma(const void* x, long long x_t, long long x_h, const void* w, int w_nk, void* y, long long y_t, long long y_h, int T,
                                  int H, int N, int K, const void* gate, long long gate_ld, cudaStream_t s) {
  if (T <= 0) return 0;
  if (K % 8 || N % 8 || x_t % 8 || x_h % 8 || y_t % 2 || y_h % 2) return -3;
  const int zt = (T + 63) / 64;
  const bool wide = static_cast<long long>(H) * ((N + 63) / 64) * zt >= 296;      // two CTAs per SM even with 64-column tiles
  const dim3 grid(wide ? (N + 63) / 64 : (N + 31) / 32, H, zt);
  auto X = reinterpret_cast<const bf16*>(x);
  auto W = reinterpret_cast<const bf16*>(w);
  auto Y = reinterpret_cast<bf16*>(y);
  auto kern = w_nk ? (wide ? head_linear_mma_kernel<true, 2> : head_linear_mma_kernel<true, 1>)
                   : (wide ? head_linear_mma_kernel<false, 2> : head_linear_mma_kernel<false, 1>);
  const cudaError_t e = launch_pdl(kern, grid, dim3(128), 0, s, X, x_t, x_h, W, Y, y_t, y_h, T, N, K, reinterpret_cast<const bf16*>(gate), gate_ld);
  return static_cast<int>(e);
}

// part_o [T, H, splits, rank_p] and part_ml [T, H, splits, 2] fp32 scratch; bf16, rank ≤ 512, pitch ≤ 640.  Pages of a multiple of 64
// tokens go through the tcgen05 kernel (latent_decode_tc.cu), others through the mma.sync kernel above.
extern "C" int mb_latent_decode(const void* q, const void* cache, const int* block_table, int max_blocks, int block_size, const int* token_seq,
                                const int* positions, const long long* slots, const void* sink, float* part_o, float* part_ml, void* out,
                                int T, float scale, int window, int splits, int num_blocks, MbLatent L, int* error_flag, cudaStream_t s) {
  if (T <= 0) return 0;
  if (L.rank_p > 512 || L.pitch > 640 || T > 65535 || splits < 1 || splits > 32) return -3;
  if (block_size % 64 == 0) {
    const int rc = mb_latent_decode_tc(q, cache, block_table, max_blocks, block_size, token_seq, positions, slots, part_o, part_ml, T, scale,
                                       window, splits, num_blocks, L, error_flag, s);
    if (rc) return rc;
  } else {
    const int mt = L.heads > 16 && Dec<2>::bytes(L.pitch) <= 227 * 1024 ? 2 : 1;
    if (Dec<1>::bytes(L.pitch) > 227 * 1024) return -3;
    const dim3 grid(splits, (L.heads + 16 * mt - 1) / (16 * mt), T);
    auto Q = reinterpret_cast<const bf16*>(q);
    auto KC = reinterpret_cast<const bf16*>(cache);
    const cudaError_t e =
        mt == 2 ? decode<2>(grid, s, Q, KC, block_table, max_blocks, block_size, token_seq, positions, slots, part_o, part_ml, scale, window, splits, num_blocks, L)
                : decode<1>(grid, s, Q, KC, block_table, max_blocks, block_size, token_seq, positions, slots, part_o, part_ml, scale, window, splits, num_blocks, L);
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  return static_cast<int>(launch_pdl(latent_merge_kernel, dim3(L.heads, T), dim3(128), 0, s, static_cast<const float*>(part_o),
                                     static_cast<const float*>(part_ml), reinterpret_cast<const bf16*>(sink), reinterpret_cast<bf16*>(out), splits, L));
}
