// Prefill of the state-space mixer (see ssm_state.cu) in chunks of 64 tokens on tensor cores.
//
// Inside a chunk, with i, j the places of two of its tokens, L_i the sum of the log decays up to and with token i, and S the state before it,
//     y_i = e^{L_i} Sᵀ C_i + Σ_{j ≤ i} e^{L_i − L_j} dt_j (C_i·B_j) x_j + D x_i        S ← e^{L_n} S + Σ_j e^{L_n − L_j} dt_j B_j x_jᵀ
// Built like linear_chunk.cu: the state stays in fp32 registers; where it, the decayed scores and the decayed B enter a product they are
// split into two bf16 parts (hi + lo).  x, B and C are bf16 after their convolution.  What differs:
//   * the decay is a number per token and head, so its powers are exponentials of differences of a running sum, made per chunk;
//   * heads of a group share B and C: where two heads fit the 128 columns of a tile, a CTA takes two neighbouring heads of a group, and
//     tiles of B and C and the products C·B are read and computed once for both;
//   * D x and the gate silu(z) are applied on the way out.
//
// Long prompts are cut into segments so that one sequence fills the GPU:
//   1. ssm_chunk_kernel<false>   per (segment, heads): the state its tokens add, from zero, and its whole log decay
//   2. ssm_scan_kernel           per (sequence, head, element): state at the start of every segment
//   3. ssm_chunk_kernel<true>    per (segment, heads): outputs; a sequence's last segment writes its state slot
// With one segment per sequence only the third runs, straight from and to the state slots.
#include "mixers.cuh"

namespace mb {
namespace sc {

using mx::bf16;
static constexpr int C = 64, P = 136, PP = C + 8, kThreads = 512;      // tokens per chunk, shared row lengths
static constexpr int kTile = C * P;                                    // elements of a C / B / x tile (≤ 128 wide)
static constexpr int kLog = 2 * 2 * 2 * C;                             // floats: [stage][head][L | dt][C]
static constexpr size_t kSmemSums = 6 * kTile * 2 + kLog * 4;          // without state and scores: two CTAs per SM
static constexpr size_t smem_out(int heads) { return (6 * kTile + 2 * 128 * P + heads * 2 * C * PP) * 2 + kLog * 4; }

__device__ __forceinline__ uint32_t s_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void cp16(void* dst, const void* src, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s_addr(dst)), "l"(src), "r"(sz) : "memory");
}
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
__device__ __forceinline__ float lo16(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float hi16(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}
// (a, b) = hi + lo, two bf16 pairs
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack2(a, b);
  lo = pack2(a - lo16(hi), b - hi16(hi));
}

struct Args {
  const bf16* proj;          // z: [T, ld], columns h·V …
  long long ld;
  const bf16* xbc;           // [T, CH]: x [H, V], B [G, N], C [G, N]
  const float *dt, *la;      // [T, H]
  MbSsm m;
  const int* segs;           // [n_seg][4]: sequence, first token, end, 1 if the sequence's last segment
  float* seg_state;          // [n_seg, H, N, V]; null: one segment per sequence
  float* seg_decay;          // [n_seg, H]
  bf16* out;                 // [T, H·V]
};

// grid (heads / HP, segments), 512 threads.  HP heads per CTA side by side in the 128 columns of a tile (HP = 2: V ≤ 64, V % 16 == 0).
template <bool OUT, int HP>
__global__ void __launch_bounds__(kThreads, OUT ? 1 : 2) ssm_chunk_kernel(Args a) {
  extern __shared__ __align__(128) uint8_t smem[];
  bf16* tile = reinterpret_cast<bf16*>(smem);        // [2][C | B | x][C][P]
  bf16* s_hi = tile + 6 * kTile;                     // [128][P]
  bf16* s_lo = s_hi + 128 * P;
  bf16* p_hi = s_lo + 128 * P;                       // [HP][C][PP]
  bf16* p_lo = p_hi + HP * C * PP;
  float* lg = reinterpret_cast<float*>(OUT ? p_lo + HP * C * PP : s_hi);   // [2][HP][L | dt][C]
  mb::pdl_trigger();
  mb::pdl_wait();
  const int N = a.m.N, V = a.m.V, H = a.m.H, G = a.m.G, inner = H * V, CH = inner + 2 * G * N;
  const int h0 = blockIdx.x * HP, seg = blockIdx.y, grp = h0 / (H / G);
  const int seq = a.segs[seg * 4], t0 = a.segs[seg * 4 + 1], t1 = a.segs[seg * 4 + 2], last = a.segs[seg * 4 + 3];
  if (!OUT && last) return;                          // nobody continues from a last segment's own sum
  const int slot = a.m.slots[seq];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int W = HP * V, kn = (N + 15) / 16;          // columns of x in a tile; 16-wide steps of N
  const bf16* src[3] = {a.xbc + inner + (G + grp) * N, a.xbc + inner + grp * N, a.xbc + h0 * V};
  // columns [width, 16·⌈width/16⌉) of the tiles are zero for good
  for (int i = threadIdx.x; i < 6 * C; i += kThreads) {
    const int w = (i / C) % 3 == 2 ? W : N;
    bf16* row = tile + i * P;
    for (int c = w; c < (w + 15) / 16 * 16; ++c) row[c] = __float2bfloat16(0.f);
  }
  const int pn = N / 8, pv = W / 8, n_piece = OUT ? C * (2 * pn + pv) : C * (pn + pv);
  auto load = [&](int c, int st) {
    const int tb = t0 + c * C;
    for (int i = threadIdx.x; i < n_piece; i += kThreads) {
      int which, j = i, w = pn;
      if (OUT && j < C * pn) which = 0;
      else {
        if (OUT) j -= C * pn;
        if (j < C * pn) which = 1;
        else { j -= C * pn; which = 2; w = pv; }
      }
      const int r = j / w, col = (j % w) * 8;
      const bool ok = tb + r < t1;
      cp16(tile + (st * 3 + which) * kTile + r * P + col, src[which] + static_cast<long long>(ok ? tb + r : t0) * CH + col, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // running sums of the log decays of chunk c: warp hp does head hp, two neighbouring tokens per lane (tokens behind the end: 0, step 0)
  auto logs = [&](int c, int st) {
    if (warp >= HP) return;
    const int t = t0 + c * C + 2 * lane;
    const long long at = static_cast<long long>(t) * H + h0 + warp;
    const float l0 = t < t1 ? a.la[at] : 0.f, l1 = t + 1 < t1 ? a.la[at + H] : 0.f;
    float s = l0 + l1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += v;
    }
    float* dst = lg + (st * HP + warp) * 2 * C + 2 * lane;
    const float before = __shfl_up_sync(0xffffffffu, s, 1);
    dst[0] = (lane > 0 ? before : 0.f) + l0;
    dst[1] = s;
    dst[C] = t < t1 ? a.dt[at] : 0.f;
    dst[C + 1] = t + 1 < t1 ? a.dt[at + H] : 0.f;
  };
  load(0, 0);
  // state: warp = (16 rows rt of N, column block ch: head ch of two, or 64 columns of one); n-th 8-column tile of the block
  const int rt = warp >> 1, ch = warp & 1;
  const int cb = HP == 2 ? ch * V : ch * 64, cw = HP == 2 ? V : min(64, V - ch * 64);      // first column of the block, its width (≤ 0: none)
  const int ct = (cw + 15) / 16;                                                            // 16-column steps of the block
  const int hs = HP == 2 ? ch : 0;                                                          // head of the block
  float s[8][4];
  const long long sz = static_cast<long long>(N) * V;
  auto state_at = [&](float* base, int r, int c) { return base + hs * sz + static_cast<long long>(r) * V + (HP == 2 ? c - cb : c); };
  float* slot_p = a.m.state + (static_cast<long long>(slot) * H + h0) * sz;
  float* seg_p = a.seg_state != nullptr ? a.seg_state + (static_cast<long long>(seg) * H + h0) * sz : nullptr;
  float* init = !OUT ? nullptr : seg_p != nullptr ? seg_p : a.m.positions[t0] > 0 ? slot_p : nullptr;
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = rt * 16 + half * 8 + g, c = n * 8 + t4 * 2;
      float2 v = make_float2(0.f, 0.f);
      if (init != nullptr && r < N && c < cw) v = *reinterpret_cast<const float2*>(state_at(init, r, cb + c));
      s[n][half * 2] = v.x;
      s[n][half * 2 + 1] = v.y;
    }
  // scores: warp = (16 tokens mt, quarter cq of the keys); outputs: quarter cq of a head's columns, or half of one of two heads'
  const int mt = warp >> 2, cq = warp & 3;
  const int ho = HP == 2 ? cq >> 1 : 0, oc = HP == 2 ? ho * V + (cq & 1) * 32 : cq * 32;    // head and first column of the outputs
  const int ow = HP == 2 ? V - (cq & 1) * 32 : V - cq * 32;                                 // columns left there
  const int chunks = (t1 - t0 + C - 1) / C;
  auto publish_state = [&]() {
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      if (n * 8 >= ct * 16) break;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = rt * 16 + half * 8 + g, c = cb + n * 8 + t4 * 2;
        uint32_t hi, lo;
        split2(s[n][half * 2], s[n][half * 2 + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(s_hi + r * P + c) = hi;
        *reinterpret_cast<uint32_t*>(s_lo + r * P + c) = lo;
      }
    }
  };
  // Two barriers per chunk: [scores and Sᵀ C] | [P·x, state update, state published, next chunk's decays]; the copy of the next chunk runs
  // from the first barrier to the end of the second phase.
  logs(0, 0);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  if (OUT) publish_state();
  float total = 0.f;                                  // log decay of the segment so far (head hs)
  for (int ci = 0; ci < chunks; ++ci) {
    const int st = ci & 1, n_tok = min(C, t1 - t0 - ci * C);
    bf16* tc = tile + st * 3 * kTile;
    bf16* tb = tc + kTile;
    bf16* tx = tb + kTile;
    const float* L = lg + st * HP * 2 * C;            // head hp: L + hp·2C, its step sizes C behind
    __syncthreads();
    if (ci + 1 < chunks) load(ci + 1, st ^ 1);
    float o[4][4];
#pragma unroll
    for (int n = 0; n < 4; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    if (OUT) {
      // the gates of this warp's outputs are on their way during the products
      uint32_t z[4][2];
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = mt * 16 + half * 8 + g, c = n * 8 + t4 * 2;
          z[n][half] = i < n_tok && c < ow ? *reinterpret_cast<const uint32_t*>(a.proj + static_cast<long long>(t0 + ci * C + i) * a.ld + h0 * V + oc + c) : 0u;
        }
      float sc[2][4] = {};
      const bool seen = cq <= mt;                    // some key of the quarter is not after every token of the tile
      for (int ks = 0; ks < kn; ++ks) {
        uint32_t aq[4], b[4];
        ldsm4(s_addr(tc + (mt * 16 + (lane & 15)) * P + ks * 16 + (lane >> 4) * 8), aq);
        if (seen) {
          ldsm4(s_addr(tb + (cq * 16 + (lane & 7) + ((lane >> 4) << 3)) * P + ks * 16 + ((lane >> 3) & 1) * 8), b);
          mma(sc[0], aq, b[0], b[1]);
          mma(sc[1], aq, b[2], b[3]);
        }
        const int srow = ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          if (n * 16 < ow) {
            const int off = srow * P + oc + n * 16 + (lane >> 4) * 8;
            ldsm4t(s_addr(s_hi + off), b);
            mma(o[2 * n], aq, b[0], b[1]);
            mma(o[2 * n + 1], aq, b[2], b[3]);
            ldsm4t(s_addr(s_lo + off), b);
            mma(o[2 * n], aq, b[0], b[1]);
            mma(o[2 * n + 1], aq, b[2], b[3]);
          }
        }
      }
      const float d0 = __expf(L[ho * 2 * C + mt * 16 + g]), d1 = __expf(L[ho * 2 * C + mt * 16 + g + 8]);
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        o[n][0] *= d0; o[n][1] *= d0;
        o[n][2] *= d1; o[n][3] *= d1;
      }
      if (seen) {
#pragma unroll
        for (int hp = 0; hp < HP; ++hp) {
          const float* Lh = L + hp * 2 * C;
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const int j = cq * 16 + n * 8 + t4 * 2;
            const float2 lj = *reinterpret_cast<const float2*>(Lh + j), dj = *reinterpret_cast<const float2*>(Lh + C + j);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
              const int i = mt * 16 + half * 8 + g;
              const float li = Lh[i];
              uint32_t hi, lo;
              split2(j <= i ? sc[n][half * 2] * __expf(li - lj.x) * dj.x : 0.f, j + 1 <= i ? sc[n][half * 2 + 1] * __expf(li - lj.y) * dj.y : 0.f, hi, lo);
              *reinterpret_cast<uint32_t*>(p_hi + (hp * C + i) * PP + j) = hi;
              *reinterpret_cast<uint32_t*>(p_lo + (hp * C + i) * PP + j) = lo;
            }
          }
        }
      }
      __syncthreads();
      for (int ks = 0; ks <= mt; ++ks) {
        uint32_t ph[4], pl[4], b[4];
        const int off = (ho * C + mt * 16 + (lane & 15)) * PP + ks * 16 + (lane >> 4) * 8;
        ldsm4(s_addr(p_hi + off), ph);
        ldsm4(s_addr(p_lo + off), pl);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          if (n * 16 < ow) {
            ldsm4t(s_addr(tx + (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * P + oc + n * 16 + (lane >> 4) * 8), b);
            mma(o[2 * n], ph, b[0], b[1]);
            mma(o[2 * n + 1], ph, b[2], b[3]);
            mma(o[2 * n], pl, b[0], b[1]);
            mma(o[2 * n + 1], pl, b[2], b[3]);
          }
        }
      }
      const float D = mx::to_f(reinterpret_cast<const bf16*>(a.m.D)[h0 + ho]);
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = mt * 16 + half * 8 + g, c = n * 8 + t4 * 2;
          if (i < n_tok && c < ow) {
            const uint32_t x = *reinterpret_cast<const uint32_t*>(tx + i * P + oc + c);
            const float y0 = fmaf(D, lo16(x), o[n][half * 2]), y1 = fmaf(D, hi16(x), o[n][half * 2 + 1]);
            *reinterpret_cast<uint32_t*>(a.out + static_cast<long long>(t0 + ci * C + i) * inner + h0 * V + oc + c) =
                pack2(y0 * mx::silu_t<bf16>(lo16(z[n][half])), y1 * mx::silu_t<bf16>(hi16(z[n][half])));
          }
        }
    }
    // S ← e^{L_n} S + (e^{L_n − L_j} dt_j B_j)ᵀ x: B is decayed and split in registers
    const float* Ls = L + hs * 2 * C;
    const float Ln = Ls[C - 1];                       // tokens behind the end do not decay
    total += Ln;
    if (rt < kn && cw > 0) {
      const float dn = __expf(Ln);
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        s[n][0] *= dn; s[n][1] *= dn; s[n][2] *= dn; s[n][3] *= dn;
      }
#pragma unroll
      for (int ks = 0; ks < C / 16; ++ks) {
        uint32_t kt[4], kh[4], kl[4], b[4];
        ldsm4t(s_addr(tb + (ks * 16 + ((lane >> 4) << 3) + (lane & 7)) * P + rt * 16 + ((lane >> 3) & 1) * 8), kt);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float2 l = *reinterpret_cast<const float2*>(Ls + ks * 16 + j * 8 + t4 * 2), d = *reinterpret_cast<const float2*>(Ls + C + ks * 16 + j * 8 + t4 * 2);
          const float f0 = __expf(Ln - l.x) * d.x, f1 = __expf(Ln - l.y) * d.y;
          split2(lo16(kt[2 * j]) * f0, hi16(kt[2 * j]) * f1, kh[2 * j], kl[2 * j]);
          split2(lo16(kt[2 * j + 1]) * f0, hi16(kt[2 * j + 1]) * f1, kh[2 * j + 1], kl[2 * j + 1]);
        }
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          if (n < ct) {
            ldsm4t(s_addr(tx + (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * P + cb + n * 16 + (lane >> 4) * 8), b);
            mma(s[2 * n], kh, b[0], b[1]);
            mma(s[2 * n + 1], kh, b[2], b[3]);
            mma(s[2 * n], kl, b[0], b[1]);
            mma(s[2 * n + 1], kl, b[2], b[3]);
          }
        }
      }
    }
    if (ci + 1 < chunks) {
      if (OUT) publish_state();
      logs(ci + 1, st ^ 1);
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
  }
  if (!OUT && rt == 0 && lane == 0 && (HP == 2 || ch == 0)) a.seg_decay[static_cast<long long>(seg) * H + h0 + hs] = total;
  float* dst = OUT ? (last ? slot_p : nullptr) : seg_p;
  if (dst == nullptr || (OUT && slot < 0)) return;
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = rt * 16 + half * 8 + g, c = n * 8 + t4 * 2;
      if (r < N && c < cw) *reinterpret_cast<float2*>(state_at(dst, r, cb + c)) = make_float2(s[n][half * 2], s[n][half * 2 + 1]);
    }
}

// grid (elements / 1024, heads, sequences): seg_state[i] ← state before segment i (4 elements per thread)
__global__ void __launch_bounds__(256) ssm_scan_kernel(MbSsm m, const int* __restrict__ segs, const int* __restrict__ seq_segs, float* seg_state,
                                                       const float* __restrict__ seg_decay, int sz) {
  mb::pdl_trigger();
  mb::pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z, H = m.H;
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (e >= sz) return;
  const int s0 = seq_segs[b], s1 = seq_segs[b + 1];
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (m.positions[segs[s0 * 4 + 1]] > 0) S = *reinterpret_cast<const float4*>(m.state + (static_cast<long long>(m.slots[b]) * H + h) * sz + e);
  constexpr int U = 4;
  for (int i0 = s0; i0 < s1; i0 += U) {
    float4 add[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i0 + u < s1 - 1) add[u] = *reinterpret_cast<const float4*>(seg_state + (static_cast<long long>(i0 + u) * H + h) * sz + e);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u;
      if (i >= s1) break;
      *reinterpret_cast<float4*>(seg_state + (static_cast<long long>(i) * H + h) * sz + e) = S;
      if (i < s1 - 1) {
        const float d = __expf(seg_decay[static_cast<long long>(i) * H + h]);
        S.x = fmaf(d, S.x, add[u].x);
        S.y = fmaf(d, S.y, add[u].y);
        S.z = fmaf(d, S.z, add[u].z);
        S.w = fmaf(d, S.w, add[u].w);
      }
    }
  }
}

template <int HP>
static cudaError_t run(const Args& a, const int* seq_segs, int n_seq, int n_seg, cudaStream_t s) {
  static bool once = false;
  if (!once) {
    cudaError_t e = cudaFuncSetAttribute(ssm_chunk_kernel<true, HP>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem_out(HP)));
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(ssm_chunk_kernel<false, HP>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kSmemSums));
    if (e != cudaSuccess) return e;
    once = true;
  }
  cudaError_t e = cudaSuccess;
  const dim3 grid(a.m.H / HP, n_seg);
  if (a.seg_state != nullptr) {
    e = launch_pdl(ssm_chunk_kernel<false, HP>, grid, dim3(kThreads), kSmemSums, s, a);
    if (e == cudaSuccess)
      e = launch_pdl(ssm_scan_kernel, dim3((a.m.N * a.m.V + 1023) / 1024, a.m.H, n_seq), dim3(256), 0, s, a.m, a.segs, seq_segs, a.seg_state,
                     static_cast<const float*>(a.seg_decay), a.m.N * a.m.V);
  }
  if (e == cudaSuccess) e = launch_pdl(ssm_chunk_kernel<true, HP>, grid, dim3(kThreads), smem_out(HP), s, a);
  return e;
}

}  // namespace sc
}  // namespace mb

using namespace mb;

extern "C" int mb_ssm_heads_per_cta(int H, int V, int G) { return V <= 64 && V % 16 == 0 && (H / G) % 2 == 0 ? 2 : 1; }

extern "C" int mb_ssm_chunk(const void* proj, long long ld, const void* xbc, const float* dt, const float* la, MbSsm m, const int* segs,
                            const int* seq_segs, float* seg_state, float* seg_decay, void* out, int n_seq, int n_seg, cudaStream_t s) {
  if (n_seg <= 0) return 0;
  if (m.N % 8 || m.V % 8 || m.N > 128 || m.V > 128 || ld % 2 || m.G <= 0 || m.H % m.G || n_seg > 65535 || n_seq > 65535) return -3;
  sc::Args a{reinterpret_cast<const sc::bf16*>(proj), ld, reinterpret_cast<const sc::bf16*>(xbc), dt, la, m, segs, seg_state, seg_decay,
             reinterpret_cast<sc::bf16*>(out)};
  return static_cast<int>(mb_ssm_heads_per_cta(m.H, m.V, m.G) == 2 ? sc::run<2>(a, seq_segs, n_seq, n_seg, s) : sc::run<1>(a, seq_segs, n_seq, n_seg, s));
}
