// Prefill attention on tcgen05 tensor cores over a paged cache of keys and values: causal, with a sliding window that keeps the first
// tokens and a softmax sink per head; grouped queries.
//
// Structure of the other prefill kernels (attention_tc.cu, attention_latent_tc.cu): 192 threads — a TMA warp, an MMA warp, four softmax
// warps with one thread per query row — two CTAs per SM, softmax weights as two bf16 parts in tensor memory over their scores.
// What differs:
//   * the 128 rows of a tile are (token, head) pairs: 128 / group tokens of all query heads that share a key head, fetched by one 3-D
//     box, so that a tile reads its window once for the whole group and a narrow window wastes few keys;
//   * keys and values come straight from their pages: a tile of 64 positions is one box of a page of ≥ 64 tokens (or several boxes
//     of smaller pages).  What a box reads past a head's own columns meets zero query columns or is never stored; rows of a page behind
//     the sequence's end are masked;
//   * differential attention (MbDiff): heads 2h and 2h + 1 are neighbouring rows; their threads exchange the two maps' outputs, and the
//     difference is normed and gated on its way out;
//   * the key tiles of a query tile are those of the kept first tokens and those of the window, or of its tokens' chunks; what lies
//     between is skipped;
//   * BIAS: r1 · ln(1 + r2 · distance) comes off the scores; outputs may pass a gate (MbScores).
#include "launch.h"
#include "ptx.cuh"

namespace mb {

int make_tmap_bf16_2d(CUtensorMap* out, const void* base, long long rows, long long cols, long long ld, int box_rows, int box_cols);
int make_tmap_bf16_3d(CUtensorMap* out, const void* base, long long outer, long long mid, long long cols, int box_outer, int box_mid,
                      int box_cols);

namespace fw {

static constexpr int BQ = 128, BKV = 64;
static constexpr int kQAtom = BQ * 128, kKVAtom = BKV * 128;      // bytes of a 64-column atom
static constexpr uint32_t kTmemCols = 256;                        // S0 | S1 (64 each) | O (128)
static constexpr float kLog2e = 1.4426950408889634f;

struct Params {
  __nv_bfloat16* o;            // [tokens], rows of o_row elements
  long long o_row;
  const __nv_bfloat16* sink;   // [heads] or null
  const int* cu_q;
  const int* positions;        // of the packed tokens
  const int* block_table;
  int max_blocks, block_size, box_rows;
  int group, tokens;           // query heads per key head, tokens per tile
  int dim, vdim;
  float scale;
  int window, keep, chunk;     // window 0: all earlier keys, or those of a chunk
  MbScores x;
  MbDiff diff;
  int* error_flag;
};

template <int NA, int NV>
struct Cfg {
  static constexpr int kQBytes = NA * kQAtom, kKBytes = NA * kKVAtom, kVBytes = NV * kKVAtom;
  static constexpr int q = 0, k = kQBytes, v = k + 2 * kKBytes, bars = v + 2 * kVBytes, total = bars + 256;
};

template <int NA, int NV, bool BIAS>
__global__ void __launch_bounds__(192, 2)
window_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                      Params p) {
  using G = Cfg<NA, NV>;
  extern __shared__ __align__(1024) uint8_t smem[];
  if (smem_u32(smem) & 1023u) {   // swizzled tiles need 1024-byte alignment
    if (threadIdx.x == 0) atomicExch(p.error_flag, 85);
    return;
  }
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + G::bars);
  uint64_t* q_full = bars;            // 1
  uint64_t* k_full = bars + 1;        // 2
  uint64_t* k_empty = bars + 3;       // 2
  uint64_t* v_full = bars + 5;        // 2
  uint64_t* v_empty = bars + 7;       // 2
  uint64_t* s_full = bars + 9;        // 2
  uint64_t* p_ready = bars + 13;      // 1
  uint64_t* pv_done = bars + 14;      // 1
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, hk = blockIdx.y;
  const int q_start = p.cu_q[b], L = p.cu_q[b + 1] - q_start;
  const int t0 = (gridDim.x - 1 - blockIdx.x) * p.tokens;      // late query tiles (long key ranges) first
  if (t0 >= L) return;
  const int first_pos = p.positions[q_start] + t0;             // positions of the tile's tokens: first_pos … last_pos
  const int last_pos = first_pos + min(p.tokens, L - t0) - 1;
  auto first_key = [&](int pos) { return p.window > 0 ? pos - p.window + 1 : p.chunk > 0 ? pos - pos % p.chunk : 0; };
  const int win_tile = max(0, first_key(first_pos)) / BKV;
  const int n_keep = p.window > 0 ? min((p.keep + BKV - 1) / BKV, win_tile) : 0;
  const int n_blocks = n_keep + last_pos / BKV + 1 - win_tile;
  auto key_of = [&](int j) { return (j < n_keep ? j : win_tile + j - n_keep) * BKV; };

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    mbar_init(p_ready, 4);
    mbar_init(pv_done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_ptr, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_ptr;
  const uint32_t tmem_o = tmem + 128;

  if (warp == 0) {
    if (elect_one()) {
      const int* bt = p.block_table + static_cast<long long>(b) * p.max_blocks;
      // 64 key positions from kv0 on: `atoms` column blocks from column c0 on.  Positions behind the last page read page 0 (masked)
      auto load_rows = [&](uint8_t* dst, const CUtensorMap* tm, uint64_t* bar, int kv0, int c0, int atoms) {
        for (int r = 0; r < BKV; r += p.box_rows) {
          const int key = kv0 + r, page = key / p.block_size;
          const int row = key <= last_pos && page < p.max_blocks ? bt[page] * p.block_size + key % p.block_size : 0;
          for (int a = 0; a < atoms; ++a) tma_load_2d(dst + a * kKVAtom + r * 128, tm, bar, c0 + a * 64, row);
        }
      };
      auto load_k = [&](int j) -> bool {
        const int st = j & 1;
        if (!mbar_wait(&k_empty[st], ((j >> 1) & 1) ^ 1)) return false;
        mbar_expect_tx(&k_full[st], G::kKBytes);
        load_rows(smem + G::k + st * G::kKBytes, &tm_k, &k_full[st], key_of(j), hk * p.dim, NA);
        return true;
      };
      mbar_expect_tx(q_full, NA * p.tokens * p.group * 128);
      for (int a = 0; a < NA; ++a) tma_load_3d(smem + G::q + a * kQAtom, &tm_q, q_full, a * 64, hk * p.group, q_start + t0);
      bool ok = load_k(0);
      for (int j = 0; j < n_blocks && ok && !*abort_flag; ++j) {
        if (j + 1 < n_blocks) ok = load_k(j + 1);
        const int st = j & 1;
        if (!ok || !mbar_wait(&v_empty[st], ((j >> 1) & 1) ^ 1)) { ok = false; break; }
        mbar_expect_tx(&v_full[st], G::kVBytes);
        load_rows(smem + G::v + st * G::kVBytes, &tm_v, &v_full[st], key_of(j), hk * p.vdim, NV);
      }
      if (!ok) { *abort_flag = 1; atomicExch(p.error_flag, 81); }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc_s = make_idesc_bf16(BQ, BKV, 0, 0);       // S = Q (K-major) · K (K-major)
      constexpr uint32_t idesc_o = make_idesc_bf16(BQ, NV * 64, 0, 1);   // O = P (tensor memory) · V (MN-major)
      const uint32_t q_addr = smem_u32(smem + G::q);
      auto issue_s = [&](int j) -> bool {
        const int st = j & 1;
        if (!mbar_wait(&k_full[st], (j >> 1) & 1)) return false;
        tc_fence_after();
        const uint32_t k_addr = smem_u32(smem + G::k + st * G::kKBytes);
        // the buffer last held P_{j−2}; its product was issued before this one by the same thread, and MMAs run in issue order
#pragma unroll
        for (int ks = 0; ks < NA * 4; ++ks)
          umma_bf16(tmem + st * BKV, make_smem_desc_sw128(q_addr + (ks >> 2) * kQAtom + (ks & 3) * 32, 16, 1024),
                    make_smem_desc_sw128(k_addr + (ks >> 2) * kKVAtom + (ks & 3) * 32, 16, 1024), idesc_s, ks != 0);
        umma_commit(&s_full[st]);
        umma_commit(&k_empty[st]);
        return true;
      };
      bool ok = mbar_wait(q_full, 0);
      if (ok) ok = issue_s(0);
      for (int j = 0; j < n_blocks && ok && !*abort_flag; ++j) {
        if (j + 1 < n_blocks) ok = issue_s(j + 1);
        if (!ok) break;
        const int st = j & 1;
        if (!mbar_wait(&v_full[st], (j >> 1) & 1) || !mbar_wait(p_ready, j & 1)) { ok = false; break; }
        tc_fence_after();
        const uint32_t v_addr = smem_u32(smem + G::v + st * G::kVBytes);
#pragma unroll
        for (int part = 0; part < 2; ++part)        // P_hi, then P_lo
#pragma unroll
          for (int ks = 0; ks < BKV / 16; ++ks)
            umma_bf16_ts(tmem_o, tmem + st * BKV + part * 32 + ks * 8, make_smem_desc_sw128(v_addr + ks * (16 * 128), kKVAtom, 1024), idesc_o,
                         (j | part | ks) != 0);
        umma_commit(&v_empty[st]);
        umma_commit(pv_done);
      }
      if (!ok) { *abort_flag = 1; atomicExch(p.error_flag, 82); }
    }
  } else {
    const int q4 = warp & 3;                  // TMEM lane quadrant
    const int row = q4 * 32 + lane;           // row of the tile: token row / group, head row % group
    const int tok = row / p.group, head = hk * p.group + row % p.group;
    const bool valid = tok < p.tokens && t0 + tok < L;
    const int pos = valid ? first_pos + tok : -1;                           // a row of nothing sees no key
    const uint32_t lane_off = static_cast<uint32_t>(q4 * 32) << 16;
    const float sl2 = BIAS ? 1.f : p.scale * kLog2e;                        // with a bias scores are in these units before the maximum
    const int lo = first_key(pos);                                          // first key of the row's window or chunk
    const int tile_lo = first_key(last_pos);                                // … of the tile's last token
    float r1 = 0.f, r2 = 0.f;
    if (BIAS && valid) {
      r1 = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.x.r1)[head]);
      r2 = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.x.r2)[head]);
    }
    const int keep = p.window > 0 ? p.keep : 0;
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_blocks && !*abort_flag; ++j) {
      const int st = j & 1;
      if (!mbar_wait(&s_full[st], (j >> 1) & 1)) { ok = false; break; }
      tc_fence_after();
      const int kv0 = key_of(j);
      const bool need_mask = !valid || kv0 + BKV > first_pos + 1 || (kv0 < tile_lo && kv0 + BKV > keep);
      uint32_t s[2][32];
      tmem_ld_32x32(tmem + lane_off + st * BKV, s[0]);
      tmem_ld_32x32(tmem + lane_off + st * BKV + 32, s[1]);
      tmem_ld_wait();
      float mx4[4] = {m_run, -INFINITY, -INFINITY, -INFINITY};   // independent chains
#pragma unroll
      for (int c = 0; c < 2; ++c) {
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          float v = __uint_as_float(s[c][i]);
          const int col = kv0 + c * 32 + i;
          if (BIAS) {
            v = fmaf(v, p.scale * kLog2e, -r1 * __log2f(fmaf(r2, static_cast<float>(pos - col), 1.f)));
            s[c][i] = __float_as_uint(v);
          }
          if (need_mask) {
            if (col > pos || (col < lo && col >= keep)) v = -INFINITY;
            s[c][i] = __float_as_uint(v);
          }
          mx4[i & 3] = fmaxf(mx4[i & 3], v);
        }
      }
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      // lazy rescaling (see attention_tc.cu): the reference maximum may trail the true one by up to 2^8
      if (m_run != -INFINITY && (mx - m_run) * sl2 <= 8.0f) mx = m_run;
      const float msc = (mx == -INFINITY) ? 0.f : mx * sl2;
      const float alpha = (m_run == -INFINITY) ? 0.f : exp2f(m_run * sl2 - msc);
      // O must be stable (previous P·V finished) before it is rescaled
      if (j > 0) {
        if (!mbar_wait(pv_done, (j - 1) & 1)) { ok = false; break; }
        tc_fence_after();
        if (!__all_sync(0xffffffffu, mx == m_run)) {
#pragma unroll 1
          for (int c = 0; c < NV * 2; ++c) {
            uint32_t o[32];
            tmem_ld_32x32(tmem_o + lane_off + c * 32, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st_32x32(tmem_o + lane_off + c * 32, o);
          }
        }
      }
      float rs4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < 2; ++c) {
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float a = exp2f(fmaf(__uint_as_float(s[c][i]), sl2, -msc)), d = exp2f(fmaf(__uint_as_float(s[c][i + 1]), sl2, -msc));
          rs4[i & 2] += a;
          rs4[(i & 2) + 1] += d;
          const uint32_t hi = pack_bf16x2(a, d);
          s[c][i] = hi;
          s[c][i + 1] = pack_bf16x2(a - __uint_as_float(hi << 16), d - __uint_as_float(hi & 0xffff0000u));
        }
      }
      uint32_t w[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) w[i] = s[i >> 4][(i & 15) * 2];
      tmem_st_32x32(tmem + lane_off + st * BKV, w);
#pragma unroll
      for (int i = 0; i < 32; ++i) w[i] = s[i >> 4][(i & 15) * 2 + 1];
      tmem_st_32x32(tmem + lane_off + st * BKV + 32, w);
      tmem_st_wait();
      l_run = l_run * alpha + (rs4[0] + rs4[1]) + (rs4[2] + rs4[3]);
      m_run = mx;
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    if (ok && !*abort_flag) {
      if (!mbar_wait(pv_done, (n_blocks - 1) & 1)) ok = false;
    }
    if (!ok) {
      *abort_flag = 1;
      atomicExch(p.error_flag, 83);
    }
    if (__all_sync(0xffffffffu, ok && !*abort_flag)) {      // the whole warp or none of it: the loads and exchanges below are collective
      tc_fence_after();
      // O / (l + exp(sink)), both relative to the larger of the running maximum and the sink
      float inv = 0.f;
      if (valid) {
        if (p.sink != nullptr) {
          const float sk = __bfloat162float(p.sink[head]) * kLog2e, ms = m_run * sl2, mm = fmaxf(ms, sk);
          const float a = exp2f(ms - mm);
          inv = __fdiv_rn(a, fmaf(l_run, a, exp2f(sk - mm)));
        } else {
          inv = __fdiv_rn(1.f, l_run);
        }
      }
      if (p.diff.lam != nullptr) {
        // both rows of a head hold o = a1 − lam·a2 after the exchange; the even one stores the first half of every 32 columns, the odd
        // one the second
        const float lam = *p.diff.lam;
        const bool odd = row & 1;
        auto difference = [&](uint32_t (&o)[32]) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float a = __uint_as_float(o[i]) * inv, other = __shfl_xor_sync(0xffffffffu, a, 1);
            o[i] = __float_as_uint(odd ? fmaf(-lam, a, other) : fmaf(-lam, other, a));
          }
        };
        float ss = 0.f;
#pragma unroll 1
        for (int c = 0; c < NV * 2; ++c) {
          uint32_t o[32];
          tmem_ld_32x32(tmem_o + lane_off + c * 32, o);
          tmem_ld_wait();
          difference(o);
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i < p.vdim) ss = fmaf(__uint_as_float(o[i]), __uint_as_float(o[i]), ss);
        }
        float f = 0.f;
        if (valid) {
          const float g = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.diff.gate)[static_cast<long long>(q_start + t0 + tok) * p.diff.gate_ld + head / 2]);
          f = __fdiv_rn(p.diff.gain, __fsqrt_rn(__fdiv_rn(ss, static_cast<float>(p.vdim)) + p.diff.eps)) * __fdividef(1.f, 1.f + __expf(-g));
        }
        __nv_bfloat16* orow = p.o + static_cast<long long>(q_start + t0 + tok) * p.o_row + static_cast<long long>(head / 2) * p.vdim;
#pragma unroll 1
        for (int c = 0; c < NV * 2; ++c) {
          uint32_t o[32];
          tmem_ld_32x32(tmem_o + lane_off + c * 32, o);
          tmem_ld_wait();
          difference(o);
          if (valid) {
#pragma unroll
            for (int i = 0; i < 16; i += 8) {
              const int col = c * 32 + (odd ? 16 : 0) + i;
              uint32_t w[4];
#pragma unroll
              for (int k = 0; k < 4; ++k)
                w[k] = odd ? pack_bf16x2(__uint_as_float(o[16 + i + 2 * k]) * f, __uint_as_float(o[16 + i + 2 * k + 1]) * f)
                           : pack_bf16x2(__uint_as_float(o[i + 2 * k]) * f, __uint_as_float(o[i + 2 * k + 1]) * f);
              if (col < p.vdim) *reinterpret_cast<uint4*>(orow + col) = make_uint4(w[0], w[1], w[2], w[3]);
            }
          }
        }
      } else {
        __nv_bfloat16* orow = p.o + static_cast<long long>(q_start + t0 + tok) * p.o_row + static_cast<long long>(head) * p.vdim;
#pragma unroll 1
        for (int c = 0; c < NV * 2; ++c) {
          uint32_t o[32];
          tmem_ld_32x32(tmem_o + lane_off + c * 32, o);
          tmem_ld_wait();
          if (valid) {
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
              if (c * 32 + i < p.vdim) {         // vdim is a multiple of 8
                if (p.x.gate != nullptr) {
                  const __nv_bfloat16* gr = reinterpret_cast<const __nv_bfloat16*>(p.x.gate) + (q_start + t0 + tok) * p.x.gate_ld +
                                            static_cast<long long>(head) * p.vdim + c * 32 + i;
                  const uint4 gv = *reinterpret_cast<const uint4*>(gr);
                  const uint32_t gw[4] = {gv.x, gv.y, gv.z, gv.w};
#pragma unroll
                  for (int k = 0; k < 8; ++k) {
                    const float z = __uint_as_float((k & 1) ? gw[k / 2] & 0xffff0000u : gw[k / 2] << 16);
                    o[i + k] = __float_as_uint(__uint_as_float(o[i + k]) * __fdividef(1.f, 1.f + __expf(-z)));
                  }
                }
                uint4 v;
                v.x = pack_bf16x2(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv);
                v.y = pack_bf16x2(__uint_as_float(o[i + 2]) * inv, __uint_as_float(o[i + 3]) * inv);
                v.z = pack_bf16x2(__uint_as_float(o[i + 4]) * inv, __uint_as_float(o[i + 5]) * inv);
                v.w = pack_bf16x2(__uint_as_float(o[i + 6]) * inv, __uint_as_float(o[i + 7]) * inv);
                *reinterpret_cast<uint4*>(orow + c * 32 + i) = v;
              }
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, kTmemCols);
  }
}

template <int NA, int NV, bool BIAS>
static int launch_as(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const Params& p, int max_q, int kv_heads, int n_seq,
                  cudaStream_t s) {
  using G = Cfg<NA, NV>;
  static bool once = false;
  if (!once) {
    cudaError_t e = cudaFuncSetAttribute(window_prefill_kernel<NA, NV, BIAS>, cudaFuncAttributeMaxDynamicSharedMemorySize, G::total);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(window_prefill_kernel<NA, NV, BIAS>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    if (e != cudaSuccess) return static_cast<int>(e);
    once = true;
  }
  window_prefill_kernel<NA, NV, BIAS><<<dim3((max_q + p.tokens - 1) / p.tokens, kv_heads, n_seq), 192, G::total, s>>>(tq, tk, tv, p);
  return static_cast<int>(cudaGetLastError());
}

template <int NA, int NV>
static int launch(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const Params& p, int max_q, int kv_heads, int n_seq,
                  cudaStream_t s) {
  return p.x.r1 != nullptr ? launch_as<NA, NV, true>(tq, tk, tv, p, max_q, kv_heads, n_seq, s) : launch_as<NA, NV, false>(tq, tk, tv, p, max_q, kv_heads, n_seq, s);
}

}  // namespace fw
}  // namespace mb

using namespace mb;

// q [≥ t_long, heads, q_pitch] with zeros behind dim (q_pitch a multiple of 64); kc [pages, block_size, kv_heads, dim], vc [.., vdim]; o rows of
// o_row elements (a multiple of 8).  dim, vdim multiples of 8 up to 128, block_size a multiple of 8, up to 128 query heads per key head, scale > 0.
extern "C" int mb_window_prefill(const void* q, const void* kc, const void* vc, void* o, long long o_row, const void* sink, const int* cu_q,
                                 const int* positions, const int* block_table, int max_blocks, int block_size, int num_blocks, int n_seq, int max_q,
                                 int t_long, float scale, MbWindow L, MbDiff d, MbScores x, int* error_flag, cudaStream_t s) {
  if (n_seq <= 0 || t_long <= 0) return 0;
  const int group = L.heads / L.kv_heads, na = (L.dim + 63) / 64, nv = (L.vdim + 63) / 64;
  if (L.dim % 8 || L.vdim % 8 || L.dim > 128 || L.vdim > 128 || L.q_pitch != na * 64 || L.heads % L.kv_heads || group > 128 || block_size % 8 ||
      o_row % 8 || !(scale > 0.f) || (d.lam != nullptr && (sink != nullptr || group % 2 || x.gate != nullptr)) || (L.chunk > 0 && L.window > 0) ||
      (x.r1 != nullptr && sink != nullptr) ||
      (x.gate != nullptr && (x.gate_ld % 8 || reinterpret_cast<uintptr_t>(x.gate) % 16)))
    return -3;
  int box = 64;
  while (block_size % box) box /= 2;
  CUtensorMap tq, tk, tv;
  const int tokens = 128 / group;
  int rc = make_tmap_bf16_3d(&tq, q, t_long, L.heads, L.q_pitch, tokens, group, 64);
  if (rc) return 1000 + rc;
  const long long rows = static_cast<long long>(num_blocks) * block_size, kw = static_cast<long long>(L.kv_heads) * L.dim, vw = static_cast<long long>(L.kv_heads) * L.vdim;
  rc = make_tmap_bf16_2d(&tk, kc, rows, kw, kw, box, 64);
  if (rc) return 2000 + rc;
  rc = make_tmap_bf16_2d(&tv, vc, rows, vw, vw, box, 64);
  if (rc) return 3000 + rc;
  fw::Params p{reinterpret_cast<__nv_bfloat16*>(o), o_row, reinterpret_cast<const __nv_bfloat16*>(sink), cu_q, positions, block_table, max_blocks,
               block_size, box, group, tokens, L.dim, L.vdim, scale, L.window, L.keep, L.chunk, x, d, error_flag};
  if (na == 1) return nv == 1 ? fw::launch<1, 1>(tq, tk, tv, p, max_q, L.kv_heads, n_seq, s) : fw::launch<1, 2>(tq, tk, tv, p, max_q, L.kv_heads, n_seq, s);
  return nv == 1 ? fw::launch<2, 1>(tq, tk, tv, p, max_q, L.kv_heads, n_seq, s) : fw::launch<2, 2>(tq, tk, tv, p, max_q, L.kv_heads, n_seq, s);
}
