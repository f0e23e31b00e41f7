// Prefill attention on tcgen05 tensor cores for keys and values expanded from cached latents: causal with an optional sliding
// window and a softmax sink per head, separate unrotated (per head) and rotated (shared by the heads) key parts.
//
// Structure of flash_fwd_tc_kernel (attention_tc.cu): one CTA = 128 query rows of one (sequence, head), two CTAs per SM, one TMA
// warp, one MMA warp, four softmax warps with one thread per query row.  What differs:
//   * S = Q_n·K_nᵀ + Q_r·K_rᵀ: NA 64-column atoms of the expanded keys [tokens, H·dim (+ H·vdim)] and one of the gathered latents'
//     rotated part, which is never copied per head.  Query padding columns are zero, so whatever a box reads past a head's own
//     columns contributes nothing;
//   * the softmax weights keep 16 bits of mantissa through the second product: P = P_hi + P_lo, both bf16, written over the
//     score buffer in tensor memory (64 fp32 columns = 32 + 32 columns of bf16 pairs) and used from there as the A operand;
//   * key blocks entirely before the tile's window are skipped; the sink enters the denominator at the end.
// Keys of a sequence are the gathered positions [base, end); its queries are the last Lq of them.
#include "launch.h"
#include "ptx.cuh"

namespace mb {

int make_tmap_bf16_2d(CUtensorMap* out, const void* base, long long rows, long long cols, long long ld, int box_rows, int box_cols);

namespace fl {

static constexpr int BQ = 128, BKV = 64;
static constexpr int kQAtom = BQ * 128, kKVAtom = BKV * 128;      // bytes of a 64-column atom
static constexpr uint32_t kTmemCols = 256;                        // S0 | S1 (64 each) | O (128)
static constexpr float kLog2e = 1.4426950408889634f;

struct Params {
  __nv_bfloat16* o;            // [tokens, H, vdim]
  const __nv_bfloat16* sink;   // [H] or null
  const __nv_bfloat16* gate;   // rows of gate_ld, [H·vdim], or null: outputs times its sigmoid
  long long gate_ld;
  const int* cu_q;
  const int* cu_k;
  int H, dim, vdim, rank_p;
  float scale;
  int window;                  // 0: all earlier keys
  int* error_flag;
};

template <int NA, int NV>
struct Cfg {
  static constexpr int kVStages = NA == 2 ? 1 : 2;
  static constexpr int kQBytes = (NA + 1) * kQAtom, kKBytes = (NA + 1) * kKVAtom, kVBytes = NV * kKVAtom;
  static constexpr int q = 0, k = kQBytes, v = k + 2 * kKBytes, bars = v + kVStages * kVBytes, total = bars + 256;
};

template <int NA, int NV>
__global__ void __launch_bounds__(192, 2)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv,
                      const __grid_constant__ CUtensorMap tm_lat, Params p) {
  using G = Cfg<NA, NV>;
  extern __shared__ __align__(1024) uint8_t smem[];
  if (smem_u32(smem) & 1023u) {   // swizzled tiles need 1024-byte alignment
    if (threadIdx.x == 0) atomicExch(p.error_flag, 35);
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
  const int b = blockIdx.z, h = blockIdx.y;
  const int q_start = p.cu_q[b], L = p.cu_q[b + 1] - q_start;
  const int k_start = p.cu_k[b], Lk = p.cu_k[b + 1] - k_start;
  const int off = Lk - L;                             // query i sits at key position i + off
  const int q0 = (gridDim.x - 1 - blockIdx.x) * BQ;   // late query blocks (long key ranges) first
  if (q0 >= L || off < 0) return;
  const int kv_end = min(Lk, q0 + BQ + off);
  const int kv_begin = p.window > 0 ? max(0, q0 + off - p.window + 1) / BKV * BKV : 0;
  const int n_blocks = (kv_end - kv_begin + BKV - 1) / BKV;

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
      auto load_k = [&](int j) -> bool {
        const int st = j & 1, row = k_start + kv_begin + j * BKV;
        if (!mbar_wait(&k_empty[st], ((j >> 1) & 1) ^ 1)) return false;
        mbar_expect_tx(&k_full[st], G::kKBytes);
        uint8_t* sk = smem + G::k + st * G::kKBytes;
        for (int a = 0; a < NA; ++a) tma_load_2d(sk + a * kKVAtom, &tm_kv, &k_full[st], h * p.dim + a * 64, row);
        tma_load_2d(sk + NA * kKVAtom, &tm_lat, &k_full[st], p.rank_p, row);
        return true;
      };
      mbar_expect_tx(q_full, G::kQBytes);
      for (int a = 0; a <= NA; ++a) tma_load_2d(smem + G::q + a * kQAtom, &tm_q, q_full, (h * (NA + 1) + a) * 64, q_start + q0);
      bool ok = load_k(0);
      for (int j = 0; j < n_blocks && ok && !*abort_flag; ++j) {
        if (j + 1 < n_blocks) ok = load_k(j + 1);
        const int st = j % G::kVStages;
        if (!ok || !mbar_wait(&v_empty[st], ((j / G::kVStages) & 1) ^ 1)) { ok = false; break; }
        mbar_expect_tx(&v_full[st], G::kVBytes);
        uint8_t* sv = smem + G::v + st * G::kVBytes;
        for (int a = 0; a < NV; ++a)
          tma_load_2d(sv + a * kKVAtom, &tm_kv, &v_full[st], p.H * p.dim + h * p.vdim + a * 64, k_start + kv_begin + j * BKV);
      }
      if (!ok) { *abort_flag = 1; atomicExch(p.error_flag, 31); }
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
        for (int ks = 0; ks < (NA + 1) * 4; ++ks)
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
        const int st = j % G::kVStages;
        if (!mbar_wait(&v_full[st], (j / G::kVStages) & 1) || !mbar_wait(p_ready, j & 1)) { ok = false; break; }
        tc_fence_after();
        const uint32_t v_addr = smem_u32(smem + G::v + st * G::kVBytes);
#pragma unroll
        for (int part = 0; part < 2; ++part)        // P_hi, then P_lo
#pragma unroll
          for (int ks = 0; ks < BKV / 16; ++ks)
            umma_bf16_ts(tmem_o, tmem + (j & 1) * BKV + part * 32 + ks * 8, make_smem_desc_sw128(v_addr + ks * (16 * 128), kKVAtom, 1024),
                         idesc_o, (j | part | ks) != 0);
        umma_commit(&v_empty[st]);
        umma_commit(pv_done);
      }
      if (!ok) { *abort_flag = 1; atomicExch(p.error_flag, 32); }
    }
  } else {
    const int q4 = warp & 3;                  // TMEM lane quadrant
    const int row = q4 * 32 + lane;           // query row within the tile
    const int qk = q0 + row + off;            // the row's own key position
    const uint32_t lane_off = static_cast<uint32_t>(q4 * 32) << 16;
    const float sl2 = p.scale * kLog2e;
    const int first = p.window > 0 ? qk - p.window + 1 : 0;       // first key position the row sees
    const int tile_first = p.window > 0 ? q0 + BQ - 1 + off - p.window + 1 : 0;   // … and the tile's last row
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_blocks && !*abort_flag; ++j) {
      const int st = j & 1;
      if (!mbar_wait(&s_full[st], (j >> 1) & 1)) { ok = false; break; }
      tc_fence_after();
      const int kv0 = kv_begin + j * BKV;
      const bool need_mask = kv0 + BKV > q0 + off + 1 || kv0 < tile_first;
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
          if (need_mask) {
            const int col = kv0 + c * 32 + i;
            if (col > qk || col < first) v = -INFINITY;       // qk < Lk: keys past the end are masked by the diagonal
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
      atomicExch(p.error_flag, 33);
    } else if (!*abort_flag) {
      tc_fence_after();
      // O / (l + exp(sink)), both relative to the larger of the running maximum and the sink
      float inv;
      if (p.sink != nullptr) {
        const float sk = __bfloat162float(p.sink[h]) * kLog2e, ms = m_run * sl2, mm = fmaxf(ms, sk);
        const float a = exp2f(ms - mm);
        inv = a / fmaf(l_run, a, exp2f(sk - mm));
      } else {
        inv = l_run > 0.f ? 1.f / l_run : 0.f;
      }
      const bool valid = q0 + row < L;
      __nv_bfloat16* orow = p.o + (static_cast<long long>(q_start + q0 + row) * p.H + h) * p.vdim;
#pragma unroll 1
      for (int c = 0; c < NV * 2; ++c) {
        uint32_t o[32];
        tmem_ld_32x32(tmem_o + lane_off + c * 32, o);
        tmem_ld_wait();
        if (valid) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c * 32 + i < p.vdim) {         // vdim is a multiple of 8
              if (p.gate != nullptr) {
                const uint4 gv = *reinterpret_cast<const uint4*>(p.gate + static_cast<long long>(q_start + q0 + row) * p.gate_ld + h * p.vdim + c * 32 + i);
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
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, kTmemCols);
  }
}

template <int NA, int NV>
static int launch(const CUtensorMap& tq, const CUtensorMap& tkv, const CUtensorMap& tl, const Params& p, int max_q, int n_seq, cudaStream_t s) {
  using G = Cfg<NA, NV>;
  static bool once = false;
  if (!once) {
    cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<NA, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, G::total);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(latent_prefill_kernel<NA, NV>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    if (e != cudaSuccess) return static_cast<int>(e);
    once = true;
  }
  latent_prefill_kernel<NA, NV><<<dim3((max_q + BQ - 1) / BQ, p.H, n_seq), 192, G::total, s>>>(tq, tkv, tl, p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace fl
}  // namespace mb

using namespace mb;

// q [t_long, H, (NA + 1)·64] zero-padded queries; kv [Tk, H·dim + H·vdim] expanded keys and values; lat [Tk, pitch] gathered cache rows;
// o [t_long, H, vdim].  dim, vdim multiples of 8, dim ≤ 128, rot ≤ 64, vdim ≤ 128, scale > 0.
extern "C" int mb_latent_prefill(const void* q, const void* kv, const void* lat, void* o, const void* sink, const void* gate, long long gate_ld,
                                 const int* cu_q, const int* cu_k, int n_seq, int max_q, int t_long, int tk, float scale, int window, MbLatent L, int* error_flag,
                                 cudaStream_t s) {
  if (n_seq <= 0 || t_long <= 0) return 0;
  if (L.dim % 8 || L.vdim % 8 || L.dim > 128 || L.rot > 64 || L.vdim > 128 || !(scale > 0.f)) return -3;
  if (gate != nullptr && (gate_ld % 8 || reinterpret_cast<uintptr_t>(gate) % 16)) return -3;
  const int na = (L.dim + 63) / 64, nv = (L.vdim + 63) / 64;
  CUtensorMap tq, tkv, tl;
  const long long qw = static_cast<long long>(L.heads) * (na + 1) * 64, kvw = static_cast<long long>(L.heads) * (L.dim + L.vdim);
  int rc = make_tmap_bf16_2d(&tq, q, t_long, qw, qw, fl::BQ, 64);
  if (rc) return 1000 + rc;
  rc = make_tmap_bf16_2d(&tkv, kv, tk, kvw, kvw, fl::BKV, 64);
  if (rc) return 2000 + rc;
  rc = make_tmap_bf16_2d(&tl, lat, tk, L.pitch, L.pitch, fl::BKV, 64);
  if (rc) return 3000 + rc;
  fl::Params p{reinterpret_cast<__nv_bfloat16*>(o), reinterpret_cast<const __nv_bfloat16*>(sink), reinterpret_cast<const __nv_bfloat16*>(gate), gate_ld, cu_q, cu_k, L.heads, L.dim, L.vdim, L.rank_p,
               scale, window, error_flag};
  if (na == 1) return nv == 1 ? fl::launch<1, 1>(tq, tkv, tl, p, max_q, n_seq, s) : fl::launch<1, 2>(tq, tkv, tl, p, max_q, n_seq, s);
  return nv == 1 ? fl::launch<2, 1>(tq, tkv, tl, p, max_q, n_seq, s) : fl::launch<2, 2>(tq, tkv, tl, p, max_q, n_seq, s);
}
