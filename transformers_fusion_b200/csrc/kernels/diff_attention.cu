// Differential attention (two score maps per head over one set of values), causal, with an optional sliding window:
//
//   a_t = softmax(scale Q_t K_t^T) V  (t = 1, 2);   o = a_1 - lambda a_2;   o <- o / rms(o) * out_scale
//
// Query row i of a sequence sees keys j with i - window < j <= i.  Three forms:
//   diff_attn_fwd      prompts, bf16, tcgen05: one CTA per (sequence, head, 128 queries).  The two maps are the two score tiles
//                      of the CTA (each with its own K tile, sharing every V tile), so that one softmax group works while the
//                      tensor core computes the other map; the difference, its norm and the scale happen in the epilogue, where
//                      a query's row of a map sits in the registers of one thread and the other map's row comes through TMEM.
//   diff_decode        one query per sequence over the paged cache, bf16, mma.sync: the query heads of a kv head are the rows of a
//                      16-row tile, map 1 in rows 0-7 (zero in the entries of map 2) and map 2 in rows 8-15, so that the keys
//                      of both maps are one row of 2 D entries and one P V product serves both.  Split over the keys; a
//                      second kernel merges the splits and applies difference, norm and scale.
//   diff_attn_any      any sizes, bf16 or fp32, prompts or decoding: fp32 FMA throughout, online softmax over 32-key tiles.
#include "tfb_elem.cuh"
#include "tfb_host.h"

namespace tfb {
TFB_BOUNDS_DEFINE(diff_attention)

constexpr float LOG2E = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------------
// prompts on tcgen05
// ------------------------------------------------------------------------------------------------
struct DiffFwdParams {
  int B, S, H, G;
  int Skv, q_off;         // keys per sequence; query i sits at key index i + q_off
  int window;             // 0: no limit
  int V;                  // value entries per head
  float scale, lambda, out_scale, eps;
  __nv_bfloat16* O;
  long long ldo;
  int* status;
};

constexpr int DA_THREADS = 320;
constexpr int DA_BM = 128;

template <int DK, int DV, int BN>
struct DiffSmem {
  static constexpr int NBK = DK / 64, NBV = DV / 64;
  static constexpr int QBOX = DA_BM * 128, KBOX = BN * 128;         // bytes of a 64-column box
  static constexpr int QT = NBK * QBOX, KT = NBK * KBOX, VT = NBV * KBOX;
  static constexpr int STAGE = 2 * KT + VT;
  static constexpr int AVAIL = 227 * 1024 - 1024 - 256 - 2 * QT;
  static constexpr int STAGES = AVAIL / STAGE > 4 ? 4 : AVAIL / STAGE;
  static constexpr int KV_OFF = 2 * QT;
  static constexpr int BAR_OFF = KV_OFF + STAGES * STAGE;
  static constexpr int TOTAL = BAR_OFF + 256 + 1024;
  static_assert(STAGES >= 2, "two stages at least");
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// running maximum over the BN scores of this thread's row; keys outside [lo, hi] (indices within the tile) do not count
template <bool MASK, int BN>
__device__ __forceinline__ float tile_max(uint32_t tS, float m, int lo, int hi) {
  float mx0 = m, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll 1
  for (int c = 0; c < BN / 32; ++c) {
    uint32_t v[32];
    tmem_ld_32x32(tS + c * 32, v);
    tmem_ld_wait();
    if (MASK) {
#pragma unroll
      for (int i = 0; i < 32; ++i)
        if (c * 32 + i > hi || c * 32 + i < lo) v[i] = 0xff800000u;
    }
#pragma unroll
    for (int i = 0; i < 32; i += 8) {
      mx0 = fmax3(mx0, __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
      mx1 = fmax3(mx1, __uint_as_float(v[i + 2]), __uint_as_float(v[i + 3]));
      mx2 = fmax3(mx2, __uint_as_float(v[i + 4]), __uint_as_float(v[i + 5]));
      mx3 = fmax3(mx3, __uint_as_float(v[i + 6]), __uint_as_float(v[i + 7]));
    }
  }
  return fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3));
}

// p = 2^(s * sl2 - mb) over the row, written back over the scores as bf16 pairs; returns the row sum
template <bool MASK, int BN>
__device__ __forceinline__ float tile_probs(uint32_t tS, float sl2, float mb, int lo, int hi) {
  float rs0 = 0.f, rs1 = 0.f, rs2 = 0.f, rs3 = 0.f;
#pragma unroll 1
  for (int c = 0; c < BN / 32; ++c) {
    uint32_t v[32], pk[16];
    tmem_ld_32x32(tS + c * 32, v);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < 16; i += 2) {
      float q[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = c * 32 + 2 * i + e;
        q[e] = ex2(fmaf(__uint_as_float(v[2 * i + e]), sl2, -mb));
        if (MASK && (j > hi || j < lo)) q[e] = 0.f;
      }
      rs0 += q[0];
      rs1 += q[1];
      rs2 += q[2];
      rs3 += q[3];
      pk[i] = pack_bf16(q[0], q[1]);
      pk[i + 1] = pack_bf16(q[2], q[3]);
    }
    tmem_st_32x16(tS + c * 16, pk);
  }
  return (rs0 + rs1) + (rs2 + rs3);
}

template <int DK, int DV, int BN>
__global__ void __launch_bounds__(DA_THREADS, 1)
diff_attn_fwd_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk, const __grid_constant__ CUtensorMap tv,
                     const DiffFwdParams p) {
  using L = DiffSmem<DK, DV, BN>;
  constexpr int ST = L::STAGES;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sQ = smem_u32(smem);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::BAR_OFF);
  const uint32_t bar_q = smem_u32(bars);
  const uint32_t bar_kv_full = bar_q + 8;
  const uint32_t bar_kv_empty = bar_kv_full + ST * 8;
  const uint32_t bar_s_full = bar_kv_empty + ST * 8;
  const uint32_t bar_p_ready = bar_s_full + 16;
  const uint32_t bar_o_full = bar_p_ready + 16;
  const uint32_t bar_o2 = bar_o_full + 16;            // map 2's normalised rows are back in TMEM
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 1 + 2 * ST + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nqb = (p.S + DA_BM - 1) / DA_BM;
  const int bh = p.B * p.H;
  const int qb = nqb - 1 - int(blockIdx.x) / bh;       // the longest (latest) query blocks first
  const int rem = int(blockIdx.x) % bh;
  const int b = rem / p.H, h = rem % p.H, hk = h / (p.H / p.G);
  const int q_first = qb * DA_BM + p.q_off, q_last = min(qb * DA_BM + DA_BM - 1, p.S - 1) + p.q_off;   // key indices
  const int j0 = p.window > 0 ? max(0, q_first - p.window + 1) / BN : 0;
  const int n_kv = min(q_last, p.Skv - 1) / BN + 1 - j0;

  if (threadIdx.x == 0) {
    mbar_init(bar_q, 1);
    for (int s = 0; s < ST; ++s) {
      mbar_init(bar_kv_full + s * 8, 1);
      mbar_init(bar_kv_empty + s * 8, 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(bar_s_full + i * 8, 1);
      mbar_init(bar_p_ready + i * 8, 128);
      mbar_init(bar_o_full + i * 8, 1);
    }
    mbar_init(bar_o2, 128);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tq);
    tma_prefetch_desc(&tk);
    tma_prefetch_desc(&tv);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  tfb::pdl_sync();
  const uint32_t tS0 = tmem_base, tO0 = tmem_base + 256;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(bar_q, 2 * L::QT);
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int i = 0; i < L::NBK; ++i) tma_load_4d(sQ + t * L::QT + i * L::QBOX, &tq, bar_q, i * 64, 2 * h + t, qb * DA_BM, b);
      for (int j = 0; j < n_kv; ++j) {
        const int st = j % ST;
        if (!mbar_wait(bar_kv_empty + st * 8, ((j / ST) & 1) ^ 1, abort_flag, p.status, ST_TIMEOUT_EMPTY)) break;
        const uint32_t fb = bar_kv_full + st * 8, base = sQ + L::KV_OFF + st * L::STAGE;
        mbar_expect_tx(fb, L::STAGE);
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int i = 0; i < L::NBK; ++i) tma_load_4d(base + t * L::KT + i * L::KBOX, &tk, fb, i * 64, 2 * hk + t, (j0 + j) * BN, b);
#pragma unroll
        for (int i = 0; i < L::NBV; ++i) tma_load_4d(base + 2 * L::KT + i * L::KBOX, &tv, fb, i * 64, hk, (j0 + j) * BN, b);
      }
      if (*abort_flag) {  // unwinding: bounded wait for copies already issued
        const uint64_t t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 200000ull) {}
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc(FMT_BF16, FMT_BF16, false, false, DA_BM, BN);
      constexpr uint32_t idesc_o = umma_idesc(FMT_BF16, FMT_BF16, false, true, DA_BM, DV);
      auto issue_s = [&](int t, int j) {
        const uint32_t sK = sQ + L::KV_OFF + (j % ST) * L::STAGE + t * L::KT, sQt = sQ + t * L::QT, tS = tS0 + t * 128;
#pragma unroll
        for (int k = 0; k < DK / 16; ++k)
          umma_f16_ss(tS, umma_smem_desc(sQt + (k >> 2) * L::QBOX + (k & 3) * 32, 16, 1024),
                      umma_smem_desc(sK + (k >> 2) * L::KBOX + (k & 3) * 32, 16, 1024), idesc_s, k > 0);
        umma_commit(bar_s_full + t * 8);
      };
      bool ok = mbar_wait(bar_q, 0, abort_flag, p.status, ST_TIMEOUT_FULL) &&
                mbar_wait(bar_kv_full, 0, abort_flag, p.status, ST_TIMEOUT_FULL);
      if (ok) {
        tc_fence_after();
        issue_s(0, 0);
        issue_s(1, 0);
      }
      for (int j = 0; j < n_kv && ok; ++j) {
        if (j + 1 < n_kv) {
          const int st1 = (j + 1) % ST;
          if (!mbar_wait(bar_kv_full + st1 * 8, ((j + 1) / ST) & 1, abort_flag, p.status, ST_TIMEOUT_FULL)) break;
          tc_fence_after();
        }
        const int st = j % ST;
        const uint32_t sV = sQ + L::KV_OFF + st * L::STAGE + 2 * L::KT;
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          if (!ok) continue;
          if (!mbar_wait(bar_p_ready + t * 8, j & 1, abort_flag, p.status, ST_TIMEOUT_TMEM_EMPTY)) {
            ok = false;
            continue;
          }
          tc_fence_after();
          const uint32_t tP = tS0 + t * 128, tO = tO0 + t * 128;
#pragma unroll
          for (int k = 0; k < BN / 16; ++k) umma_f16_ts(tO, tP + k * 8, umma_smem_desc(sV + k * 2048, L::KBOX, 1024), idesc_o, k > 0);
          if (j + 1 < n_kv) issue_s(t, j + 1);         // its commit also covers the P V product above
          else umma_commit(bar_o_full + t * 8);
        }
        if (ok) umma_commit(bar_kv_empty + st * 8);
      }
    }
  } else {
    const int t = (warp - 2) >> 2, quad = warp & 3, r = quad * 32 + lane;
    const int q_idx = qb * DA_BM + r;
    const uint32_t lane_off = uint32_t(quad * 32) << 16;
    const uint32_t tS = tS0 + t * 128 + lane_off, tO = tO0 + t * 128 + lane_off;
    const float sl2 = p.scale * LOG2E;
    const int hi_g = min(q_idx + p.q_off, p.Skv - 1);
    const int lo_g = p.window > 0 ? q_idx + p.q_off - p.window + 1 : 0;
    float m = -INFINITY, l = 0.f, alpha_prev = 1.f;
    float o[DV];
#pragma unroll
    for (int i = 0; i < DV; ++i) o[i] = 0.f;
    bool ok = true;
    for (int j = 0; j < n_kv; ++j) {
      if (!mbar_wait_warp(bar_s_full + t * 8, j & 1, abort_flag, p.status, ST_TIMEOUT_TMEM_FULL)) {
        ok = false;
        break;
      }
      tc_fence_after();
      const int k0 = (j0 + j) * BN;
      const bool need_mask = k0 + BN - 1 > q_first || k0 + BN > p.Skv || (p.window > 0 && k0 < q_last - p.window + 1);
      const int lo = lo_g - k0, hi = hi_g - k0;
      const float mx = need_mask ? tile_max<true, BN>(tS, m, lo, hi) : tile_max<false, BN>(tS, m, lo, hi);
      if (j > 0) {  // O(j-1) is complete: the commit behind S(j) was issued after it
#pragma unroll
        for (int c = 0; c < DV / 32; ++c) {
          uint32_t v[32];
          tmem_ld_32x32(tO + c * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[c * 32 + i] = fmaf(o[c * 32 + i], alpha_prev, __uint_as_float(v[i]));
        }
      }
      const float mb = (mx == -INFINITY) ? 0.f : mx * sl2;
      const float alpha = (m == -INFINITY) ? 0.f : ex2(m * sl2 - mb);
      const float rs = need_mask ? tile_probs<true, BN>(tS, sl2, mb, lo, hi) : tile_probs<false, BN>(tS, sl2, mb, lo, hi);
      l = fmaf(l, alpha, rs);
      m = mx;
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(bar_p_ready + t * 8);
      alpha_prev = alpha;
    }
    if (ok && mbar_wait_warp(bar_o_full + t * 8, 0, abort_flag, p.status, ST_TIMEOUT_TMEM_FULL)) {
      tc_fence_after();
      const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(tO + c * 32, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c * 32 + i] = fmaf(o[c * 32 + i], alpha_prev, __uint_as_float(v[i])) * inv;
      }
      if (t == 1) {      // hand the row over through this row's own TMEM columns
#pragma unroll
        for (int c = 0; c < DV / 16; ++c) {
          uint32_t v[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(o[c * 16 + i]);
          tmem_st_32x16(tO + c * 16, v);
        }
        tmem_st_wait();
        tc_fence_before();
        mbar_arrive(bar_o2);
      } else if (mbar_wait_warp(bar_o2, 0, abort_flag, p.status, ST_TIMEOUT_TMEM_FULL)) {
        tc_fence_after();
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < DV / 32; ++c) {
          uint32_t v[32];
          tmem_ld_32x32(tO + 128 + c * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {                // entries past V are zero in both maps
            const float d = fmaf(-p.lambda, __uint_as_float(v[i]), o[c * 32 + i]);
            o[c * 32 + i] = d;
            ss = fmaf(d, d, ss);
          }
        }
        if (q_idx < p.S) {
          const float f = p.out_scale / sqrtf(ss / p.V + p.eps);
          __nv_bfloat16* op = p.O + ((long long)b * p.S + q_idx) * p.ldo + h * p.V;
#pragma unroll
          for (int c = 0; c < DV / 8; ++c) {
            if (c * 8 < p.V) {
              uint4 u;
              u.x = pack_bf16(o[c * 8 + 0] * f, o[c * 8 + 1] * f);
              u.y = pack_bf16(o[c * 8 + 2] * f, o[c * 8 + 3] * f);
              u.z = pack_bf16(o[c * 8 + 4] * f, o[c * 8 + 5] * f);
              u.w = pack_bf16(o[c * 8 + 6] * f, o[c * 8 + 7] * f);
              *reinterpret_cast<uint4*>(op + c * 8) = u;
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
    tmem_dealloc(tmem_base, 512);
  }
}

template <int DK, int DV, int BN>
static int launch_diff_fwd(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, int D,
                           const DiffFwdParams& p, cudaStream_t st) {
  using L = DiffSmem<DK, DV, BN>;
  static DeviceOnce once;
  auto kern = diff_attn_fwd_kernel<DK, DV, BN>;
  if (int e = ensure_dyn_smem(once, kern, L::TOTAL)) return e;
  CUtensorMap tq, tk, tv;
  int rc;
  const uint64_t d = D, vv = p.V, S = p.S, Skv = p.Skv, B = p.B;
  if ((rc = make_tmap_4d(&tq, q, 2, {d, uint64_t(2 * p.H), S, B}, {d * 2, uint64_t(ldq) * 2, uint64_t(ldq) * 2 * S}, {64, 1, DA_BM, 1}))) return rc;
  if ((rc = make_tmap_4d(&tk, k, 2, {d, uint64_t(2 * p.G), Skv, B}, {d * 2, uint64_t(ldk) * 2, uint64_t(ldk) * 2 * Skv}, {64, 1, BN, 1}))) return rc;
  if ((rc = make_tmap_4d(&tv, v, 2, {vv, uint64_t(p.G), Skv, B}, {vv * 2, uint64_t(ldv) * 2, uint64_t(ldv) * 2 * Skv}, {64, 1, BN, 1}))) return rc;
  launch_k(kern, ((p.S + DA_BM - 1) / DA_BM) * p.B * p.H, DA_THREADS, L::TOTAL, st, tq, tk, tv, p);
  return int(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------
// decoding on mma.sync
// ------------------------------------------------------------------------------------------------
struct DiffDecodeArgs {
  const __nv_bfloat16* q;   // [B, ldq]: H heads of [map 1 | map 2], D entries each
  long long ldq;
  const __nv_bfloat16 *kpool, *vpool;   // [slots][G][2 D], [slots][G][V]
  long long nslots;
  const int* block_table;
  int max_pages, page;
  const int* positions;     // [B] position of the query (it sees itself: its row is in the cache)
  int H, G, D, V, window, splits;
  float scale;
  float *acc, *ml;          // [B, G, chunks, splits, 16, V], [..., 16, 2]
  int* status;
};

constexpr int DD_THREADS = 128;
constexpr int DD_CHUNK = 32;

__device__ __forceinline__ void dd_ldsm(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void dd_ldsm_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void dd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// KS2: pairs of 16-entry k steps covering the 2 D entries of a key row (2 D <= 32 KS2); NV2: pairs of 8-entry value blocks
// (V <= 16 NV2).  Row pitches in shared memory are those sizes + 16 bytes, so that ldmatrix reads eight rows without bank
// conflicts; entries past 2 D (V) are zeroed once and never written again.
template <int KS2, int NV2>
__global__ void __launch_bounds__(DD_THREADS) diff_decode_kernel(const DiffDecodeArgs p) {
  tfb::pdl_sync();
  extern __shared__ __align__(128) uint8_t dsm[];
  constexpr int KP = KS2 * 64 + 16, VP = NV2 * 32 + 16;          // byte pitches
  constexpr int KTILE = DD_CHUNK * KP, VTILE = DD_CHUNK * VP, WARP = KTILE + VTILE;
  const int R = p.H / p.G, b = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int chunks = (R + 7) >> 3, g = blockIdx.y / chunks, rc = blockIdx.y % chunks, sp = blockIdx.z;
  const int nr = min(8, R - rc * 8);                             // query heads of this block
  const uint32_t s0 = smem_u32(dsm);
  const uint32_t sQ = s0, sK = s0 + 16 * KP + warp * WARP, sV = sK + KTILE;
  const uint32_t bar_k = s0 + 16 * KP + (DD_THREADS / 32) * WARP + warp * 16, bar_v = bar_k + 8;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(dsm + 16 * KP + (DD_THREADS / 32) * WARP + 64);
  if (lane == 0) {
    mbar_init(bar_k, 1);
    mbar_init(bar_v, 1);
    if (warp == 0) *abort_flag = 0;
    mbar_fence_init();
  }
  for (int i = tid; i < (16 * KP + (DD_THREADS / 32) * WARP) / 16; i += DD_THREADS)
    reinterpret_cast<uint4*>(dsm)[i] = make_uint4(0u, 0u, 0u, 0u);
  const int pos = p.positions[b];
  const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;          // oldest visible key
  const int base = first / p.page * p.page;                                   // chunks start on a page border
  const int span = pos + 1 - base;
  const int per = ((span + p.splits - 1) / p.splits + DD_CHUNK - 1) / DD_CHUNK * DD_CHUNK;
  const int t_begin = base + sp * per, t_end = min(pos + 1, t_begin + per);
  const int* bt = p.block_table + (long long)b * p.max_pages;
  __syncthreads();
  {
    const int per_map = p.D / 8;                                  // 16-byte pieces
    for (int i = tid; i < 2 * nr * per_map; i += DD_THREADS) {
      const int t = i / (nr * per_map), j = i - t * nr * per_map, r = j / per_map, c = j % per_map;
      const uint4 u = *reinterpret_cast<const uint4*>(p.q + (long long)b * p.ldq + (long long)((g * R + rc * 8 + r) * 2 + t) * p.D + c * 8);
      *reinterpret_cast<uint4*>(dsm + (t * 8 + r) * KP + t * p.D * 2 + c * 16) = u;
    }
  }
  fence_proxy_async_smem();                                       // the zeroed tiles are refilled by bulk copies
  __syncthreads();

  float o[2 * NV2][4];
#pragma unroll
  for (int n = 0; n < 2 * NV2; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};    // rows lane / 4 and lane / 4 + 8, log2 units
  const float sl2 = p.scale * LOG2E;
  const uint32_t kb = uint32_t(p.D) * 4, vb = uint32_t(p.V) * 2;     // bytes of a key / value row of one kv head

  // lane r brings row r of a chunk as one bulk copy; rows past the end keep the finite bytes of an earlier chunk (or zero)
  // and are masked in the scores, so that their probabilities are exactly zero
  auto page_for = [&](int t0, int nv) -> long long {
    long long page = lane < nv ? bt[(t0 + lane) / p.page] : 0;
    TFB_BOUNDS(page >= 0 && (page + 1) * p.page <= p.nslots, 52, page, p.nslots / p.page);
    if (page < 0 || (page + 1) * p.page > p.nslots) page = 0;
    return page;
  };
  auto issue = [&](const __nv_bfloat16* pool, uint32_t bytes, uint32_t pitch, long long page, int t0, int nv, uint32_t tile, uint32_t bar) {
    if (lane == 0) mbar_expect_tx(bar, uint32_t(nv) * bytes);
    __syncwarp();
    if (lane < nv) {
      const long long row = (page * p.page + (t0 + lane) % p.page) * p.G + g;
      bulk_load(tile + lane * pitch, pool + row * (bytes >> 1), bytes, bar);
    }
  };
  auto drain = [&](uint32_t ph) {
    const uint64_t t0 = globaltimer_ns();
    while (!(mbar_try_wait(bar_k, ph) && mbar_try_wait(bar_v, ph))) {
      if (globaltimer_ns() - t0 > 2000000ull) { report(p.status, ST_TIMEOUT_DRAIN); break; }
    }
  };
  constexpr int STEP = (DD_THREADS / 32) * DD_CHUNK;
  uint32_t phase = 0;
  const int t_first = t_begin + warp * DD_CHUNK;
  if (t_first < t_end) {
    const int nv = min(DD_CHUNK, t_end - t_first);
    const long long pg = page_for(t_first, nv);
    issue(p.kpool, kb, KP, pg, t_first, nv, sK, bar_k);
    issue(p.vpool, vb, VP, pg, t_first, nv, sV, bar_v);
  }
  for (int t0 = t_first; t0 < t_end; t0 += STEP) {
    const int nvalid = min(DD_CHUNK, t_end - t0), nv_next = min(DD_CHUNK, t_end - (t0 + STEP));
    const long long pg_next = nv_next > 0 ? page_for(t0 + STEP, nv_next) : 0;
    if (!mbar_wait_warp(bar_k, phase, abort_flag, p.status, ST_TIMEOUT_FULL)) { drain(phase); break; }
    float sc[DD_CHUNK / 8][4];
#pragma unroll
    for (int nb = 0; nb < DD_CHUNK / 8; ++nb) sc[nb][0] = sc[nb][1] = sc[nb][2] = sc[nb][3] = 0.f;
#pragma unroll
    for (int k2 = 0; k2 < KS2; ++k2) {
      if (k2 * 32 >= 2 * p.D) break;
      uint32_t a0[4], a1[4];
      const uint32_t qrow = sQ + ((lane & 7) + ((lane >> 3) & 1) * 8) * KP + (lane >> 4) * 16 + k2 * 64;
      dd_ldsm(qrow, a0);
      dd_ldsm(qrow + 32, a1);
#pragma unroll
      for (int nb = 0; nb < DD_CHUNK / 8; ++nb) {
        uint32_t kf[4];
        dd_ldsm(sK + (nb * 8 + (lane & 7)) * KP + k2 * 64 + (lane >> 3) * 16, kf);
        dd_mma(sc[nb], a0, kf[0], kf[1]);
        dd_mma(sc[nb], a1, kf[2], kf[3]);
      }
    }
    if (nv_next > 0) {                       // the K tile is free: fetch the next chunk's keys
      __syncwarp();
      fence_proxy_async_smem();
      issue(p.kpool, kb, KP, pg_next, t0 + STEP, nv_next, sK, bar_k);
    }
    float mx[2] = {m_run[0], m_run[1]};
#pragma unroll
    for (int nb = 0; nb < DD_CHUNK / 8; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int tok = nb * 8 + (lane & 3) * 2 + (e & 1);
        const float s = (tok < nvalid && t0 + tok >= first) ? sc[nb][e] * sl2 : -INFINITY;
        sc[nb][e] = s;
        mx[e >> 1] = fmaxf(mx[e >> 1], s);
      }
    float alpha[2], mb[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
      mb[i] = mx[i] == -INFINITY ? 0.f : mx[i];
      alpha[i] = m_run[i] == -INFINITY ? 0.f : exp2f(m_run[i] - mb[i]);
      m_run[i] = mx[i];
      l_run[i] *= alpha[i];
    }
    uint32_t pa[DD_CHUNK / 16][4];
#pragma unroll
    for (int nb = 0; nb < DD_CHUNK / 8; ++nb) {
      const float p0 = exp2f(sc[nb][0] - mb[0]), p1 = exp2f(sc[nb][1] - mb[0]);
      const float p2 = exp2f(sc[nb][2] - mb[1]), p3 = exp2f(sc[nb][3] - mb[1]);
      l_run[0] += p0 + p1;
      l_run[1] += p2 + p3;
      pa[nb >> 1][(nb & 1) * 2] = pack_bf16(p0, p1);
      pa[nb >> 1][(nb & 1) * 2 + 1] = pack_bf16(p2, p3);
    }
#pragma unroll
    for (int n = 0; n < 2 * NV2; ++n) {
      o[n][0] *= alpha[0];
      o[n][1] *= alpha[0];
      o[n][2] *= alpha[1];
      o[n][3] *= alpha[1];
    }
    if (!mbar_wait_warp(bar_v, phase, abort_flag, p.status, ST_TIMEOUT_FULL)) { drain(phase); break; }
    phase ^= 1u;
#pragma unroll
    for (int kk = 0; kk < DD_CHUNK / 16; ++kk)
#pragma unroll
      for (int n2 = 0; n2 < NV2; ++n2) {
        if (n2 * 16 >= p.V) break;
        uint32_t vf[4];
        dd_ldsm_t(sV + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VP + n2 * 32 + (lane >> 4) * 16, vf);
        dd_mma(o[2 * n2], pa[kk], vf[0], vf[1]);
        dd_mma(o[2 * n2 + 1], pa[kk], vf[2], vf[3]);
      }
    __syncwarp();
    if (nv_next > 0) {
      fence_proxy_async_smem();
      issue(p.vpool, vb, VP, pg_next, t0 + STEP, nv_next, sV, bar_v);
    }
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
  }
  // ---- merge the four warps (the tiles are free now) ----
  __syncthreads();
  float* red_m = reinterpret_cast<float*>(dsm);          // [4][16]
  float* red_l = red_m + 64;                             // [4][16]
  float* red_o = red_l + 64;                             // [4][16][16 NV2]
  constexpr int OW = 16 * NV2;
  const int row = lane >> 2;
  if ((lane & 3) == 0) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      red_m[warp * 16 + row + 8 * i] = m_run[i];
      red_l[warp * 16 + row + 8 * i] = l_run[i];
    }
  }
#pragma unroll
  for (int n = 0; n < 2 * NV2; ++n)
#pragma unroll
    for (int i = 0; i < 2; ++i)
      *reinterpret_cast<float2*>(red_o + (warp * 16 + row + 8 * i) * OW + n * 8 + (lane & 3) * 2) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
  __syncthreads();
  const long long out = (((long long)b * p.G + g) * chunks + rc) * p.splits + sp;
  for (int rr = warp; rr < 16; rr += DD_THREADS / 32) {
    if ((rr & 7) >= nr) continue;
    float M = -INFINITY, f[4], Lsum = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) M = fmaxf(M, red_m[w * 16 + rr]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = red_m[w * 16 + rr];
      f[w] = mw == -INFINITY ? 0.f : exp2f(mw - M);
      Lsum = fmaf(red_l[w * 16 + rr], f[w], Lsum);
    }
    for (int c = lane; c < p.V; c += 32) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) v = fmaf(red_o[(w * 16 + rr) * OW + c], f[w], v);
      p.acc[(out * 16 + rr) * p.V + c] = v;
    }
    if (lane == 0) {
      p.ml[(out * 16 + rr) * 2] = M;
      p.ml[(out * 16 + rr) * 2 + 1] = Lsum;
    }
  }
}

// one warp per (sequence, head): merge the splits of both maps, difference, norm, scale
__global__ void __launch_bounds__(128) diff_combine_kernel(const float* __restrict__ acc, const float* __restrict__ ml, __nv_bfloat16* __restrict__ o,
                                                           long long ldo, int B, int H, int G, int V, int splits, float lambda, float out_scale,
                                                           float eps) {
  tfb::pdl_sync();
  const int i = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= B * H) return;
  const int b = i / H, h = i % H, R = H / G, chunks = (R + 7) >> 3, g = h / R, r = h % R;
  const long long base = (((long long)b * G + g) * chunks + (r >> 3)) * splits;
  float M[2] = {-INFINITY, -INFINITY}, L[2] = {0.f, 0.f};
  for (int s = 0; s < splits; ++s)
    for (int t = 0; t < 2; ++t) M[t] = fmaxf(M[t], ml[((base + s) * 16 + t * 8 + (r & 7)) * 2]);
  for (int s = 0; s < splits; ++s)
    for (int t = 0; t < 2; ++t) {
      const float* q = ml + ((base + s) * 16 + t * 8 + (r & 7)) * 2;
      if (q[0] != -INFINITY) L[t] = fmaf(q[1], exp2f(q[0] - M[t]), L[t]);
    }
  constexpr int MAXC = 8;          // V <= 256
  float d[MAXC], ss = 0.f;
#pragma unroll
  for (int c = 0; c < MAXC; ++c) {
    d[c] = 0.f;
    const int col = c * 32 + lane;
    if (col < V) {
      float a[2] = {0.f, 0.f};
      for (int s = 0; s < splits; ++s)
        for (int t = 0; t < 2; ++t) {
          const long long row = (base + s) * 16 + t * 8 + (r & 7);
          const float m = ml[row * 2];
          if (m != -INFINITY) a[t] = fmaf(acc[row * V + col], exp2f(m - M[t]), a[t]);
        }
      d[c] = a[0] / L[0] - lambda * (a[1] / L[1]);
      ss = fmaf(d[c], d[c], ss);
    }
  }
  const float f = out_scale / sqrtf(warp_add(ss) / V + eps);
#pragma unroll
  for (int c = 0; c < MAXC; ++c) {
    const int col = c * 32 + lane;
    if (col < V) o[(long long)b * ldo + h * V + col] = __float2bfloat16(d[c] * f);
  }
}

template <int KS2, int NV2>
static int launch_diff_decode(const DiffDecodeArgs& p, int B, cudaStream_t st) {
  constexpr int KP = KS2 * 64 + 16, VP = NV2 * 32 + 16;
  constexpr int SMEM = 16 * KP + (DD_THREADS / 32) * DD_CHUNK * (KP + VP) + 128;
  static_assert(SMEM >= int(sizeof(float)) * (128 + 4 * 16 * 16 * NV2), "the merge buffers reuse the tiles");
  static DeviceOnce once;
  auto kern = diff_decode_kernel<KS2, NV2>;
  if (int e = ensure_dyn_smem(once, kern, SMEM)) return e;
  const int chunks = (p.H / p.G + 7) / 8;
  launch_k(kern, dim3(B, p.G * chunks, p.splits), DD_THREADS, SMEM, st, p);
  return int(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------
// any sizes, fp32 arithmetic
// ------------------------------------------------------------------------------------------------
template <class T>
struct DiffAnyArgs {
  const T* q;               // [B*S, ldq]
  long long ldq;
  const T *k, *v;           // contiguous: [B*Skv, ldk], [B*Skv, ldv]; paged: pools [slots][G 2 D], [slots][G V]
  long long ldk, ldv, nslots;
  const int* block_table;   // paged only
  int max_pages, page;
  const int* positions;     // paged: position of the one query of each sequence
  T* o;
  long long ldo;
  int B, S, Skv, q_off, H, G, D, V, window;
  float scale, lambda, out_scale, eps;
};

constexpr int AN_Q = 16;    // query rows per block: positions of one head (prompts) or heads of one kv head (decoding)
constexpr int AN_K = 32;    // keys per tile

template <class T, bool PAGED>
__global__ void __launch_bounds__(128) diff_attn_any_kernel(const DiffAnyArgs<T> p) {
  tfb::pdl_sync();
  extern __shared__ float am[];
  const int D = p.D, V = p.V, R = p.H / p.G, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, DP = D + 1;
  float* sQ = am;                       // [2 AN_Q][D]
  float* sK = sQ + 2 * AN_Q * D;        // [2][AN_K][D + 1]
  float* sV = sK + 2 * AN_K * DP;       // [AN_K][V]
  float* sP = sV + AN_K * V;            // [2 AN_Q][AN_K]
  float* sO = sP + 2 * AN_Q * AN_K;     // [2 AN_Q][V]
  float* sA = sO + 2 * AN_Q * V;        // [2 AN_Q] rescale of this tile
  float* sL = sA + 2 * AN_Q;            // [2 AN_Q] row sums
  int b, g, h0, i0, n, lo_min, hi_max;
  if (PAGED) {
    const int chunks = (R + AN_Q - 1) / AN_Q;
    b = blockIdx.y;
    g = blockIdx.x / chunks;
    h0 = g * R + (blockIdx.x % chunks) * AN_Q;
    n = min(AN_Q, (g + 1) * R - h0);
    i0 = 0;
    hi_max = p.positions[b];
    lo_min = p.window > 0 ? max(0, hi_max - p.window + 1) : 0;
  } else {
    b = blockIdx.z;
    h0 = blockIdx.y;
    g = h0 / R;
    i0 = blockIdx.x * AN_Q;
    n = min(AN_Q, p.S - i0);
    hi_max = min(i0 + n - 1 + p.q_off, p.Skv - 1);
    lo_min = p.window > 0 ? max(0, i0 + p.q_off - p.window + 1) : 0;
  }
  for (int i = tid; i < 2 * AN_Q * D; i += 128) {
    const int rm = i / D, d = i % D, r = rm >> 1, t = rm & 1;
    float x = 0.f;
    if (r < n) {
      const long long row = PAGED ? b : (long long)b * p.S + i0 + r;
      const int h = PAGED ? h0 + r : h0;
      x = to_f(p.q[row * p.ldq + (long long)(2 * h + t) * D + d]);
    }
    sQ[i] = x;
  }
  for (int i = tid; i < 2 * AN_Q * V; i += 128) sO[i] = 0.f;
  float m_run[8], l_run[8];             // this warp's rows: warp, warp + 4, ...
#pragma unroll
  for (int i = 0; i < 8; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }
  for (int t0 = lo_min; t0 <= hi_max; t0 += AN_K) {
    const int nk = min(AN_K, hi_max + 1 - t0);
    __syncthreads();
    for (int i = tid; i < AN_K * 2 * D; i += 128) {
      const int j = i / (2 * D), e = i % (2 * D), t = e / D, d = e % D;
      float x = 0.f;
      if (j < nk) {
        long long row;
        if (PAGED) {
          long long page = p.block_table[(long long)b * p.max_pages + (t0 + j) / p.page];
          TFB_BOUNDS(page >= 0 && (page + 1) * p.page <= p.nslots, 52, page, p.nslots / p.page);
          if (page < 0 || (page + 1) * p.page > p.nslots) page = 0;
          row = page * p.page + (t0 + j) % p.page;
        } else {
          row = (long long)b * p.Skv + t0 + j;
        }
        x = to_f(p.k[row * p.ldk + (long long)g * 2 * D + e]);
      }
      sK[(t * AN_K + j) * DP + d] = x;
    }
    for (int i = tid; i < AN_K * V; i += 128) {
      const int j = i / V, d = i % V;
      float x = 0.f;
      if (j < nk) {
        long long row;
        if (PAGED) {
          long long page = p.block_table[(long long)b * p.max_pages + (t0 + j) / p.page];
          if (page < 0 || (page + 1) * p.page > p.nslots) page = 0;
          row = page * p.page + (t0 + j) % p.page;
        } else {
          row = (long long)b * p.Skv + t0 + j;
        }
        x = to_f(p.v[row * p.ldv + (long long)g * V + d]);
      }
      sV[i] = x;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int rm = warp + 4 * i, r = rm >> 1, t = rm & 1;
      const float* q = sQ + rm * D;
      const float* k = sK + (t * AN_K + lane) * DP;
      float s = 0.f;
      for (int d = 0; d < D; ++d) s = fmaf(q[d], k[d], s);
      const int hi = PAGED ? hi_max : i0 + r + p.q_off, lo = p.window > 0 ? hi - p.window + 1 : 0, j = t0 + lane;
      s = (r < n && lane < nk && j <= hi && j >= lo) ? s * p.scale : -INFINITY;
      const float mx = fmaxf(m_run[i], warp_max(s));
      const float mb = mx == -INFINITY ? 0.f : mx;
      const float a = m_run[i] == -INFINITY ? 0.f : expf(m_run[i] - mb);
      const float e = expf(s - mb);
      l_run[i] = fmaf(l_run[i], a, warp_add(e));
      m_run[i] = mx;
      sP[rm * AN_K + lane] = e;
      if (lane == 0) sA[rm] = a;
    }
    __syncthreads();
    for (int i = tid; i < 2 * AN_Q * V; i += 128) {
      const int rm = i / V, d = i % V;
      float acc = sO[i] * sA[rm];
#pragma unroll 8
      for (int j = 0; j < AN_K; ++j) acc = fmaf(sP[rm * AN_K + j], sV[j * V + d], acc);
      sO[i] = acc;
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (lane == 0) sL[warp + 4 * i] = l_run[i];
  __syncthreads();
  for (int r = warp; r < n; r += 4) {
    const float i1 = 1.f / sL[2 * r], i2 = p.lambda / sL[2 * r + 1];
    float ss = 0.f;
    for (int d = lane; d < V; d += 32) {
      const float x = sO[2 * r * V + d] * i1 - sO[(2 * r + 1) * V + d] * i2;
      sO[2 * r * V + d] = x;
      ss = fmaf(x, x, ss);
    }
    const float f = p.out_scale / sqrtf(warp_add(ss) / V + p.eps);
    const long long row = PAGED ? b : (long long)b * p.S + i0 + r;
    const int h = PAGED ? h0 + r : h0;
    for (int d = lane; d < V; d += 32) p.o[row * p.ldo + (long long)h * V + d] = from_f<T>(sO[2 * r * V + d] * f);
  }
}

template <class T, bool PAGED>
static int launch_any(const DiffAnyArgs<T>& p, cudaStream_t st) {
  const long long smem = 4ll * (2 * AN_Q * p.D + 2 * AN_K * (p.D + 1) + AN_K * p.V + 2 * AN_Q * AN_K + 2 * AN_Q * p.V + 4 * AN_Q);
  if (smem > 220 * 1024) return TFB_ERR_LIMIT;
  static DeviceOnce once;
  auto kern = diff_attn_any_kernel<T, PAGED>;
  if (int e = ensure_dyn_smem(once, kern, 220 * 1024)) return e;
  const int R = p.H / p.G;
  const dim3 grid = PAGED ? dim3(p.G * ((R + AN_Q - 1) / AN_Q), p.B) : dim3((p.S + AN_Q - 1) / AN_Q, p.H, p.B);
  launch_k(kern, grid, 128, size_t(smem), st, p);
  return int(cudaGetLastError());
}

static bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace tfb

using bf16 = __nv_bfloat16;

// q [B*S, ldq]: H heads of two maps of D entries; k [B*Skv, ldk]: G heads of two maps; v [B*Skv, ldv]: G heads of V entries.
// The queries are the last S of the Skv positions.  o [B*S, ldo]: H heads of V entries.  window 0: plain causal.
TFB_API int tfb_diff_attn_fwd(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, void* o, long long ldo,
                              int B, int S, int Skv, int H, int G, int D, int V, int window, float scale, float lambda, float out_scale,
                              float eps, int f32, int* status, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || S <= 0 || Skv < S || G <= 0 || H % G || H > 65535 || D <= 0 || V <= 0 || window < 0) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool tc = !f32 && D % 8 == 0 && V % 8 == 0 && D <= 128 && V <= 128 && ldq % 8 == 0 && ldk % 8 == 0 && ldv % 8 == 0 && ldo % 8 == 0 &&
                  al16(q) && al16(k) && al16(v) && al16(o);
  if (tc) {
    DiffFwdParams p{B, S, H, G, Skv, Skv - S, window, V, scale, lambda, out_scale, eps, static_cast<bf16*>(o), ldo, status};
    if (D <= 64) return V <= 64 ? launch_diff_fwd<64, 64, 128>(q, ldq, k, ldk, v, ldv, D, p, st) : launch_diff_fwd<64, 128, 128>(q, ldq, k, ldk, v, ldv, D, p, st);
    return V <= 64 ? launch_diff_fwd<128, 64, 64>(q, ldq, k, ldk, v, ldv, D, p, st) : launch_diff_fwd<128, 128, 64>(q, ldq, k, ldk, v, ldv, D, p, st);
  }
#define TFB_ANY(T)                                                                                                                     \
  launch_any<T, false>(DiffAnyArgs<T>{static_cast<const T*>(q), ldq, static_cast<const T*>(k), static_cast<const T*>(v), ldk, ldv, 0,  \
                                      nullptr, 0, 1, nullptr, static_cast<T*>(o), ldo, B, S, Skv, Skv - S, H, G, D, V, window, scale,  \
                                      lambda, out_scale, eps}, st)
  return f32 ? TFB_ANY(float) : TFB_ANY(bf16);
#undef TFB_ANY
}

// 1 when tfb_diff_decode takes the tensor-core form for these sizes (it then needs the acc / ml workspaces)
TFB_API int tfb_diff_decode_tc(int D, int V, int f32) { return !f32 && D % 8 == 0 && V % 8 == 0 && D <= 128 && V <= 256; }

// One query per sequence at positions[b] over the cached rows of pages [slots][G][2 D] / [slots][G][V].
TFB_API int tfb_diff_decode(const void* q, long long ldq, const void* kpool, const void* vpool, long long nslots, const int* block_table,
                            int max_pages, int page, const int* positions, void* o, long long ldo, float* acc, float* ml, int splits, int B,
                            int H, int G, int D, int V, int window, float scale, float lambda, float out_scale, float eps, int f32,
                            int* status, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || G <= 0 || H % G || D <= 0 || V <= 0 || window < 0 || page <= 0 || DD_CHUNK % page) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (tfb_diff_decode_tc(D, V, f32) && ldq % 8 == 0 && al16(q) && al16(kpool) && al16(vpool)) {
    if (!acc || !ml || splits < 1 || splits > 65535) return TFB_ERR_ARG;
    DiffDecodeArgs p{static_cast<const bf16*>(q), ldq, static_cast<const bf16*>(kpool), static_cast<const bf16*>(vpool), nslots, block_table,
                     max_pages, page, positions, H, G, D, V, window, splits, scale, acc, ml, status};
    int rc;
    if (D <= 64) rc = V <= 64 ? launch_diff_decode<4, 4>(p, B, st) : V <= 128 ? launch_diff_decode<4, 8>(p, B, st) : launch_diff_decode<4, 16>(p, B, st);
    else rc = V <= 128 ? launch_diff_decode<8, 8>(p, B, st) : launch_diff_decode<8, 16>(p, B, st);
    if (rc) return rc;
    launch_k(diff_combine_kernel, (B * H + 3) / 4, 128, 0, st, acc, ml, static_cast<bf16*>(o), ldo, B, H, G, V, splits, lambda, out_scale, eps);
    return int(cudaGetLastError());
  }
#define TFB_ANY(T)                                                                                                                          \
  launch_any<T, true>(DiffAnyArgs<T>{static_cast<const T*>(q), ldq, static_cast<const T*>(kpool), static_cast<const T*>(vpool),             \
                                     (long long)G * 2 * D, (long long)G * V, nslots, block_table, max_pages, page, positions,               \
                                     static_cast<T*>(o), ldo, B, 1, 0, 0, H, G, D, V, window, scale, lambda, out_scale, eps}, st)
  return f32 ? TFB_ANY(float) : TFB_ANY(bf16);
#undef TFB_ANY
}
