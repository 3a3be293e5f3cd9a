// Causal softmax attention with grouped key / value heads, keys and values of different sizes and a set of options:
//
//   window, keep_first  a query at position i sees the keys j with i - j < window or j < keep_first (window 0: all j <= i)
//   chunk               it sees the keys of its own chunk of positions (multiples of `chunk` on), and those first ones
//   softcap             scores become cap tanh(score / cap)
//   sink                the denominator counts one more key without a value, of score 0 or of a score per head
//   temp                the query at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1)
//   gate                heads (one logit each) or their entries (one logit each) are multiplied by its sigmoid
//
//   head_attn_fwd      prompts, bf16, tcgen05: one CTA per (sequence, head, 256 queries) as two 128-query tiles that share every key /
//                      value tile and take turns on the tensor core; key tiles that no query sees are skipped; scores, options
//                      and sums are fp32, the gate is applied in the epilogue
//   head_decode        one query per sequence over paged keys and values, bf16, mma.sync: the query heads of a kv head are the rows of a
//                      16-row tile; each warp streams every fourth 32-key chunk through bulk copies of its own.  Split over the
//                      keys; head_combine merges the splits and applies sink and gate.
//   head_any           any sizes, bf16 or fp32, prompts or decoding: fp32 FMA throughout, online softmax over 32-key tiles.
#include "tfb_elem.cuh"
#include "tfb_host.h"
#include "tfb_mma.cuh"

namespace tfb {
TFB_BOUNDS_DEFINE(head_attention)

constexpr float LOG2E = 1.4426950408889634f;

struct HeadOpt {
  int window, chunk, keep;
  float cap;
  int sink;               // 1: score 0; 2: sinks[h]
  const void* sinks;      // [H], in the type of the queries
  float temp_coef;
  int temp_every;

  // the first key that the query behind key i sees, kept ones aside (i, like the keys, counted from a multiple of `chunk`)
  __host__ __device__ __forceinline__ int first_key(int i) const {
    return window > 0 ? (i >= window ? i - window + 1 : 0) : chunk > 0 ? i - i % chunk : 0;
  }
  __host__ __device__ __forceinline__ bool bounded() const { return window > 0 || chunk > 0; }
};

template <class T>
__device__ __forceinline__ float sink_score(const HeadOpt& o, int h) { return o.sink == 2 ? to_f(static_cast<const T*>(o.sinks)[h]) : 0.f; }

__device__ __forceinline__ float query_temp(const HeadOpt& o, int pos) {
  return o.temp_coef == 0.f ? 1.f : fmaf(o.temp_coef, logf(float((pos + 1) / o.temp_every + 1)), 1.f);
}

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// for the output gates; relative error about 3e-7
__device__ __forceinline__ float sigmoid_gate(float x) { return rcp(1.f + ex2(-LOG2E * x)); }

// tanh by its definition; absolute error about 2e-7
__device__ __forceinline__ float tanh_any(float x) {
  const float t = fmaf(-2.f, rcp(1.f + ex2(2.f * LOG2E * fabsf(x))), 1.f);
  return copysignf(t, x);
}
// tanh of a pair with |x| <= 1: x P(x^2), P of degree six by Chebyshev interpolation of tanh(x) / x over x^2 in [0, 1]; absolute
// error below 2e-7.  On the FMA pipe: the exponentials of the softmax have the other one to themselves.
__device__ __forceinline__ u64 tanh2_small(u64 x) {
  const float c[7] = {0.9999999403953552f, -0.33332857489585876f, 0.13325397670269012f, -0.05346517637372017f, 0.020305519923567772f,
                      -0.006217069923877716f, 0.0010455535957589746f};
  const u64 y = mul2(x, x);
  u64 p = pack2(c[6], c[6]);
#pragma unroll
  for (int i = 5; i >= 0; --i) p = fma2(p, y, pack2(c[i], c[i]));
  return mul2(p, x);
}

// keys of a 32-key piece that a query sees: bits lo .. hi and 0 .. keep - 1 (indices relative to the piece)
__device__ __forceinline__ uint32_t low_bits(int n) { return n <= 0 ? 0u : (n >= 32 ? 0xffffffffu : (1u << n) - 1u); }
__device__ __forceinline__ uint32_t seen_bits(int lo, int hi, int keep) { return low_bits(hi + 1) & (~low_bits(lo) | low_bits(keep)); }

// ------------------------------------------------------------------------------------------------
// prompts on tcgen05
// ------------------------------------------------------------------------------------------------
struct HeadAttnParams {
  int B, S, H, G;
  int Skv, q_off;         // keys per sequence; query i sees keys 0 .. i + q_off
  int D, V;
  float scale;
  HeadOpt opt;
  int pos0;               // position of the first query
  const __nv_bfloat16* gate;    // [B*S, ldg] or null
  long long ldg;
  int gate_entry;         // one logit per entry of the heads (otherwise one per head)
  __nv_bfloat16* O;
  long long ldo;
  int* status;
};

constexpr int HA_THREADS = 320;
constexpr int HA_BM = 128, HA_BN = 128;
constexpr int HA_BOX = 128 * 128;       // bytes of 128 rows of 64 entries

template <int DK, int DV>
struct HeadSmem {
  static constexpr int NBK = DK / 64, NBV = DV / 64;
  static constexpr int QT = NBK * HA_BOX, KT = NBK * HA_BOX, VT = NBV * HA_BOX, STAGE = KT + VT;
  static constexpr int AVAIL = 227 * 1024 - 1024 - 256 - 2 * QT;
  static constexpr int STAGES = AVAIL / STAGE > 4 ? 4 : AVAIL / STAGE;
  static constexpr int KV_OFF = 2 * QT;
  static constexpr int BAR_OFF = KV_OFF + STAGES * STAGE;
  static constexpr int TOTAL = BAR_OFF + 256 + 1024;
  static_assert(STAGES >= 2, "two stages at least");
};

// Of the 128 scores of this thread's row: the running maximum and the largest magnitude (CAP).  MASK: only the keys that the row sees
// (indices within the tile) count.
template <bool MASK, bool CAP>
__device__ __forceinline__ float2 tile_max(uint32_t tS, float m, int lo, int hi, int keep) {
  float mx0 = m, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY, big0 = 0.f, big1 = 0.f;
#pragma unroll 1
  for (int c = 0; c < HA_BN / 32; ++c) {
    uint32_t v[32];
    tmem_ld_32x32(tS + c * 32, v);
    tmem_ld_wait();
    if (CAP) {
#pragma unroll
      for (int i = 0; i < 32; i += 4) {
        big0 = fmax3(big0, fabsf(__uint_as_float(v[i])), fabsf(__uint_as_float(v[i + 1])));
        big1 = fmax3(big1, fabsf(__uint_as_float(v[i + 2])), fabsf(__uint_as_float(v[i + 3])));
      }
    }
    if (MASK) {
      const uint32_t seen = seen_bits(lo - c * 32, hi - c * 32, keep - c * 32);
#pragma unroll
      for (int i = 0; i < 32; ++i)
        if (!(seen >> i & 1u)) v[i] = 0xff800000u;
    }
#pragma unroll
    for (int i = 0; i < 32; i += 8) {
      mx0 = fmax3(mx0, __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
      mx1 = fmax3(mx1, __uint_as_float(v[i + 2]), __uint_as_float(v[i + 3]));
      mx2 = fmax3(mx2, __uint_as_float(v[i + 4]), __uint_as_float(v[i + 5]));
      mx3 = fmax3(mx3, __uint_as_float(v[i + 6]), __uint_as_float(v[i + 7]));
    }
  }
  return make_float2(fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)), fmaxf(big0, big1));
}

// p = 2^(s * sl2 - mb), or 2^(kc tanh(s * sl2) - mb) with CAP 1 (|s * sl2| <= 1) and 2 (any), over the row, written back over the scores
// as bf16 pairs; returns the row sum
template <bool MASK, int CAP>
__device__ __forceinline__ float tile_probs(uint32_t tS, float sl2, float kc, float mb, int lo, int hi, int keep) {
  float rs[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 1
  for (int c = 0; c < HA_BN / 32; ++c) {
    uint32_t v[32], pk[16];
    tmem_ld_32x32(tS + c * 32, v);
    tmem_ld_wait();
    const uint32_t seen = MASK ? seen_bits(lo - c * 32, hi - c * 32, keep - c * 32) : 0u;
#pragma unroll
    for (int i = 0; i < 16; i += 2) {
      float q[4];
      if constexpr (CAP == 1) {
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const u64 x = mul2(pack2(__uint_as_float(v[2 * i + e]), __uint_as_float(v[2 * i + e + 1])), pack2(sl2, sl2));
          const float2 t = unpack2(fma2(tanh2_small(x), pack2(kc, kc), pack2(-mb, -mb)));
          q[e] = ex2(t.x);
          q[e + 1] = ex2(t.y);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if constexpr (CAP == 0) q[e] = ex2(fmaf(__uint_as_float(v[2 * i + e]), sl2, -mb));
        if constexpr (CAP == 2) q[e] = ex2(fmaf(tanh_any(__uint_as_float(v[2 * i + e]) * sl2), kc, -mb));
        if (MASK && !(seen >> (2 * i + e) & 1u)) q[e] = 0.f;
        rs[e] += q[e];
      }
      pk[i] = pack_bf16(q[0], q[1]);
      pk[i + 1] = pack_bf16(q[2], q[3]);
    }
    tmem_st_32x16(tS + c * 16, pk);
  }
  return (rs[0] + rs[1]) + (rs[2] + rs[3]);
}

// MODE 0: causal, a gate per head at most; 1: all options but the cap; 2: all of them
template <int DK, int DV, int MODE>
__global__ void __launch_bounds__(HA_THREADS, 1)
head_attn_fwd_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk, const __grid_constant__ CUtensorMap tv,
                     const HeadAttnParams p) {
  using L = HeadSmem<DK, DV>;
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
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 1 + 2 * ST + 6);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int npair = (p.S + 2 * HA_BM - 1) / (2 * HA_BM);
  const int bh = p.B * p.H;
  const int pair = npair - 1 - int(blockIdx.x) / bh;   // the longest (latest) query blocks first
  const int rem = int(blockIdx.x) % bh;
  const int b = rem / p.H, h = rem % p.H, hk = h / (p.H / p.G);
  // key blocks: those of the kept first keys, then from the window of the first query on
  int lo_blk = 0, n_first = 0;
  if (MODE > 0 && p.opt.bounded()) {
    lo_blk = p.opt.first_key(pair * 2 * HA_BM + p.q_off) / HA_BN;
    n_first = min((p.opt.keep + HA_BN - 1) / HA_BN, lo_blk);
  }
  auto block_of = [&](int j) { return j < n_first ? j : lo_blk + j - n_first; };
  int n_t[2];                                          // key blocks each tile visits (0: the tile lies past the end)
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    const int q0 = (pair * 2 + t) * HA_BM;
    n_t[t] = q0 >= p.S ? 0 : n_first + (min(q0 + HA_BM, p.S) - 1 + p.q_off) / HA_BN + 1 - lo_blk;
  }
  const int n_kv = max(n_t[0], n_t[1]);

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
        for (int i = 0; i < L::NBK; ++i) tma_load_4d(sQ + t * L::QT + i * HA_BOX, &tq, bar_q, i * 64, h, (pair * 2 + t) * HA_BM, b);
      for (int j = 0; j < n_kv; ++j) {
        const int st = j % ST;
        if (!mbar_wait(bar_kv_empty + st * 8, ((j / ST) & 1) ^ 1, abort_flag, p.status, ST_TIMEOUT_EMPTY)) break;
        const uint32_t fb = bar_kv_full + st * 8, base = sQ + L::KV_OFF + st * L::STAGE;
        mbar_expect_tx(fb, L::STAGE);
#pragma unroll
        for (int i = 0; i < L::NBK; ++i) tma_load_4d(base + i * HA_BOX, &tk, fb, i * 64, hk, block_of(j) * HA_BN, b);
#pragma unroll
        for (int i = 0; i < L::NBV; ++i) tma_load_4d(base + L::KT + i * HA_BOX, &tv, fb, i * 64, hk, block_of(j) * HA_BN, b);
      }
      if (*abort_flag) {  // unwinding: bounded wait for copies already issued
        const uint64_t t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 200000ull) {}
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc(FMT_BF16, FMT_BF16, false, false, HA_BM, HA_BN);
      constexpr uint32_t idesc_o = umma_idesc(FMT_BF16, FMT_BF16, false, true, HA_BM, DV);
      auto issue_s = [&](int t, int j) {
        const uint32_t sK = sQ + L::KV_OFF + (j % ST) * L::STAGE, sQt = sQ + t * L::QT, tS = tS0 + t * 128;
#pragma unroll
        for (int k = 0; k < DK / 16; ++k) {
          if (k * 16 >= p.D) break;                  // entries past the head are zeros
          const uint32_t off = (k >> 2) * HA_BOX + (k & 3) * 32;
          umma_f16_ss(tS, umma_smem_desc(sQt + off, 16, 1024), umma_smem_desc(sK + off, 16, 1024), idesc_s, k > 0);
        }
        umma_commit(bar_s_full + t * 8);
      };
      bool ok = mbar_wait(bar_q, 0, abort_flag, p.status, ST_TIMEOUT_FULL) &&
                mbar_wait(bar_kv_full, 0, abort_flag, p.status, ST_TIMEOUT_FULL);
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int t = 0; t < 2; ++t)
          if (n_t[t] > 0) issue_s(t, 0);
      }
      for (int j = 0; j < n_kv && ok; ++j) {
        if (j + 1 < n_kv) {
          const int st1 = (j + 1) % ST;
          if (!mbar_wait(bar_kv_full + st1 * 8, ((j + 1) / ST) & 1, abort_flag, p.status, ST_TIMEOUT_FULL)) break;
          tc_fence_after();
        }
        const int st = j % ST;
        const uint32_t sV = sQ + L::KV_OFF + st * L::STAGE + L::KT;
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          if (!ok || j >= n_t[t]) continue;
          if (!mbar_wait(bar_p_ready + t * 8, j & 1, abort_flag, p.status, ST_TIMEOUT_TMEM_EMPTY)) {
            ok = false;
            continue;
          }
          tc_fence_after();
          const uint32_t tP = tS0 + t * 128, tO = tO0 + t * 128;
#pragma unroll
          for (int k = 0; k < HA_BN / 16; ++k)     // V tile: [key rows][64-column boxes], MN-major B
            umma_f16_ts(tO, tP + k * 8, umma_smem_desc(sV + k * 2048, HA_BOX, 1024), idesc_o, k > 0);
          if (j + 1 < n_t[t]) issue_s(t, j + 1);   // its commit also covers the P V product above
          else umma_commit(bar_o_full + t * 8);
        }
        if (ok) umma_commit(bar_kv_empty + st * 8);
      }
    }
  } else {
    const int t = (warp - 2) >> 2, quad = warp & 3, r = quad * 32 + lane;
    const int q0 = (pair * 2 + t) * HA_BM, q_idx = q0 + r;
    const int n_mine = t ? n_t[1] : n_t[0];
    const uint32_t lane_off = uint32_t(quad * 32) << 16;
    const uint32_t tS = tS0 + t * 128 + lane_off, tO = tO0 + t * 128 + lane_off;
    const float temp = MODE > 0 ? query_temp(p.opt, p.pos0 + q_idx) : 1.f;
    const float kc = MODE == 2 ? p.opt.cap * LOG2E : 0.f;
    const float sl2 = MODE == 2 ? p.scale * temp / p.opt.cap : p.scale * temp * LOG2E;
    const int hi_g = min(q_idx + p.q_off, p.Skv - 1);
    const bool bounded = MODE > 0 && p.opt.bounded();
    const int keep_g = bounded ? p.opt.keep : 0, lo_g = bounded ? p.opt.first_key(q_idx + p.q_off) : 0;
    const int lo_last = bounded ? p.opt.first_key(q0 + HA_BM - 1 + p.q_off) : 0;      // of the tile's last row
    float m = -INFINITY, l = 0.f, alpha_prev = 1.f, mb_prev = 0.f;
    float o[DV];
#pragma unroll
    for (int i = 0; i < DV; ++i) o[i] = 0.f;
    bool ok = true;
    for (int j = 0; j < n_mine; ++j) {
      if (!mbar_wait_warp(bar_s_full + t * 8, j & 1, abort_flag, p.status, ST_TIMEOUT_TMEM_FULL)) {
        ok = false;
        break;
      }
      tc_fence_after();
      const int k0 = block_of(j) * HA_BN, hi = hi_g - k0, lo = lo_g - k0, keep = keep_g - k0;
      const bool need_mask = k0 + HA_BN - 1 > q0 + p.q_off || k0 + HA_BN > p.Skv ||
                             (bounded && lo_last > k0 && k0 + HA_BN > keep_g);
      // a row may see no key of a block (a query past the end of its sequence, whose row is not stored, or a block before the window
      // of a later query)
      const float2 mxb = need_mask ? tile_max<true, MODE == 2>(tS, m, lo, hi, keep) : tile_max<false, MODE == 2>(tS, m, lo, hi, keep);
      const float mx = mxb.x;
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
      const float mb = (mx == -INFINITY) ? 0.f : (MODE == 2 ? kc * tanh_any(mx * sl2) : mx * sl2);
      const float alpha = (m == -INFINITY) ? 0.f : ex2(mb_prev - mb);
      float rs;
      if constexpr (MODE == 2) {
        if (__any_sync(0xffffffffu, mxb.y * sl2 > 1.f))
          rs = need_mask ? tile_probs<true, 2>(tS, sl2, kc, mb, lo, hi, keep) : tile_probs<false, 2>(tS, sl2, kc, mb, lo, hi, keep);
        else
          rs = need_mask ? tile_probs<true, 1>(tS, sl2, kc, mb, lo, hi, keep) : tile_probs<false, 1>(tS, sl2, kc, mb, lo, hi, keep);
      } else {
        rs = need_mask ? tile_probs<true, 0>(tS, sl2, kc, mb, lo, hi, keep) : tile_probs<false, 0>(tS, sl2, kc, mb, lo, hi, keep);
      }
      mb_prev = mb;
      l = fmaf(l, alpha, rs);
      m = mx;
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(bar_p_ready + t * 8);
      alpha_prev = alpha;
    }
    if (ok && n_mine > 0 && mbar_wait_warp(bar_o_full + t * 8, 0, abort_flag, p.status, ST_TIMEOUT_TMEM_FULL)) {
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(tO + c * 32, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c * 32 + i] = fmaf(o[c * 32 + i], alpha_prev, __uint_as_float(v[i]));
      }
      if (q_idx < p.S) {
        const long long row = (long long)b * p.S + q_idx;
        float f = l > 0.f ? 1.f / l : 0.f;
        if (MODE > 0 && p.opt.sink) {
          const float sk = sink_score<__nv_bfloat16>(p.opt, h) * LOG2E, M = fmaxf(mb_prev, sk), fm = ex2(mb_prev - M);
          f = fm / fmaf(l, fm, ex2(sk - M));
        }
        if (p.gate && !(MODE > 0 && p.gate_entry)) f *= sigmoid_exact(__bfloat162float(p.gate[row * p.ldg + h]));
        __nv_bfloat16* op = p.O + row * p.ldo + h * p.V;
#pragma unroll
        for (int c = 0; c < DV / 8; ++c) {
          if (c * 8 < p.V) {
            if (MODE > 0 && p.gate_entry) {
              float g[8];
              load_n<8>(p.gate + row * p.ldg + h * p.V + c * 8, g);
#pragma unroll
              for (int e = 0; e < 8; ++e) o[c * 8 + e] *= sigmoid_gate(g[e]);
            }
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

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int DK, int DV, int MODE>
static int launch_head_attn(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const HeadAttnParams& p,
                            cudaStream_t st) {
  using L = HeadSmem<DK, DV>;
  static DeviceOnce once;
  auto kern = head_attn_fwd_kernel<DK, DV, MODE>;
  if (int e = ensure_dyn_smem(once, kern, L::TOTAL)) return e;
  CUtensorMap tq, tk, tv;
  int rc;
  const uint64_t d = p.D, vv = p.V, S = p.S, Skv = p.Skv, B = p.B;
  if ((rc = make_tmap_4d(&tq, q, 2, {d, uint64_t(p.H), S, B}, {d * 2, uint64_t(ldq) * 2, uint64_t(ldq) * 2 * S}, {64, 1, HA_BM, 1}))) return rc;
  if ((rc = make_tmap_4d(&tk, k, 2, {d, uint64_t(p.G), Skv, B}, {d * 2, uint64_t(ldk) * 2, uint64_t(ldk) * 2 * Skv}, {64, 1, HA_BN, 1}))) return rc;
  if ((rc = make_tmap_4d(&tv, v, 2, {vv, uint64_t(p.G), Skv, B}, {vv * 2, uint64_t(ldv) * 2, uint64_t(ldv) * 2 * Skv}, {64, 1, HA_BN, 1}))) return rc;
  launch_k(kern, ((p.S + 2 * HA_BM - 1) / (2 * HA_BM)) * p.B * p.H, HA_THREADS, L::TOTAL, st, tq, tk, tv, p);
  return int(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------
// decoding over paged keys and values
// ------------------------------------------------------------------------------------------------
struct HeadDecodeArgs {
  const __nv_bfloat16* q;     // [B, ldq]: H heads of D entries
  long long ldq;
  const __nv_bfloat16 *k, *v; // [slots][G D], [slots][G V]
  long long nslots;
  const int* block_table;
  int max_pages, page;
  const int* positions;       // [B] position of the query (it sees itself: its row is in the cache)
  int H, G, D, V, splits;
  float scale;
  HeadOpt opt;
  float *acc, *ml;            // [B, H, splits, V], [B, H, splits, 2]: unnormalised sums; maximum (log2 units), sum
  int* status;
};

constexpr int HD_THREADS = 128, HD_WARPS = HD_THREADS / 32, HD_CHUNK = 32;

// DK, DV: entries of a key / value row in shared memory (zeros past D / V); RT: query heads of a block (8 or 16)
template <int DK, int DV>
struct DecodeSmem {
  static constexpr int KP = DK * 2 + 16, VP = DV * 2 + 16;     // byte pitches: ldmatrix reads eight rows without bank conflicts
  static constexpr int KT = HD_CHUNK * KP, VT = HD_CHUNK * VP;
  static constexpr int Q = 16 * KP, BAR = Q + HD_WARPS * (KT + VT), TOTAL = BAR + 128;
  static_assert(BAR >= 4 * HD_WARPS * 16 * (DV + 2), "the merge buffers reuse the staging area");
};

template <int DK, int DV, int RT>
__global__ void __launch_bounds__(HD_THREADS) head_decode_kernel(const HeadDecodeArgs p) {
  tfb::pdl_sync();
  using L = DecodeSmem<DK, DV>;
  constexpr int KS = DK / 16, NB = DV / 8, NR = RT / 8;        // k steps, 8-column blocks of the output, rows of a thread
  extern __shared__ __align__(128) uint8_t sm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int R = p.H / p.G, chunks = (R + RT - 1) / RT;
  const int b = blockIdx.x, g = blockIdx.y / chunks, h0 = g * R + blockIdx.y % chunks * RT, sp = blockIdx.z;
  const int rows = min(RT, (g + 1) * R - h0);
  const uint32_t s0 = smem_u32(sm), sK = s0 + L::Q + warp * (L::KT + L::VT), sV = sK + L::KT;
  uint8_t* tileK = sm + L::Q + warp * (L::KT + L::VT);
  uint8_t* tileV = tileK + L::KT;
  const uint32_t bar_k = s0 + L::BAR + warp * 16, bar_v = bar_k + 8;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(sm + L::BAR + 64);
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  if (lane == 0) {
    mbar_init(bar_k, 1);
    mbar_init(bar_v, 1);
    if (warp == 0) *abort_flag = 0;
    mbar_fence_init();
  }
  // what no copy writes but the products read: entries past D and V
  for (int i = lane; i < HD_CHUNK * ((DK - p.D) / 8); i += 32)
    *reinterpret_cast<uint4*>(tileK + i % HD_CHUNK * L::KP + p.D * 2 + i / HD_CHUNK * 16) = zero;
  for (int i = lane; i < HD_CHUNK * ((DV - p.V) / 8); i += 32)
    *reinterpret_cast<uint4*>(tileV + i % HD_CHUNK * L::VP + p.V * 2 + i / HD_CHUNK * 16) = zero;
  for (int i = tid; i < 16 * (DK / 8); i += HD_THREADS) {
    const int r = i / (DK / 8), c = i % (DK / 8) * 8;
    *reinterpret_cast<uint4*>(sm + r * L::KP + c * 2) =
        (r < rows && c < p.D) ? *reinterpret_cast<const uint4*>(p.q + b * p.ldq + (long long)(h0 + r) * p.D + c) : zero;
  }
  __syncthreads();
  uint32_t qa[KS][4];
#pragma unroll
  for (int k = 0; k < KS; ++k) ldsm(s0 + ((lane & 7) + ((lane >> 3) & 1) * 8) * L::KP + k * 32 + (lane >> 4) * 16, qa[k]);

  // the keys that the query sees, in order: the kept first ones, then the window
  const int pos = p.positions[b], lo = p.opt.first_key(pos), first = min(p.opt.bounded() ? p.opt.keep : 0, lo);
  const int total = first + pos + 1 - lo;
  const int per = ((total + p.splits - 1) / p.splits + HD_CHUNK - 1) / HD_CHUNK * HD_CHUNK;
  const int t_begin = sp * per, t_end = min(total, t_begin + per);
  const float temp = query_temp(p.opt, pos);
  const float kc = p.opt.cap > 0.f ? p.opt.cap * LOG2E : 0.f, sl2 = p.opt.cap > 0.f ? p.scale * temp / p.opt.cap : p.scale * temp * LOG2E;
  const int* bt = p.block_table + (long long)b * p.max_pages;

  auto slot_of = [&](int t) -> long long {       // cache slot of the t-th key
    const int at = t < first ? t : t - first + lo;
    long long page = bt[at / p.page];
    TFB_BOUNDS(page >= 0 && (page + 1) * p.page <= p.nslots, 52, page, p.nslots / p.page);
    if (page < 0 || (page + 1) * p.page > p.nslots) page = 0;
    return page * p.page + at % p.page;
  };
  // lane r sends row r of a chunk; rows past the end are zeros
  auto issue = [&](const __nv_bfloat16* pool, int width, uint8_t* tile, uint32_t s_tile, int pitch, long long slot, int nv, uint32_t bar) {
    if (lane == 0) mbar_expect_tx(bar, uint32_t(nv) * width * 2);
    __syncwarp();
    if (lane < nv) bulk_load(s_tile + lane * pitch, pool + (slot * p.G + g) * width, width * 2, bar);
    else
      for (int c = 0; c < width * 2; c += 16) *reinterpret_cast<uint4*>(tile + lane * pitch + c) = zero;
  };
  auto drain = [&](uint32_t ph) {                // after a wait that ran out: a bounded time for the copies still in flight
    const uint64_t t0 = globaltimer_ns();
    while (!(mbar_try_wait(bar_k, ph) && mbar_try_wait(bar_v, ph))) {
      if (globaltimer_ns() - t0 > 2000000ull) { report(p.status, ST_TIMEOUT_DRAIN); break; }
    }
  };

  float o[NB][4];
#pragma unroll
  for (int n = 0; n < NB; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m_run[NR], l_run[NR];                    // rows lane / 4 (and + 8); l over this thread's columns
#pragma unroll
  for (int i = 0; i < NR; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }
  constexpr int STEP = HD_WARPS * HD_CHUNK;
  uint32_t phase = 0;
  const int t_first = t_begin + warp * HD_CHUNK;
  if (t_first < t_end) {
    const int nv = min(HD_CHUNK, t_end - t_first);
    const long long slot = lane < nv ? slot_of(t_first + lane) : 0;
    issue(p.k, p.D, tileK, sK, L::KP, slot, nv, bar_k);
    issue(p.v, p.V, tileV, sV, L::VP, slot, nv, bar_v);
  }
  for (int t0 = t_first; t0 < t_end; t0 += STEP) {
    const int nvalid = min(HD_CHUNK, t_end - t0), nv_next = min(HD_CHUNK, t_end - (t0 + STEP));    // <= 0: the warp's last chunk
    const long long slot_next = lane < nv_next ? slot_of(t0 + STEP + lane) : 0;
    if (!mbar_wait_warp(bar_k, phase, abort_flag, p.status, ST_TIMEOUT_FULL)) { drain(phase); break; }
    __syncwarp();
    float sc[HD_CHUNK / 8][4];
#pragma unroll
    for (int n = 0; n < HD_CHUNK / 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
    for (int k = 0; k < KS / 2; ++k) {
#pragma unroll
      for (int n = 0; n < HD_CHUNK / 8; ++n) {
        uint32_t f[4];
        ldsm(sK + (n * 8 + (lane & 7)) * L::KP + k * 64 + (lane >> 3) * 16, f);
        mma_bf16(sc[n], qa[2 * k], f[0], f[1]);
        mma_bf16(sc[n], qa[2 * k + 1], f[2], f[3]);
      }
    }
    if (nv_next > 0) {                           // the key tile is free: fetch the next chunk's keys
      __syncwarp();
      fence_proxy_async_smem();
      issue(p.k, p.D, tileK, sK, L::KP, slot_next, nv_next, bar_k);
    }
    float alpha[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      float mx = m_run[i];
#pragma unroll
      for (int n = 0; n < HD_CHUNK / 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float x = sc[n][2 * i + e] * sl2;
          if (kc > 0.f) x = kc * tanh_any(x);
          x = n * 8 + (lane & 3) * 2 + e < nvalid ? x : -INFINITY;
          sc[n][2 * i + e] = x;
          mx = fmaxf(mx, x);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      alpha[i] = ex2(m_run[i] - mx);             // finite mx: a chunk has a key
      m_run[i] = mx;
      l_run[i] *= alpha[i];
    }
    uint32_t pa[HD_CHUNK / 16][4];
#pragma unroll
    for (int n = 0; n < HD_CHUNK / 8; ++n)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        uint32_t w = 0u;
        if (i < NR) {
          const float p0 = ex2(sc[n][2 * i] - m_run[i < NR ? i : 0]), p1 = ex2(sc[n][2 * i + 1] - m_run[i < NR ? i : 0]);
          l_run[i < NR ? i : 0] += p0 + p1;
          w = pack_bf16(p0, p1);
        }
        pa[n >> 1][(n & 1) * 2 + i] = w;
      }
#pragma unroll
    for (int n = 0; n < NB; ++n)
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        o[n][2 * i] *= alpha[i];
        o[n][2 * i + 1] *= alpha[i];
      }
    if (!mbar_wait_warp(bar_v, phase, abort_flag, p.status, ST_TIMEOUT_FULL)) { drain(phase); break; }
    phase ^= 1u;
#pragma unroll
    for (int k = 0; k < HD_CHUNK / 16; ++k)
#pragma unroll
      for (int n = 0; n < NB / 2; ++n) {
        uint32_t f[4];
        ldsm_t(sV + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * L::VP + n * 32 + (lane >> 4) * 16, f);
        mma_bf16(o[2 * n], pa[k], f[0], f[1]);
        mma_bf16(o[2 * n + 1], pa[k], f[2], f[3]);
      }
    if (nv_next > 0) {
      __syncwarp();
      fence_proxy_async_smem();
      issue(p.v, p.V, tileV, sV, L::VP, slot_next, nv_next, bar_v);
    }
  }
  // merge the four warps (the staging area is free now)
  __syncthreads();
  float* red_m = reinterpret_cast<float*>(sm);               // [4][16]
  float* red_l = red_m + HD_WARPS * 16;                      // [4][16]
  float* red_o = red_l + HD_WARPS * 16;                      // [4][16][DV]
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
    const int row = (lane >> 2) + 8 * i;
    if ((lane & 3) == 0) {
      red_m[warp * 16 + row] = m_run[i];
      red_l[warp * 16 + row] = l_run[i];
    }
#pragma unroll
    for (int n = 0; n < NB; ++n)
      *reinterpret_cast<float2*>(red_o + (warp * 16 + row) * DV + n * 8 + (lane & 3) * 2) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
  }
  __syncthreads();
  const long long base = ((long long)b * p.H + h0) * p.splits + sp;
  for (int i = tid; i < rows * (p.V / 4); i += HD_THREADS) {
    const int r = i / (p.V / 4), d = i % (p.V / 4) * 4;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < HD_WARPS; ++w) M = fmaxf(M, red_m[w * 16 + r]);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    float sum = 0.f;
#pragma unroll
    for (int w = 0; w < HD_WARPS; ++w) {
      if (red_m[w * 16 + r] == -INFINITY) continue;
      const float f = ex2(red_m[w * 16 + r] - M);
      const float4 u = *reinterpret_cast<const float4*>(red_o + (w * 16 + r) * DV + d);
      v.x = fmaf(u.x, f, v.x);
      v.y = fmaf(u.y, f, v.y);
      v.z = fmaf(u.z, f, v.z);
      v.w = fmaf(u.w, f, v.w);
      sum = fmaf(red_l[w * 16 + r], f, sum);
    }
    *reinterpret_cast<float4*>(p.acc + (base + (long long)r * p.splits) * p.V + d) = v;
    if (d == 0) {
      p.ml[(base + (long long)r * p.splits) * 2] = M;
      p.ml[(base + (long long)r * p.splits) * 2 + 1] = sum;
    }
  }
}

// one warp per (sequence, head): merge the splits (at most 32), sink, gate
__global__ void __launch_bounds__(128) head_combine_kernel(const float* __restrict__ acc, const float* __restrict__ ml, const __nv_bfloat16* __restrict__ gate,
                                                           long long ldg, int gate_entry, __nv_bfloat16* __restrict__ o, long long ldo, int n, int H,
                                                           int V, int splits, const HeadOpt opt) {
  tfb::pdl_sync();
  const int id = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (id >= n) return;
  const int b = id / H, h = id % H;
  const long long base = (long long)id * splits;
  const float m = lane < splits ? ml[(base + lane) * 2] : -INFINITY;
  const float M = warp_max(m);
  float f = m == -INFINITY ? 0.f : ex2(m - M);
  float l = warp_add(lane < splits ? ml[(base + lane) * 2 + 1] * f : 0.f), fm = 1.f;
  if (opt.sink) {
    const float sk = sink_score<__nv_bfloat16>(opt, h) * LOG2E, M2 = fmaxf(M, sk);
    fm = ex2(M - M2);
    l = fmaf(l, fm, ex2(sk - M2));
  }
  f *= fm / l;
  if (gate && !gate_entry) f *= sigmoid_exact(__bfloat162float(gate[b * ldg + h]));
  for (int d = lane * 4; d < (V + 127) / 128 * 128; d += 128) {
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    for (int s = 0; s < splits; ++s) {
      const float fs = __shfl_sync(0xffffffffu, f, s);
      if (fs == 0.f || d >= V) continue;
      const float4 u = *reinterpret_cast<const float4*>(acc + (base + s) * V + d);
      v[0] = fmaf(u.x, fs, v[0]);
      v[1] = fmaf(u.y, fs, v[1]);
      v[2] = fmaf(u.z, fs, v[2]);
      v[3] = fmaf(u.w, fs, v[3]);
    }
    if (d >= V) continue;
    if (gate && gate_entry) {
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] *= sigmoid_gate(__bfloat162float(gate[b * ldg + (long long)h * V + d + e]));
    }
    store_n<4>(o + b * ldo + (long long)h * V + d, v);
  }
}

template <int DK, int DV>
static int launch_head_decode(const HeadDecodeArgs& p, int B, cudaStream_t st) {
  using L = DecodeSmem<DK, DV>;
  const int R = p.H / p.G;
  if (R <= 8) {
    static DeviceOnce once;
    auto kern = head_decode_kernel<DK, DV, 8>;
    if (int e = ensure_dyn_smem(once, kern, L::TOTAL)) return e;
    launch_k(kern, dim3(B, p.G, p.splits), HD_THREADS, L::TOTAL, st, p);
  } else {
    static DeviceOnce once;
    auto kern = head_decode_kernel<DK, DV, 16>;
    if (int e = ensure_dyn_smem(once, kern, L::TOTAL)) return e;
    launch_k(kern, dim3(B, p.G * ((R + 15) / 16), p.splits), HD_THREADS, L::TOTAL, st, p);
  }
  return int(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------
// any sizes, fp32 arithmetic
// ------------------------------------------------------------------------------------------------
template <class T>
struct HeadAnyArgs {
  const T* q;               // [B*S, ldq], H heads of D entries
  long long ldq;
  const T *k, *v;           // prompts: [B*Skv, ldk / ldv], G heads; decoding: pools [slots][ldk / ldv]
  long long ldk, ldv, nslots;
  const int* block_table;   // decoding only
  int max_pages, page;
  const int* positions;     // decoding: position of the one query of each sequence
  const T* gate;            // [B*S, ldg] or null
  long long ldg;
  int gate_entry;
  T* o;
  long long ldo;
  int S, Skv, q_off, pos0, H, G, D, V, QR;
  float scale;
  HeadOpt opt;
};

constexpr int AN_K = 32;    // keys per tile

// QR (4, 8 or 16) query rows per block: positions of one head (prompts), or heads of one kv head of a sequence (decoding)
template <class T, bool PAGED>
__global__ void __launch_bounds__(128) head_any_kernel(const HeadAnyArgs<T> p) {
  tfb::pdl_sync();
  extern __shared__ float am[];
  const int D = p.D, V = p.V, QR = p.QR, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, DP = D + 1, R = p.H / p.G;
  float* sQ = am;                       // [QR][D]
  float* sK = sQ + QR * D;              // [AN_K][D + 1]
  float* sV = sK + AN_K * DP;           // [AN_K][V]
  float* sP = sV + AN_K * V;            // [QR][AN_K]
  float* sO = sP + QR * AN_K;           // [QR][V]
  float* sA = sO + QR * V;              // [QR] rescale of this tile, then row sums
  const int chunks = (R + QR - 1) / QR;
  const int b = PAGED ? blockIdx.y : blockIdx.z;
  const int g = PAGED ? blockIdx.x / chunks : blockIdx.y / R;
  const int h0 = PAGED ? g * R + blockIdx.x % chunks * QR : blockIdx.y, i0 = PAGED ? 0 : blockIdx.x * QR;
  const int n = PAGED ? min(QR, (g + 1) * R - h0) : min(QR, p.S - i0);
  const int hi_first = PAGED ? p.positions[b] : i0 + p.q_off, hi_max = PAGED ? hi_first : min(hi_first + n - 1, p.Skv - 1);
  auto row_of = [&](int r) -> long long { return PAGED ? b : (long long)b * p.S + i0 + r; };
  auto head_of = [&](int r) { return PAGED ? h0 + r : h0; };
  for (int i = tid; i < QR * D; i += 128) {
    const int r = i / D;
    sQ[i] = r < n ? to_f(p.q[row_of(r) * p.ldq + (long long)head_of(r) * D + i % D]) : 0.f;
  }
  for (int i = tid; i < QR * V; i += 128) sO[i] = 0.f;
  float m_run[4], l_run[4], f_row[4];   // this warp's rows: warp, warp + 4, ...
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    m_run[i] = -INFINITY;
    l_run[i] = 0.f;
    f_row[i] = p.scale * query_temp(p.opt, PAGED ? hi_first : p.pos0 + i0 + warp + 4 * i);
  }
  // keys that some row sees, in order: the kept first ones, then from the first row's window on
  const int keep = p.opt.bounded() ? p.opt.keep : 0, lo = p.opt.first_key(hi_first), first = min(keep, lo);
  const int total = first + hi_max + 1 - lo;
  for (int t0 = 0; t0 < total; t0 += AN_K) {
    const int nk = min(AN_K, total - t0);
    __syncthreads();
    for (int j = warp; j < AN_K; j += 4) {
      const int at = t0 + j < first ? t0 + j : t0 + j - first + lo;
      long long row = (long long)b * p.Skv + at;
      if (PAGED && j < nk) {
        long long page = p.block_table[(long long)b * p.max_pages + at / p.page];
        TFB_BOUNDS(page >= 0 && (page + 1) * p.page <= p.nslots, 52, page, p.nslots / p.page);
        if (page < 0 || (page + 1) * p.page > p.nslots) page = 0;
        row = page * p.page + at % p.page;
      }
      for (int d = lane; d < D; d += 32) sK[j * DP + d] = j < nk ? to_f(p.k[row * p.ldk + (long long)g * D + d]) : 0.f;
      for (int d = lane; d < V; d += 32) sV[j * V + d] = j < nk ? to_f(p.v[row * p.ldv + (long long)g * V + d]) : 0.f;
    }
    __syncthreads();
    const int at = t0 + lane < first ? t0 + lane : t0 + lane - first + lo;     // this lane's key
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = warp + 4 * i;
      if (r >= QR) continue;
      const float* q = sQ + r * D;
      const float* k = sK + lane * DP;
      float s = 0.f;
      for (int d = 0; d < D; ++d) s = fmaf(q[d], k[d], s);
      s *= f_row[i];
      if (p.opt.cap > 0.f) s = p.opt.cap * tanhf(s / p.opt.cap);
      const int hi = PAGED ? hi_first : i0 + r + p.q_off;
      if (!(r < n && lane < nk && at <= hi && (at >= p.opt.first_key(hi) || at < keep))) s = -INFINITY;
      const float mx = fmaxf(m_run[i], warp_max(s));
      const float mb = mx == -INFINITY ? 0.f : mx;
      const float a = m_run[i] == -INFINITY ? 0.f : expf(m_run[i] - mb);
      const float e = expf(s - mb);
      l_run[i] = fmaf(l_run[i], a, warp_add(e));
      m_run[i] = mx;
      sP[r * AN_K + lane] = e;
      if (lane == 0) sA[r] = a;
    }
    __syncthreads();
    for (int i = tid; i < QR * V; i += 128) {
      const int r = i / V, d = i % V;
      float acc = sO[i] * sA[r];
#pragma unroll 8
      for (int j = 0; j < AN_K; ++j) acc = fmaf(sP[r * AN_K + j], sV[j * V + d], acc);
      sO[i] = acc;
    }
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = warp + 4 * i;
    if (lane != 0 || r >= QR) continue;
    float f = 1.f / l_run[i];
    if (p.opt.sink && r < n) {
      const float sk = sink_score<T>(p.opt, head_of(r)), M = fmaxf(m_run[i], sk), fm = expf(m_run[i] - M);
      f = fm / fmaf(l_run[i], fm, expf(sk - M));
    }
    sA[r] = f;
  }
  __syncthreads();
  for (int r = warp; r < n; r += 4) {
    const long long row = row_of(r);
    const int h = head_of(r);
    float f = sA[r];
    if (p.gate && !p.gate_entry) f *= sigmoid_exact(to_f(p.gate[row * p.ldg + h]));
    for (int d = lane; d < V; d += 32) {
      float v = sO[r * V + d] * f;
      if (p.gate && p.gate_entry) v *= sigmoid_exact(to_f(p.gate[row * p.ldg + (long long)h * V + d]));
      p.o[row * p.ldo + (long long)h * V + d] = from_f<T>(v);
    }
  }
}

template <class T, bool PAGED>
static int launch_any(HeadAnyArgs<T> p, int B, cudaStream_t st) {
  long long smem = 0;
  for (p.QR = 16; p.QR >= 4; p.QR >>= 1) {
    smem = 4ll * (p.QR * p.D + AN_K * (p.D + 1) + AN_K * p.V + p.QR * AN_K + p.QR * p.V + p.QR);
    if (smem <= 220 * 1024) break;
  }
  if (p.QR < 4) return TFB_ERR_LIMIT;
  static DeviceOnce once;
  auto kern = head_any_kernel<T, PAGED>;
  if (int e = ensure_dyn_smem(once, kern, 220 * 1024)) return e;
  const int R = p.H / p.G;
  const dim3 grid = PAGED ? dim3(p.G * ((R + p.QR - 1) / p.QR), B) : dim3((p.S + p.QR - 1) / p.QR, p.H, B);
  launch_k(kern, grid, 128, size_t(smem), st, p);
  return int(cudaGetLastError());
}

static bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
static bool bad_opt(const HeadOpt& o) {
  return o.window < 0 || o.chunk < 0 || (o.window && o.chunk) || o.keep < 0 || !(o.cap >= 0.f) || o.temp_every < 1 || o.sink < 0 || o.sink > 2 ||
         (o.sink == 2 && !o.sinks);
}

}  // namespace tfb

using bf16 = __nv_bfloat16;

// q [B*S, ldq]: H heads of D entries; k, v [B*Skv, ldk / ldv]: G heads of D / V entries; gate [B*S, ldg]: one logit per head, or per entry
// of the heads (gate_entry), or null.  The queries are the last S of the Skv keys; query i stands at position pos0 + i.  With a window or
// chunks, keys between the kept first ones and the first query's window, or the start of its chunk, may be left out of k and v (with chunks
// and no kept ones, the first key then stands at a multiple of the chunk).  sink, sinks: see HeadOpt.  o [B*S, ldo]: H heads of V entries.
TFB_API int tfb_head_attn(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, void* o, long long ldo,
                          const void* gate, long long ldg, int gate_entry, int B, int S, int Skv, int H, int G, int D, int V, float scale, int window,
                          int chunk, int keep, float cap, int sink, const void* sinks, float temp_coef, int temp_every, int pos0, int f32, int* status,
                          void* stream) {
  using namespace tfb;
  const HeadOpt opt{window, chunk, keep, cap, sink, sinks, temp_coef, temp_every};
  if (B <= 0 || B > 65535 || S <= 0 || Skv < S || G <= 0 || H % G || H > 65535 || D <= 0 || V <= 0 || pos0 < 0 || bad_opt(opt)) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  // the running maximum is taken of the scores before the factors: those have to be positive
  const bool tc = !f32 && D % 8 == 0 && V % 8 == 0 && D <= 128 && V <= 128 && ldq % 8 == 0 && ldk % 8 == 0 && ldv % 8 == 0 && ldo % 8 == 0 &&
                  al16(q) && al16(k) && al16(v) && al16(o) && scale > 0.f && temp_coef >= 0.f && (!gate || !gate_entry || (ldg % 8 == 0 && al16(gate)));
  if (tc) {
    HeadAttnParams p{B, S, H, G, Skv, Skv - S, D, V, scale, opt, pos0, static_cast<const bf16*>(gate), ldg, gate ? gate_entry : 0,
                     static_cast<bf16*>(o), ldo, status};
    const int mode = cap > 0.f ? 2 : (opt.bounded() || sink || temp_coef != 0.f || p.gate_entry) ? 1 : 0;
#define TFB_HA(DK, DV)                                                                                                            \
  return mode == 0 ? launch_head_attn<DK, DV, 0>(q, ldq, k, ldk, v, ldv, p, st)                                                   \
                   : mode == 1 ? launch_head_attn<DK, DV, 1>(q, ldq, k, ldk, v, ldv, p, st) : launch_head_attn<DK, DV, 2>(q, ldq, k, ldk, v, ldv, p, st)
    if (D <= 64) {
      if (V <= 64) TFB_HA(64, 64);
      TFB_HA(64, 128);
    }
    if (V <= 64) TFB_HA(128, 64);
    TFB_HA(128, 128);
#undef TFB_HA
  }
#define TFB_ANY(T)                                                                                                                            \
  launch_any<T, false>(HeadAnyArgs<T>{static_cast<const T*>(q), ldq, static_cast<const T*>(k), static_cast<const T*>(v), ldk, ldv, 0, nullptr, 0, 1, \
                                      nullptr, static_cast<const T*>(gate), ldg, gate_entry, static_cast<T*>(o), ldo, S, Skv, Skv - S, pos0, H, G, D, \
                                      V, 16, scale, opt}, B, st)
  return f32 ? TFB_ANY(float) : TFB_ANY(bf16);
#undef TFB_ANY
}

// Key splits of the tensor-core form of tfb_head_decode for up to max_keys keys per query (it then needs acc and ml); 0: the other form.
// The blocks of a step run in rounds of as many as fit on the device at once: the split with the fewest keys times rounds, and
// something for every split's own start and merge.
TFB_API int tfb_head_decode_plan(int B, int H, int G, int D, int V, int max_keys, int f32) {
  if (f32 || B <= 0 || G <= 0 || H % G || D % 8 || V % 8 || D <= 0 || V <= 0 || D > 128 || V > 128) return 0;
  const int R = H / G;
  const long long items = (long long)B * G * (R <= 8 ? 1 : (R + 15) / 16), slots = (long long)tfb::sm_count() * (D <= 64 && V <= 64 ? 5 : 3);
  int best = 1;
  double cost = 1e30;
  for (int s = 1; s <= 32 && (s == 1 || max_keys / s >= 128); ++s) {
    const double c = double((items * s + slots - 1) / slots) * (double(max_keys) / s + 96);
    if (c < cost) {
      cost = c;
      best = s;
    }
  }
  return best;
}

// One query per sequence at positions[b] over the cached rows (k [nslots][G D], v [nslots][G V]); q [B, ldq], o [B, ldo].
TFB_API int tfb_head_decode(const void* q, long long ldq, const void* k, const void* v, long long nslots, const int* block_table, int max_pages,
                            int page, const int* positions, void* o, long long ldo, const void* gate, long long ldg, int gate_entry, float* acc,
                            float* ml, int splits, int B, int H, int G, int D, int V, float scale, int window, int chunk, int keep, float cap, int sink,
                            const void* sinks, float temp_coef, int temp_every, int f32, int* status, void* stream) {
  using namespace tfb;
  const HeadOpt opt{window, chunk, keep, cap, sink, sinks, temp_coef, temp_every};
  if (B <= 0 || B > 65535 || G <= 0 || H % G || D <= 0 || V <= 0 || page <= 0 || nslots < page || bad_opt(opt)) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (acc && tfb_head_decode_plan(B, H, G, D, V, 1, f32) > 0) {
    if (!ml || splits < 1 || splits > 32 || ldq % 8 || ldo % 4 || !al16(q) || !al16(k) || !al16(v) || !al16(o)) return TFB_ERR_ARG;
    HeadDecodeArgs p{static_cast<const bf16*>(q), ldq, static_cast<const bf16*>(k), static_cast<const bf16*>(v), nslots, block_table, max_pages, page,
                     positions, H, G, D, V, splits, scale, opt, acc, ml, status};
    const int rc = D <= 64 ? (V <= 64 ? launch_head_decode<64, 64>(p, B, st) : launch_head_decode<64, 128>(p, B, st))
                           : (V <= 64 ? launch_head_decode<128, 64>(p, B, st) : launch_head_decode<128, 128>(p, B, st));
    if (rc) return rc;
    launch_k(head_combine_kernel, (B * H + 3) / 4, 128, 0, st, acc, ml, static_cast<const bf16*>(gate), ldg, gate_entry, static_cast<bf16*>(o), ldo,
             B * H, H, V, splits, opt);
    return int(cudaGetLastError());
  }
#define TFB_ANY(T)                                                                                                                              \
  launch_any<T, true>(HeadAnyArgs<T>{static_cast<const T*>(q), ldq, static_cast<const T*>(k), static_cast<const T*>(v), (long long)G * D,       \
                                     (long long)G * V, nslots, block_table, max_pages, page, positions, static_cast<const T*>(gate), ldg, gate_entry, \
                                     static_cast<T*>(o), ldo, 1, 0, 0, 0, H, G, D, V, 16, scale, opt}, B, st)
  return f32 ? TFB_ANY(float) : TFB_ANY(bf16);
#undef TFB_ANY
}
