// Latent attention: per token one latent c of R entries is cached, from which every head h reads its key W_uk,h c and its value
// W_uv,h c; causal softmax without positions, one output gate per head.
//
//   latent_append      norm of the latents and their append to the pages
//   prompts            attend over keys and values that a product has read out of the latents: head_attention.cu
//   head_linear        one small product per head for the rows of a decode step (mma.sync): queries into the latent space,
//                      q . W_uk c = (W_uk^T q) . c; the values come out of the attention's result, sum_j a_j W_uv c_j =
//                      W_uv sum_j a_j c_j, by the per-head form of skinny_linear.cu
//   latent_decode      one query per sequence over the paged latents, bf16, mma.sync: the query heads are the rows of one or two 16-row
//                      tiles, and the latents are keys and values of all of them, so a cached row is read once.  Split over
//                      the keys; a second kernel merges the splits.
//   latent_any         decoding, any sizes, bf16 or fp32: fp32 FMA throughout, online softmax over 32-key tiles.
#include "tfb_elem.cuh"
#include "tfb_host.h"
#include "tfb_mma.cuh"

namespace tfb {
TFB_BOUNDS_DEFINE(latent_attention)

constexpr float LOG2E = 1.4426950408889634f;

// ------------------------------------------------------------------------------------------------
// v = c / rms(c) * w, to out and to the pools' slots; one warp per row
// ------------------------------------------------------------------------------------------------
template <class T, int VEC>
__global__ void __launch_bounds__(256) latent_append_kernel(const T* __restrict__ c, long long ldc, const T* __restrict__ w, float eps,
                                                            const long long* __restrict__ slots, T* __restrict__ out, long long ldo,
                                                            T* __restrict__ pool, long long nslots, int width, int rows, int R) {
  tfb::pdl_sync();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  const T* src = c + r * ldc;
  float ss = 0.f;
  for (int i = lane * VEC; i < R; i += 32 * VEC) {
    float v[VEC];
    load_n<VEC>(src + i, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(v[e], v[e], ss);
  }
  const float f = 1.f / sqrtf(warp_add(ss) / R + eps);
  long long slot = slots ? slots[r] : -1;
  TFB_BOUNDS(slot < nslots, 51, slot, nslots);
  if (slot >= nslots) slot = -1;
  for (int i = lane * VEC; i < R; i += 32 * VEC) {
    float v[VEC], g[VEC];
    load_n<VEC>(src + i, v);
    load_n<VEC>(w + i, g);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = v[e] * f * g[e];
    if (out) store_n<VEC>(out + r * ldo + i, v);
    if (slot >= 0) store_n<VEC>(pool + slot * width + i, v);
  }
}

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float redux_max(float x) {      // over the warp, one instruction
  float y;
  asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(y) : "f"(x));
  return y;
}

// ------------------------------------------------------------------------------------------------
// one product per head for few rows, weights stored [K, N]: out[m, h * out_head + n] = sum_k x[m, h * x_head + k] W_h[k, n].
// 64 rows x 32 columns per block, the next 128-deep chunk in registers while one is used.
// ------------------------------------------------------------------------------------------------
struct HeadLinearArgs {
  const __nv_bfloat16 *x, *w;
  long long ldx, ldw;
  __nv_bfloat16* out;
  long long ldo;
  int M, N, K, x_head, out_head;     // columns N .. out_head of a head are written as zeros
  int vec_x, vec_w;                  // 16-byte loads are aligned
};

constexpr int HL_M = 64, HL_N = 32, HL_K = 128;

__device__ __forceinline__ uint4 load8(const __nv_bfloat16* p, int n, int vec) {   // n of 8 entries, the others zero
  if (n <= 0) return make_uint4(0u, 0u, 0u, 0u);
  if (vec && n >= 8) return *reinterpret_cast<const uint4*>(p);
  uint32_t u[4] = {0u, 0u, 0u, 0u};
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (i < n) u[i >> 1] |= uint32_t(__bfloat16_as_ushort(p[i])) << ((i & 1) * 16);
  return make_uint4(u[0], u[1], u[2], u[3]);
}

__global__ void __launch_bounds__(128) head_linear_kernel(const HeadLinearArgs p) {
  tfb::pdl_sync();
  constexpr int PA = HL_K * 2 + 16, PB = HL_N * 2 + 16;                              // byte pitches
  constexpr int CA = HL_K / 8, CB = HL_N / 8;                                        // 16-byte pieces of a row
  constexpr int NA = HL_M * CA / 128, NB = HL_K * CB / 128;
  __shared__ __align__(16) uint8_t sA[HL_M * PA];
  __shared__ __align__(16) uint8_t sB[HL_K * PB];
  const int n0 = blockIdx.x * HL_N, h = blockIdx.y, m0 = blockIdx.z * HL_M;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const __nv_bfloat16* x = p.x + (long long)h * p.x_head;
  const __nv_bfloat16* w = p.w + (long long)h * p.K * p.ldw;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  uint4 ra[NA], rb[NB];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      const int e = tid + i * 128, r = e / CB, c = (e % CB) * 8;
      rb[i] = k0 + r < p.K ? load8(w + (k0 + r) * p.ldw + n0 + c, p.N - n0 - c, p.vec_w) : zero;
    }
#pragma unroll
    for (int i = 0; i < NA; ++i) {
      const int e = tid + i * 128, r = e / CA, c = (e % CA) * 8;
      ra[i] = m0 + r < p.M ? load8(x + (m0 + r) * p.ldx + k0 + c, p.K - k0 - c, p.vec_x) : zero;
    }
  };
  float acc[4][4];
#pragma unroll
  for (int n = 0; n < 4; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
  fetch(0);
  for (int k0 = 0; k0 < p.K; k0 += HL_K) {
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NA; ++i) {
      const int e = tid + i * 128;
      *reinterpret_cast<uint4*>(sA + (e / CA) * PA + (e % CA) * 16) = ra[i];
    }
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      const int e = tid + i * 128;
      *reinterpret_cast<uint4*>(sB + (e / CB) * PB + (e % CB) * 16) = rb[i];
    }
    __syncthreads();
    if (k0 + HL_K < p.K) fetch(k0 + HL_K);
    if (m0 + warp * 16 >= p.M) continue;
    const uint32_t a0 = smem_u32(sA) + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PA + (lane >> 4) * 16;
    const uint32_t b0 = smem_u32(sB) + ((lane & 7) + ((lane >> 3) & 1) * 8) * PB + (lane >> 4) * 16;
#pragma unroll
    for (int ks = 0; ks < HL_K / 16; ++ks) {
      if (k0 + ks * 16 >= p.K) break;
      uint32_t a[4];
      ldsm(a0 + ks * 32, a);
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) {
        uint32_t b[4];
        ldsm_t(b0 + ks * 16 * PB + nb * 32, b);
        mma_bf16(acc[2 * nb], a, b[0], b[1]);
        mma_bf16(acc[2 * nb + 1], a, b[2], b[3]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int m = m0 + warp * 16 + (lane >> 2) + 8 * i;
    if (m >= p.M) continue;
    __nv_bfloat16* o = p.out + m * p.ldo + (long long)h * p.out_head;
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = n0 + n * 8 + (lane & 3) * 2 + e;
        if (col < p.out_head) o[col] = __float2bfloat16(acc[n][2 * i + e]);
      }
  }
}

// ------------------------------------------------------------------------------------------------
// decoding over the paged latents on mma.sync
// ------------------------------------------------------------------------------------------------
struct LatentDecodeArgs {
  const __nv_bfloat16* q;     // [B, ldq]: H heads of W entries
  long long ldq;
  const __nv_bfloat16* pool;  // [slots][W]
  long long nslots;
  const int* block_table;
  int max_pages, page;
  const int* positions;       // [B] position of the query (it sees itself: its row is in the cache)
  int H, W, splits;
  float scale;
  __nv_bfloat16* o;           // [B, ldo] (one split)
  long long ldo;
  float *acc, *ml;            // [B, H, splits, W], [B, H, splits, 2] (several)
  int* status;
};

constexpr int LD_THREADS = 256;
constexpr int LD_KEYS = 64, LD_HALF = 32;      // keys of a step; keys of a ring slot

// RC: columns of a latent in shared memory (zeros past W); MT: 16-row tiles of query heads.  Of the eight warps, two share the keys
// and four the columns in the scores (the partial scores meet in shared memory); each takes an eighth of the columns in the
// product with the weights.
template <int RC, int MT>
struct LatentSmem {
  static constexpr int RP = RC * 2 + 16;                 // byte pitch of a row: ldmatrix reads eight rows without bank conflicts
  static constexpr int SLOT = LD_HALF * RP;
  static constexpr int SP = LD_KEYS + 8;                 // floats of a score row
  static constexpr int PP = LD_KEYS * 2 + 16;            // bytes of a weight row
  static constexpr int S_BYTES = 4 * MT * 16 * SP * 4, P_BYTES = MT * 16 * PP, A_BYTES = MT * 16 * 8;
  static constexpr int REST = S_BYTES + P_BYTES + A_BYTES + 128;
  static constexpr int FIT = (226 * 1024 - REST) / SLOT;
  static constexpr int NS = FIT > 8 ? 8 : FIT;           // ring slots
  static constexpr int S_OFF = NS * SLOT, P_OFF = S_OFF + S_BYTES, A_OFF = P_OFF + P_BYTES, BAR_OFF = A_OFF + A_BYTES;
  static constexpr int TOTAL = BAR_OFF + 128;
  static_assert(NS >= 4, "two steps at least");
};

template <int RC, int MT>
__global__ void __launch_bounds__(LD_THREADS, 1) latent_decode_kernel(const LatentDecodeArgs p) {
  using L = LatentSmem<RC, MT>;
  constexpr int NS = L::NS, RP = L::RP, KS = RC / 64, NT = RC / 64;   // k steps of a warp's column quarter; 8-column blocks of its eighth
  extern __shared__ __align__(128) uint8_t sm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int b = blockIdx.x, h0 = blockIdx.y * MT * 16, sp = blockIdx.z;
  const int kg = warp & 1, rg = warp >> 1;
  const uint32_t s0 = smem_u32(sm), bars = s0 + L::BAR_OFF;
  float* sS = reinterpret_cast<float*>(sm + L::S_OFF);
  float* sAl = reinterpret_cast<float*>(sm + L::A_OFF);                // rescale of a row; at the end: its maximum, then its sum
  volatile int* abort_flag = reinterpret_cast<volatile int*>(sm + L::BAR_OFF + 64);
  if (tid == 0) {
    for (int s = 0; s < NS; ++s) mbar_init(bars + s * 8, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  tfb::pdl_sync();
  uint32_t qa[MT][KS][4];                                              // this warp's columns of the queries
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = h0 + m * 16 + (lane >> 2) + (e & 1) * 8, c = rg * (RC / 4) + k * 16 + (lane & 3) * 2 + (e >> 1) * 8;
        qa[m][k][e] = (h < p.H && c < p.W) ? *reinterpret_cast<const uint32_t*>(p.q + b * p.ldq + (long long)h * p.W + c) : 0u;
      }
  const int n_keys = p.positions[b] + 1;
  const int per = ((n_keys + p.splits - 1) / p.splits + LD_KEYS - 1) / LD_KEYS * LD_KEYS;
  const int t_begin = sp * per, count = max(0, min(n_keys, t_begin + per) - t_begin);
  const int nt = (count + LD_KEYS - 1) / LD_KEYS, nh = (count + LD_HALF - 1) / LD_HALF;
  // what no copy writes but the products read: columns past W, and rows past the end in a slot that no earlier rows have filled
  if (p.W < RC) {
    const int pieces = (RC - p.W) / 8;
    for (int i = tid; i < NS * LD_HALF * pieces; i += LD_THREADS)
      *reinterpret_cast<uint4*>(sm + (i / pieces) * RP + p.W * 2 + (i % pieces) * 16) = make_uint4(0u, 0u, 0u, 0u);
  }
  {
    const int from = min(count, NS * LD_HALF), to = min(nt * LD_KEYS, NS * LD_HALF);
    for (int i = tid; i < (to - from) * (RP / 16); i += LD_THREADS) reinterpret_cast<uint4*>(sm + from * RP)[i] = make_uint4(0u, 0u, 0u, 0u);
  }
  fence_proxy_async_smem();
  __syncthreads();

  // lanes 0-7 of warp w bring rows 4 w .. 4 w + 3 of two halves; pages divide a half (checked by the caller), so a row's place in its
  // page never changes
  const int my_row = warp * 4 + (lane & 3), my_half = lane >> 2, in_page = my_row % p.page;
  const int* bt = p.block_table + (long long)b * p.max_pages + (t_begin + my_row) / p.page;
  const int pages_half = LD_HALF / p.page;
  auto page_of = [&](int h) { return (lane < 8 && h < nh && h * LD_HALF + my_row < count) ? bt[h * pages_half] : 0; };
  auto issue = [&](int h, long long page) {                            // h: this lane's half
    if (lane >= 8 || h >= nh) return;
    const int rows = min(LD_HALF, count - h * LD_HALF), slot = h % NS;
    if (warp == 0 && (lane & 3) == 0) mbar_expect_tx(bars + slot * 8, uint32_t(rows) * p.W * 2);
    if (my_row < rows) {
      TFB_BOUNDS(page >= 0 && (page + 1) * p.page <= p.nslots, 52, page, p.nslots / p.page);
      if (page < 0 || (page + 1) * p.page > p.nslots) page = 0;
      bulk_load(s0 + slot * L::SLOT + my_row * RP, p.pool + (page * p.page + in_page) * p.W, p.W * 2, bars + slot * 8);
    }
  };
#pragma unroll
  for (int h = 0; h < NS; h += 2)
    if (h + my_half < NS) issue(h + my_half, page_of(h + my_half));
  int page_next = page_of(NS + my_half);

  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;
  float m_run[2 * MT], l_run[2 * MT];                                  // rows 2 MT warp + i; the sum: this lane's part
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }
  const float sl2 = p.scale * LOG2E;
  bool ok = true;

  // step j: values of tile j - 1 and scores of tile j back to back (no barrier between them), then the softmax of tile j
  for (int j = 0; j <= nt && nt > 0; ++j) {
    if (j > 0) {
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float a0 = sAl[m * 16 + (lane >> 2)], a1 = sAl[m * 16 + (lane >> 2) + 8];
        if (__all_sync(0xffffffffu, a0 == 1.f && a1 == 1.f)) continue;       // no maximum of these rows has moved
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          o[m][n][0] *= a0;
          o[m][n][1] *= a0;
          o[m][n][2] *= a1;
          o[m][n][3] *= a1;
        }
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const uint32_t slot = s0 + ((2 * (j - 1) + half) % NS) * L::SLOT;
        uint32_t pa[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int k = 0; k < 2; ++k)
            ldsm(s0 + L::P_OFF + (m * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * L::PP + half * 64 + k * 32 + (lane >> 4) * 16, pa[m][k]);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          uint32_t f[4];
          ldsm_t(slot + lane * RP + (warp * (RC / 8) + n * 8) * 2, f);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(o[m][n], pa[m][0], f[0], f[1]);
            mma_bf16(o[m][n], pa[m][1], f[2], f[3]);
          }
        }
      }
    }
    if (j < nt) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int h = 2 * j + half;
        if (ok && h < nh && !mbar_wait_warp(bars + (h % NS) * 8, (h / NS) & 1, abort_flag, p.status, ST_TIMEOUT_FULL)) ok = false;
      }
      // scores of 32 keys over a quarter of the columns
      float sc[MT][4][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n) sc[m][n][0] = sc[m][n][1] = sc[m][n][2] = sc[m][n][3] = 0.f;
      const uint32_t krow = s0 + ((2 * j + kg) % NS) * L::SLOT + ((lane & 7) + (lane >> 4) * 8) * RP + rg * (RC / 2) + ((lane >> 3) & 1) * 16;
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t f0[4], f1[4];
        ldsm(krow + k * 32, f0);
        ldsm(krow + 16 * RP + k * 32, f1);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16(sc[m][0], qa[m][k], f0[0], f0[1]);
          mma_bf16(sc[m][1], qa[m][k], f0[2], f0[3]);
          mma_bf16(sc[m][2], qa[m][k], f1[0], f1[1]);
          mma_bf16(sc[m][3], qa[m][k], f1[2], f1[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int i = 0; i < 2; ++i)
            *reinterpret_cast<float2*>(sS + (rg * MT * 16 + m * 16 + (lane >> 2) + 8 * i) * L::SP + kg * 32 + n * 8 + (lane & 3) * 2) =
                make_float2(sc[m][n][2 * i], sc[m][n][2 * i + 1]);
    }
    __syncthreads();
    if (j == nt) break;
    // every warp is done with tile j - 1: its slots take the next two halves
    if (j > 0) {
      const int h = NS + 2 * (j - 1) + my_half;
      if (ok) {
        fence_proxy_async_smem();
        issue(h, page_next);
      }
      page_next = page_of(h + 2);
    }
    const int n_valid = count - j * LD_KEYS;
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
      const int row = warp * 2 * MT + i;
      float2 s = *reinterpret_cast<const float2*>(sS + row * L::SP + 2 * lane);
#pragma unroll
      for (int g = 1; g < 4; ++g) {
        const float2 u = *reinterpret_cast<const float2*>(sS + (g * MT * 16 + row) * L::SP + 2 * lane);
        s.x += u.x;
        s.y += u.y;
      }
      s.x = 2 * lane < n_valid ? s.x * sl2 : -INFINITY;
      s.y = 2 * lane + 1 < n_valid ? s.y * sl2 : -INFINITY;
      const float mx = fmaxf(m_run[i], redux_max(fmaxf(s.x, s.y)));     // finite: a tile has a key
      const float alpha = ex2(m_run[i] - mx);
      const float p0 = ex2(s.x - mx), p1 = ex2(s.y - mx);
      m_run[i] = mx;
      l_run[i] = fmaf(l_run[i], alpha, p0 + p1);
      *reinterpret_cast<uint32_t*>(sm + L::P_OFF + row * L::PP + lane * 4) = pack_bf16(p0, p1);
      if (lane == 0) sAl[row] = alpha;
    }
    __syncthreads();
  }
  if (!ok) {   // give copies already issued a bounded time to land before shared memory goes away
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) {}
  }
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) l_run[i] = warp_add(l_run[i]);
  __syncthreads();
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
      sAl[warp * 2 * MT + i] = m_run[i];
      sAl[MT * 16 + warp * 2 * MT + i] = l_run[i];
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = m * 16 + (lane >> 2) + 8 * i, h = h0 + row;
      if (h >= p.H) continue;
      if (p.splits == 1) {
        const float inv = 1.f / sAl[MT * 16 + row];
        __nv_bfloat16* dst = p.o + b * p.ldo + (long long)h * p.W;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const int c = warp * (RC / 8) + n * 8 + (lane & 3) * 2;
          if (c < p.W) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(o[m][n][2 * i] * inv, o[m][n][2 * i + 1] * inv);
        }
      } else {
        const long long at = ((long long)b * p.H + h) * p.splits + sp;
        if (nt > 0) {
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            const int c = warp * (RC / 8) + n * 8 + (lane & 3) * 2;
            if (c < p.W) *reinterpret_cast<float2*>(p.acc + at * p.W + c) = make_float2(o[m][n][2 * i], o[m][n][2 * i + 1]);
          }
        }
        if (warp == 0 && (lane & 3) == 0) {
          p.ml[at * 2] = sAl[row];
          p.ml[at * 2 + 1] = sAl[MT * 16 + row];
        }
      }
    }
}

// one block per (sequence, head): merge the splits
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ acc, const float* __restrict__ ml, __nv_bfloat16* __restrict__ o,
                                                             long long ldo, int H, int W, int splits) {
  tfb::pdl_sync();
  __shared__ float f[128];
  const int b = blockIdx.x / H, h = blockIdx.x % H;
  const long long base = (long long)blockIdx.x * splits;
  if (threadIdx.x < 32) {                   // splits <= 128
    float m = -INFINITY;
    for (int s = threadIdx.x; s < splits; s += 32) m = fmaxf(m, ml[(base + s) * 2]);
    m = warp_max(m);
    float l = 0.f;
    for (int s = threadIdx.x; s < splits; s += 32) {
      const float ms = ml[(base + s) * 2], e = ms == -INFINITY ? 0.f : exp2f(ms - m);
      f[s] = e;
      l = fmaf(ml[(base + s) * 2 + 1], e, l);
    }
    l = warp_add(l);
    for (int s = threadIdx.x; s < splits; s += 32) f[s] /= l;
  }
  __syncthreads();
  for (int c = threadIdx.x * 4; c < W; c += 512) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
      if (f[s] == 0.f) continue;
      const float4 u = *reinterpret_cast<const float4*>(acc + (base + s) * W + c);
      v.x = fmaf(u.x, f[s], v.x);
      v.y = fmaf(u.y, f[s], v.y);
      v.z = fmaf(u.z, f[s], v.z);
      v.w = fmaf(u.w, f[s], v.w);
    }
    uint2 r;
    r.x = pack_bf16(v.x, v.y);
    r.y = pack_bf16(v.z, v.w);
    *reinterpret_cast<uint2*>(o + b * ldo + (long long)h * W + c) = r;
  }
}

template <int RC, int MT>
static int launch_latent_decode(const LatentDecodeArgs& p, int B, cudaStream_t st) {
  using L = LatentSmem<RC, MT>;
  static DeviceOnce once;
  auto kern = latent_decode_kernel<RC, MT>;
  if (int e = ensure_dyn_smem(once, kern, L::TOTAL)) return e;
  launch_k(kern, dim3(B, (p.H + MT * 16 - 1) / (MT * 16), p.splits), LD_THREADS, L::TOTAL, st, p);
  return int(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------
// any sizes, fp32 arithmetic
// ------------------------------------------------------------------------------------------------
template <class T>
struct LatentAnyArgs {
  const T* q;               // [B, ldq], H heads of W entries, R of them used
  long long ldq;
  const T* pool;            // [slots][W]: keys and values of every head
  long long nslots;
  const int* block_table;
  int max_pages, page;
  const int* positions;     // [B] position of the one query of each sequence
  T* o;
  long long ldo;
  int H, R, W, QR;
  float scale;
};

constexpr int AN_K = 32;    // keys per tile

// QR (4, 8 or 16) heads of one sequence per block
template <class T>
__global__ void __launch_bounds__(128) latent_any_kernel(const LatentAnyArgs<T> p) {
  tfb::pdl_sync();
  extern __shared__ float am[];
  const int D = p.R, QR = p.QR, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, DP = D + 1;
  float* sQ = am;                       // [QR][D]
  float* sK = sQ + QR * D;              // [AN_K][D + 1]
  float* sP = sK + AN_K * DP;           // [QR][AN_K]
  float* sO = sP + QR * AN_K;           // [QR][D]
  float* sA = sO + QR * D;              // [QR] rescale of this tile, then row sums
  const int b = blockIdx.y, h0 = blockIdx.x * QR, n = min(QR, p.H - h0), hi = p.positions[b];
  for (int i = tid; i < QR * D; i += 128) {
    const int r = i / D;
    sQ[i] = r < n ? to_f(p.q[b * p.ldq + (long long)(h0 + r) * p.W + i % D]) : 0.f;
    sO[i] = 0.f;
  }
  float m_run[4], l_run[4];             // this warp's rows: warp, warp + 4, ...
#pragma unroll
  for (int i = 0; i < 4; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }
  for (int t0 = 0; t0 <= hi; t0 += AN_K) {
    const int nk = min(AN_K, hi + 1 - t0);
    __syncthreads();
    for (int j = warp; j < AN_K; j += 4) {
      long long row = 0;
      if (j < nk) {
        long long page = p.block_table[(long long)b * p.max_pages + (t0 + j) / p.page];
        TFB_BOUNDS(page >= 0 && (page + 1) * p.page <= p.nslots, 52, page, p.nslots / p.page);
        if (page < 0 || (page + 1) * p.page > p.nslots) page = 0;
        row = page * p.page + (t0 + j) % p.page;
      }
      for (int d = lane; d < D; d += 32) sK[j * DP + d] = j < nk ? to_f(p.pool[row * p.W + d]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = warp + 4 * i;
      if (r >= QR) continue;
      const float* q = sQ + r * D;
      const float* k = sK + lane * DP;
      float s = 0.f;
      for (int d = 0; d < D; ++d) s = fmaf(q[d], k[d], s);
      s = (r < n && lane < nk) ? s * p.scale : -INFINITY;
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
    for (int i = tid; i < QR * D; i += 128) {
      const int r = i / D, d = i % D;
      float acc = sO[i] * sA[r];
#pragma unroll 8
      for (int j = 0; j < AN_K; ++j) acc = fmaf(sP[r * AN_K + j], sK[j * DP + d], acc);
      sO[i] = acc;
    }
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 4; ++i)
    if (lane == 0 && warp + 4 * i < QR) sA[warp + 4 * i] = l_run[i];
  __syncthreads();
  for (int r = warp; r < n; r += 4) {
    const float f = 1.f / sA[r];
    for (int d = lane; d < p.W; d += 32) p.o[b * p.ldo + (long long)(h0 + r) * p.W + d] = from_f<T>(d < D ? sO[r * D + d] * f : 0.f);
  }
}

template <class T>
static int launch_latent_any(LatentAnyArgs<T> p, int B, cudaStream_t st) {
  long long smem = 0;
  for (p.QR = 16; p.QR >= 4; p.QR >>= 1) {
    smem = 4ll * (2 * p.QR * p.R + AN_K * (p.R + 1) + p.QR * AN_K + p.QR);
    if (smem <= 220 * 1024) break;
  }
  if (p.QR < 4) return TFB_ERR_LIMIT;
  static DeviceOnce once;
  auto kern = latent_any_kernel<T>;
  if (int e = ensure_dyn_smem(once, kern, 220 * 1024)) return e;
  launch_k(kern, dim3((p.H + p.QR - 1) / p.QR, B), 128, size_t(smem), st, p);
  return int(cudaGetLastError());
}

static bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace tfb

using bf16 = __nv_bfloat16;

// rows c [rows, ldc] of R entries -> out (may be null) and the pool [nslots][width] at slots (null: none; negative: not this row)
TFB_API int tfb_latent_append(const void* c, long long ldc, const void* w, float eps, const long long* slots, void* out, long long ldo, void* pool,
                              long long nslots, int width, int rows, int R, int f32, void* stream) {
  using namespace tfb;
  if (rows <= 0 || R <= 0 || width < R) return TFB_ERR_ARG;
  if (!slots || nslots == 0) slots = nullptr;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vec = f32 ? 4 : 8, grid = (rows + 7) / 8;
  const bool v = R % vec == 0 && ldc % vec == 0 && ldo % vec == 0 && width % vec == 0 && al16(c) && al16(w) && al16(out) && al16(pool);
#define TFB_LA(T, VEC) launch_k(latent_append_kernel<T, VEC>, grid, 256, 0, st, static_cast<const T*>(c), ldc, static_cast<const T*>(w), eps, slots, \
                                static_cast<T*>(out), ldo, static_cast<T*>(pool), nslots, width, rows, R)
  if (f32) { if (v) TFB_LA(float, 4); else TFB_LA(float, 1); }
  else { if (v) TFB_LA(bf16, 8); else TFB_LA(bf16, 1); }
#undef TFB_LA
  return int(cudaGetLastError());
}

// One product per head: x [M, ldx] (x_head entries between heads, K of them used), w: heads blocks [K, N] stacked on the rows, out [M, ldo]
// (out_head >= N entries between heads; those past N become zero).
TFB_API int tfb_head_linear(const void* x, long long ldx, int x_head, const void* w, long long ldw, void* out, long long ldo, int out_head, int M,
                            int heads, int N, int K, void* stream) {
  using namespace tfb;
  if (M <= 0 || heads <= 0 || heads > 65535 || K <= 0 || N <= 0 || x_head < K || out_head < N) return TFB_ERR_ARG;
  HeadLinearArgs p{static_cast<const bf16*>(x), static_cast<const bf16*>(w), ldx, ldw, static_cast<bf16*>(out), ldo, M, N, K, x_head, out_head,
                   x_head % 8 == 0 && ldx % 8 == 0 && al16(x), ldw % 8 == 0 && al16(w)};
  launch_k(head_linear_kernel, dim3((out_head + HL_N - 1) / HL_N, heads, (M + HL_M - 1) / HL_M), 128, 0, static_cast<cudaStream_t>(stream), p);
  return int(cudaGetLastError());
}

// Key splits of the tensor-core form of tfb_latent_decode for these sizes (it then needs acc / ml for more than one); 0: the other form.
// A wide latent's CTA fills an SM, and all of a step's CTAs should run at once: a second wave of a few would double the time.
TFB_API int tfb_latent_decode_plan(int B, int H, int W, int max_keys, int f32) {
  if (f32 || W > 512 || W % 8) return 0;
  const long long items = (long long)B * ((H + 31) / 32), slots = 148ll * (W > 256 ? 1 : 2);
  long long s = slots / (items > 0 ? items : 1);
  const long long most = (max_keys + 2 * tfb::LD_KEYS - 1) / (2 * tfb::LD_KEYS);     // two tiles each at least
  if (s > most) s = most;
  return int(s < 1 ? 1 : (s > 64 ? 64 : s));
}

// One query per sequence at positions[b] over the cached rows of the pool [slots][W] (latents of R entries, zeros behind them); q and o
// [B, ldq / ldo]: H heads of W entries.
TFB_API int tfb_latent_decode(const void* q, long long ldq, const void* pool, long long nslots, const int* block_table, int max_pages, int page,
                              const int* positions, void* o, long long ldo, float* acc, float* ml, int splits, int B, int H, int R, int W,
                              float scale, int f32, int* status, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || H <= 0 || R <= 0 || W < R || page <= 0 || LD_HALF % page) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (splits > 0 && tfb_latent_decode_plan(B, H, W, 1, f32) > 0) {
    if (splits > 128 || (splits > 1 && (!acc || !ml)) || ldq % 8 || ldo % 8 || !al16(q) || !al16(pool) || !al16(o)) return TFB_ERR_ARG;
    LatentDecodeArgs p{static_cast<const bf16*>(q), ldq, static_cast<const bf16*>(pool), nslots, block_table, max_pages, page, positions, H, W,
                       splits, scale, static_cast<bf16*>(o), ldo, acc, ml, status};
    int rc;
#define TFB_LD(RC) (H <= 16 ? launch_latent_decode<RC, 1>(p, B, st) : launch_latent_decode<RC, 2>(p, B, st))
    if (W <= 64) rc = TFB_LD(64);
    else if (W <= 128) rc = TFB_LD(128);
    else if (W <= 256) rc = TFB_LD(256);
    else rc = TFB_LD(512);
#undef TFB_LD
    if (rc) return rc;
    if (splits > 1) launch_k(latent_combine_kernel, B * H, 128, 0, st, acc, ml, static_cast<bf16*>(o), ldo, H, W, splits);
    return int(cudaGetLastError());
  }
#define TFB_ANY(T)                                                                                                                    \
  launch_latent_any<T>(LatentAnyArgs<T>{static_cast<const T*>(q), ldq, static_cast<const T*>(pool), nslots, block_table, max_pages, page, positions, \
                                        static_cast<T*>(o), ldo, H, R, W, 16, scale}, B, st)
  return f32 ? TFB_ANY(float) : TFB_ANY(bf16);
#undef TFB_ANY
}
