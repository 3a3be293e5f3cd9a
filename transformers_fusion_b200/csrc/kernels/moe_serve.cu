// Mixture-of-experts feed-forward for serving: any sizes and pitches, bf16 or fp32 rows, no statistics and nothing kept for a
// backward pass (the training form is moe_routing.cu).
//
//   moe_route          per token: the k largest of logits (+ bias) (fp32, the lower index first among equals) and the softmax over them,
//                      or the k largest sigmoids among the experts of the best groups, weighted by them over their sum, or the k
//                      largest entries of the softmax over all experts, weighted by themselves;
//                      then the rows of the expert buffers: every expert's assignments are consecutive rows from a multiple
//                      of 128 on, so that a 128-row tile of the grouped product belongs to one expert.  Few tokens (decode
//                      steps): one block does all of it; many: selection with per-block counts, then the scan and row numbers.
//   moe_gather         token rows to their assignments' rows
//   moe_glu            act(gate) * up of the assigned rows (a decode step's buffers are mostly padding)
//   moe_weighted_sum   y[t] = base[t] [* sigmoid(gate[t])] + sum_k w[t, k] * rows[row_of[t, k]], summed in fp32
#include <limits.h>

#include "tfb_elem.cuh"
#include "tfb_host.h"

namespace tfb {
TFB_BOUNDS_DEFINE(moe_serve)

struct RouteArgs {
  const float* logits;        // [T, ld]
  long long ld;
  const void* bias;           // [E], bf16 or fp32, or null
  int bias_f32, T, E, K;
  int* idx;                   // [T, K]
  float* w;                   // [T, K]
  int *rank, *row_of;         // [T, K]
  int* expert_of_tile;        // [tiles]
  int* counts;                // [E]
  int tiles;
  int sigmoid, groups, keep;  // scores are sigmoids, of the experts of `keep` of `groups` groups of E / groups neighbours
  int all;                    // the softmax is over all experts, not over the chosen ones
  float scale;
};

__device__ __forceinline__ float biased_logit(const RouteArgs& p, const float* z, int e) {
  if (p.sigmoid) return 1.f / (1.f + expf(-z[e]));
  if (!p.bias) return z[e];
  return z[e] + (p.bias_f32 ? static_cast<const float*>(p.bias)[e] : to_f(static_cast<const __nv_bfloat16*>(p.bias)[e]));
}
// unsigned numbers in the order of the floats; 0 stands for "taken"
__device__ __forceinline__ uint32_t ordered(float v) {
  const uint32_t u = __float_as_uint(v);
  return u ^ (uint32_t(int32_t(u) >> 31) | 0x80000000u);
}
__device__ __forceinline__ float unordered(uint32_t k) { return __uint_as_float(k & 0x80000000u ? k ^ 0x80000000u : ~k); }

// Chooses the experts of token t (one warp); `count` (shared memory) numbers the assignments of each expert.  note(i, expert, rank)
// is called once per assignment i = t K + k.
// PER > 0: up to 32 PER experts and K <= 32, the logits in registers (lane l: experts l, l + 32, ...).  PER 0: any sizes; K
// rounds, each the largest entry that comes after the last one in the order (value descending, index ascending).
template <int PER, class Note>
__device__ __forceinline__ void choose_experts(const RouteArgs& p, int t, int lane, int* count, Note note) {
  const float* z = p.logits + t * p.ld;
  if constexpr (PER > 0) {
    uint32_t key[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) key[i] = lane + i * 32 < p.E ? ordered(biased_logit(p, z, lane + i * 32)) : 0u;
    if (p.sigmoid && p.keep < p.groups) {      // lane g holds the mark of group g; then the experts of the others are taken out
      const int n = p.E / p.groups;
      uint32_t mark = 0u;
      for (int g = 0; g < p.groups; ++g) {
        uint32_t b1 = 0u, b2 = 0u;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
          const int e = lane + i * 32;
          if (e < p.E && e / n == g) {
            b2 = max(b2, min(b1, key[i]));
            b1 = max(b1, key[i]);
          }
        }
        const uint32_t t1 = __reduce_max_sync(0xffffffffu, b1);
        const uint32_t owner = __ffs(__ballot_sync(0xffffffffu, b1 == t1)) - 1;
        const uint32_t t2 = __reduce_max_sync(0xffffffffu, uint32_t(lane) == owner ? b2 : b1);
        const float s = unordered(t1) + (t2 ? unordered(t2) : 0.f);
        if (lane == g) mark = ordered(s);
      }
      uint32_t kept = 0u;
      for (int k = 0; k < p.keep; ++k) {
        const uint32_t best = __reduce_max_sync(0xffffffffu, mark);
        const uint32_t g = __ffs(__ballot_sync(0xffffffffu, mark == best)) - 1;
        kept |= 1u << g;
        if (uint32_t(lane) == g) mark = 0u;
      }
#pragma unroll
      for (int i = 0; i < PER; ++i)
        if (lane + i * 32 < p.E && !((kept >> ((lane + i * 32) / n)) & 1u)) key[i] = 0u;
    }
    float first = 0.f, sum = 0.f, mine = 0.f, total = 0.f;
    int e_mine = 0;
    if (p.all) {
      uint32_t top = 0u;
#pragma unroll
      for (int i = 0; i < PER; ++i) top = max(top, key[i]);
      first = unordered(__reduce_max_sync(0xffffffffu, top));
#pragma unroll
      for (int i = 0; i < PER; ++i)
        if (key[i]) total += expf(unordered(key[i]) - first);
      total = warp_add(total);
    }
    for (int k = 0; k < p.K; ++k) {
      uint32_t best = key[0];
      int e = lane;
#pragma unroll
      for (int i = 1; i < PER; ++i)
        if (key[i] > best) { best = key[i]; e = lane + i * 32; }
      const uint32_t top = __reduce_max_sync(0xffffffffu, best);
      int chosen = int(__reduce_min_sync(0xffffffffu, best == top ? uint32_t(e) : 0x7fffffffu));
      if (chosen >= p.E) chosen = k;        // logits that compare with nothing
#pragma unroll
      for (int i = 0; i < PER; ++i)
        if (chosen == lane + i * 32) key[i] = 0u;
      const float v = unordered(top);
      if (k == 0) first = v;
      const float x = p.sigmoid ? v : expf(v - first);
      sum += x;
      if (lane == k) { mine = x; e_mine = chosen; }
    }
    if (lane < p.K) {
      const int i = t * p.K + lane;
      p.idx[i] = e_mine;
      p.w[i] = p.sigmoid ? mine / (sum + 1e-20f) * p.scale : mine / (p.all ? total : sum);
      note(i, e_mine, atomicAdd(count + e_mine, 1));
    }
  } else {
    float last = INFINITY, first = 0.f, sum = 0.f, total = 0.f;
    int last_e = -1;
    if (p.all) {
      float top = -INFINITY;
      for (int e = lane; e < p.E; e += 32) top = fmaxf(top, biased_logit(p, z, e));
      top = warp_max(top);
      for (int e = lane; e < p.E; e += 32) total += expf(biased_logit(p, z, e) - top);
      total = warp_add(total);
    }
    for (int k = 0; k < p.K; ++k) {
      float best = -INFINITY;
      int e_best = INT_MAX;
      for (int e = lane; e < p.E; e += 32) {
        const float v = biased_logit(p, z, e);
        const bool after = v < last || (v == last && e > last_e);
        if (after && (v > best || e_best == INT_MAX)) { best = v; e_best = e; }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, best, o);
        const int e = __shfl_xor_sync(0xffffffffu, e_best, o);
        if (e != INT_MAX && (e_best == INT_MAX || v > best || (v == best && e < e_best))) { best = v; e_best = e; }
      }
      if (e_best == INT_MAX) e_best = k;
      last = best;
      last_e = e_best;
      if (k == 0) first = best;
      const float x = p.sigmoid ? best : expf(best - first);
      sum += x;
      if (lane == 0) {
        const int i = t * p.K + k;
        p.idx[i] = e_best;
        p.w[i] = x;
        note(i, e_best, atomicAdd(count + e_best, 1));
      }
    }
    __syncwarp();
    const float f = p.sigmoid ? p.scale / (sum + 1e-20f) : 1.f / (p.all ? total : sum);
    for (int k = lane; k < p.K; k += 32) p.w[(long long)t * p.K + k] *= f;
  }
}

// start[e] (shared memory) = first row of expert e, and expert_of_tile if this block writes it; all NTHR threads of a block
template <int NTHR>
__device__ __forceinline__ void plan_segments(const RouteArgs& p, const int* count, int* start, bool write) {
  __shared__ int part[32], carry;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (threadIdx.x == 0) carry = 0;
  __syncthreads();
  for (int e0 = 0; e0 < p.E; e0 += NTHR) {
    const int e = e0 + threadIdx.x;
    const int n = e < p.E ? (count[e] + 127) / 128 : 0;
    int s = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += v;
    }
    if (lane == 31) part[warp] = s;
    __syncthreads();
    if (warp == 0) {
      int q = lane < NTHR / 32 ? part[lane] : 0;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, q, o);
        if (lane >= o) q += v;
      }
      part[lane] = q;
    }
    __syncthreads();
    const int base = carry + (warp ? part[warp - 1] : 0) + s - n;
    if (e < p.E) {
      start[e] = base * 128;
      if (write)
        for (int i = 0; i < n && base + i < p.tiles; ++i) p.expert_of_tile[base + i] = e;
    }
    __syncthreads();
    if (threadIdx.x == 0) carry += part[31];
    __syncthreads();
  }
  if (write)
    for (int i = carry + threadIdx.x; i < p.tiles; i += NTHR) p.expert_of_tile[i] = -1;
}

constexpr int ROUTE_SMALL = 256, ROUTE_SMALL_ASSIGN = 4096;     // tokens and assignments that one block takes
template <int PER>
__global__ void __launch_bounds__(1024) moe_route_small_kernel(const RouteArgs p) {
  tfb::pdl_sync();
  extern __shared__ int sh[];               // count[E], start[E], expert[T K], rank[T K]
  int *count = sh, *start = sh + p.E, *s_e = start + p.E, *s_r = s_e + p.T * p.K;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int e = threadIdx.x; e < p.E; e += 1024) count[e] = 0;
  __syncthreads();
  for (int t = warp; t < p.T; t += 32)
    choose_experts<PER>(p, t, lane, count, [&](int i, int e, int r) { s_e[i] = e; s_r[i] = r; });
  __syncthreads();
  plan_segments<1024>(p, count, start, true);
  __syncthreads();
  for (int i = threadIdx.x; i < p.T * p.K; i += 1024) p.row_of[i] = start[s_e[i]] + s_r[i];
}

constexpr int ROUTE_TOKENS = 32;      // tokens of a block
template <int PER>
__global__ void __launch_bounds__(256) moe_route_choose_kernel(const RouteArgs p) {
  tfb::pdl_sync();
  extern __shared__ int count[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t0 = blockIdx.x * ROUTE_TOKENS, t1 = min(p.T, t0 + ROUTE_TOKENS);
  for (int e = threadIdx.x; e < p.E; e += 256) count[e] = 0;
  __syncthreads();
  for (int t = t0 + warp; t < t1; t += 8) choose_experts<PER>(p, t, lane, count, [&](int i, int, int r) { p.rank[i] = r; });
  __syncthreads();
  for (int e = threadIdx.x; e < p.E; e += 256) count[e] = count[e] ? atomicAdd(p.counts + e, count[e]) : 0;
  __syncthreads();
  for (int i = t0 * p.K + threadIdx.x; i < t1 * p.K; i += 256) p.rank[i] += count[p.idx[i]];
}
constexpr int ROUTE_ROWS = 2048;      // assignments of a block
__global__ void __launch_bounds__(256) moe_route_rows_kernel(const RouteArgs p) {
  tfb::pdl_sync();
  extern __shared__ int start[];
  plan_segments<256>(p, p.counts, start, blockIdx.x == 0);
  __syncthreads();
  const long long i0 = blockIdx.x * (long long)ROUTE_ROWS, n = (long long)p.T * p.K;
  for (int i = threadIdx.x; i < ROUTE_ROWS && i0 + i < n; i += 256) p.row_of[i0 + i] = start[p.idx[i0 + i]] + p.rank[i0 + i];
}

template <int PER>
static int launch_route(const RouteArgs& p, cudaStream_t st) {
  const size_t e4 = size_t(p.E) * 4;
  const long long a = (long long)p.T * p.K;
  if (p.T <= ROUTE_SMALL && a <= ROUTE_SMALL_ASSIGN && p.E <= 1024) {
    launch_k(moe_route_small_kernel<PER>, 1, 1024, 2 * e4 + size_t(a) * 8, st, p);
    return int(cudaGetLastError());
  }
  if (cudaError_t e = cudaMemsetAsync(p.counts, 0, e4, st)) return int(e);
  launch_k(moe_route_choose_kernel<PER>, (p.T + ROUTE_TOKENS - 1) / ROUTE_TOKENS, 256, e4, st, p);
  launch_k(moe_route_rows_kernel, int((a + ROUTE_ROWS - 1) / ROUTE_ROWS), 256, e4, st, p);
  return int(cudaGetLastError());
}

template <class T, int VEC>
__global__ void __launch_bounds__(256) moe_gather_kernel(const T* __restrict__ x, long long ldx, const int* __restrict__ row_of, T* __restrict__ xp,
                                                         long long ldp, long long assignments, int K, int H) {
  tfb::pdl_sync();
  const int per = H / VEC;
  const long long n = assignments * per;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += gridDim.x * 256ll) {
    const long long a = i / per;
    const int c = int(i - a * per) * VEC;
    float v[VEC];
    load_n<VEC>(x + a / K * ldx + c, v);
    store_n<VEC>(xp + row_of[a] * ldp + c, v);
  }
}

template <class T, int VEC, int ACT>
__global__ void __launch_bounds__(256) moe_glu_kernel(const T* __restrict__ in, long long ldi, const int* __restrict__ row_of, T* __restrict__ out,
                                                      long long ldo, long long assignments, int F, float limit) {
  tfb::pdl_sync();
  const int per = F / VEC;
  const long long n = assignments * per;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += gridDim.x * 256ll) {
    const long long a = i / per, row = row_of[a];
    const int c = int(i - a * per) * VEC;
    float g[VEC], u[VEC];
    load_n<VEC>(in + row * ldi + c, g);
    load_n<VEC>(in + row * ldi + F + c, u);
#pragma unroll
    for (int e = 0; e < VEC; ++e) g[e] = glu_value<ACT>(g[e], u[e], limit);
    store_n<VEC>(out + row * ldo + c, g);
  }
}

template <class T, int VEC>
__global__ void __launch_bounds__(256) moe_weighted_sum_kernel(const T* __restrict__ yp, long long ldp, const int* __restrict__ row_of,
                                                               const float* __restrict__ w, const T* __restrict__ base, long long ldb,
                                                               const float* __restrict__ gate, long long ldg, T* __restrict__ y, long long ldy,
                                                               int Tn, int K, int H) {
  tfb::pdl_sync();
  const int per = H / VEC;
  const long long n = (long long)Tn * per;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += gridDim.x * 256ll) {
    const long long t = i / per;
    const int c = int(i - t * per) * VEC;
    float acc[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
    for (int k = 0; k < K; ++k) {
      float v[VEC];
      load_n<VEC>(yp + row_of[t * K + k] * ldp + c, v);
      const float f = w[t * K + k];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = fmaf(f, v[e], acc[e]);
    }
    if (base) {
      float v[VEC];
      load_n<VEC>(base + t * ldb + c, v);
      const float f = gate ? 1.f / (1.f + expf(-gate[t * ldg])) : 1.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = fmaf(f, v[e], acc[e]);
    }
    store_n<VEC>(y + t * ldy + c, acc);
  }
}

static bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
static int blocks_for(long long items) {
  const long long b = (items + 255) / 256, cap = 148ll * 16;
  return int(b < 1 ? 1 : (b < cap ? b : cap));
}

}  // namespace tfb

using bf16 = __nv_bfloat16;

// logits [T, ld] fp32, bias [E] (bias_f32: fp32, otherwise bf16) or null; groups, keep, scale: see RouteArgs;
// score: 0 softmax over the chosen, 1 sigmoid, 2 softmax over all.  idx, row_of, rank (scratch): int [T, K]; w: fp32 [T, K]; counts
// (scratch): int [E]; expert_of_tile: int [tiles], tiles >= T K / 128 + min(E, T K).
TFB_API int tfb_moe_route(const float* logits, const void* bias, int T, int E, int K, int* idx, float* w, int* row_of, int* expert_of_tile,
                          int* counts, int* rank, int tiles, long long ld, int bias_f32, int score, int groups, int keep, float scale,
                          void* stream) {
  using namespace tfb;
  if (T <= 0 || E <= 0 || K <= 0 || K > E || score < 0 || score > 2) return TFB_ERR_ARG;
  const int sigmoid = score == 1;
  if (sigmoid && (bias || groups <= 0 || E % groups || keep <= 0 || keep > groups || K > E / groups * keep)) return TFB_ERR_ARG;
  if (!sigmoid && groups != 1) return TFB_ERR_ARG;
  const bool grouped = sigmoid && keep < groups;
  const long long a = (long long)T * K;
  if (tiles < a / 128 + (E < a ? E : a)) return TFB_ERR_ARG;
  if (E > 8192 || a > INT_MAX / 2) return TFB_ERR_LIMIT;
  RouteArgs p{logits, ld, bias, bias_f32, T, E, K, idx, w, rank, row_of, expert_of_tile, counts, tiles, sigmoid, groups, keep, score == 2, scale};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (grouped && (groups > 32 || E > 1024 || K > 32)) return TFB_ERR_LIMIT;
  if (grouped && E > 256) return launch_route<32>(p, st);
  if (K > 32 || E > 256) return launch_route<0>(p, st);
  return E <= 32 ? launch_route<1>(p, st) : E <= 64 ? launch_route<2>(p, st) : E <= 128 ? launch_route<4>(p, st) : launch_route<8>(p, st);
}

#define TFB_BY_TYPE(KERN, GRID, VECOK, ...)                                                                \
  do {                                                                                                     \
    if (f32) { if (VECOK) launch_k(KERN<float, 4>, GRID, 256, 0, st, __VA_ARGS__(float)); else launch_k(KERN<float, 1>, GRID, 256, 0, st, __VA_ARGS__(float)); } \
    else { if (VECOK) launch_k(KERN<bf16, 8>, GRID, 256, 0, st, __VA_ARGS__(bf16)); else launch_k(KERN<bf16, 1>, GRID, 256, 0, st, __VA_ARGS__(bf16)); } \
  } while (0)

TFB_API int tfb_moe_gather(const void* x, long long ldx, const int* row_of, void* xp, long long ldp, int T, int K, int H, int f32, void* stream) {
  using namespace tfb;
  if (T <= 0 || K <= 0 || H <= 0) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vec = f32 ? 4 : 8;
  const bool v = H % vec == 0 && ldx % vec == 0 && ldp % vec == 0 && al16(x) && al16(xp);
  const long long a = (long long)T * K;
#define TFB_ARGS(T) static_cast<const T*>(x), ldx, row_of, static_cast<T*>(xp), ldp, a, K, H
  TFB_BY_TYPE(moe_gather_kernel, blocks_for(a * (v ? H / vec : H)), v, TFB_ARGS);
#undef TFB_ARGS
  return int(cudaGetLastError());
}

// rows [gate | up] of 2 F entries -> act(gate) * up, for the `assignments` rows that row_of names; act, limit: see glu_value
TFB_API int tfb_moe_glu(const void* in, long long ldi, const int* row_of, void* out, long long ldo, int assignments, int F, int act, float limit, int f32,
                        void* stream) {
  using namespace tfb;
  if (assignments <= 0 || F <= 0 || act < 0 || act > GLU_CLAMPED) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vec = f32 ? 4 : 8;
  const bool v = F % vec == 0 && ldi % vec == 0 && ldo % vec == 0 && al16(in) && al16(out);
  const long long a = assignments;
  const int grid = blocks_for(a * (v ? F / vec : F));
#define TFB_GLU1(T, VEC, ACT) \
  launch_k(moe_glu_kernel<T, VEC, ACT>, grid, 256, 0, st, static_cast<const T*>(in), ldi, row_of, static_cast<T*>(out), ldo, a, F, limit)
#define TFB_GLU(T, VEC)                                    \
  do {                                                     \
    if (act == GLU_CLAMPED) TFB_GLU1(T, VEC, GLU_CLAMPED); \
    else if (act == GLU_GELU) TFB_GLU1(T, VEC, GLU_GELU);  \
    else TFB_GLU1(T, VEC, GLU_SILU);                       \
  } while (0)
  if (f32) { if (v) TFB_GLU(float, 4); else TFB_GLU(float, 1); }
  else { if (v) TFB_GLU(bf16, 8); else TFB_GLU(bf16, 1); }
#undef TFB_GLU
#undef TFB_GLU1
  return int(cudaGetLastError());
}

TFB_API int tfb_moe_weighted_sum(const void* yp, long long ldp, const int* row_of, const float* w, const void* base, long long ldb,
                                 const float* gate, long long ldg, void* y, long long ldy, int T, int K, int H, int f32, void* stream) {
  using namespace tfb;
  if (T <= 0 || K <= 0 || H <= 0) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vec = f32 ? 4 : 8;
  const bool v = H % vec == 0 && ldp % vec == 0 && ldy % vec == 0 && al16(yp) && al16(y) && (!base || (ldb % vec == 0 && al16(base)));
#define TFB_ARGS(Ty) static_cast<const Ty*>(yp), ldp, row_of, w, static_cast<const Ty*>(base), ldb, gate, ldg, static_cast<Ty*>(y), ldy, T, K, H
  TFB_BY_TYPE(moe_weighted_sum_kernel, blocks_for((long long)T * (v ? H / vec : H)), v, TFB_ARGS);
#undef TFB_ARGS
  return int(cudaGetLastError());
}
