// Hyper-connected residual: S streams of 32-bit rows instead of one.  Around a sublayer
//
//   u = sum_s in[s] x_s;   y = sublayer(norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y      (all t at once from the old streams)
//
// What lies between two sublayers is one pass over the row: norms of the outputs of the one (of two mixers side by side: each its own,
// their share of the sum), the new streams, and the normed input of the other.  The norm of that input is an RMS norm in groups:
// `groups` equal consecutive parts of the row, each divided by its own root mean square.
//
// One block per row.  A thread owns the same columns of all streams, so the mixing needs no exchange; only the statistics do.
#include "tfb_elem.cuh"
#include "tfb_host.h"

namespace tfb {
TFB_BOUNDS_DEFINE(streams)

constexpr int MAX_STREAMS = 16;

struct StreamArgs {
  const long long* ids;       // null, or the streams all start as scale * table[id]
  const void* table;
  long long ld_table;
  float scale;
  int vocab;
  float* x;                   // [n, S, H]
  int S, H;
  const void *y, *y2;         // outputs of the sublayer [n, ldy], or null
  long long ldy, ldy2;
  const void *w_post, *w_post2;   // [H] weights of RMS norms on y and y2, or null
  float share;                // of the sum of y and y2
  const void *mix, *out;      // [S, S], [S] of the sublayer that returned y
  const void *in;             // [S] of the next one; null: the sum of the streams
  const void* w;              // [H] weight of the norm of what the next one reads, or null: nothing is returned
  int groups;
  void* a;                    // [n, lda]
  long long lda;
  const int* rows;            // null, or: output row i comes from row rows[i], and x is left alone
  float eps;
};

__device__ __forceinline__ float2 block_add2(float2 v, float2* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
    v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
  }
  const int nw = blockDim.x >> 5, lane = threadIdx.x & 31;
  if (nw == 1) return v;
  if (lane == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = lane < nw ? red[lane] : make_float2(0.f, 0.f);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
    v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
  }
  __syncthreads();
  return v;
}

// ST: streams (0: any number up to MAX_STREAMS).  Dynamic shared memory: H / VEC sums of squares and `groups` factors, with more than one group.
template <class T, int ST, int VEC, int NV>
__global__ void stream_norm_kernel(const StreamArgs p) {
  tfb::pdl_sync();
  constexpr int SM = ST ? ST : MAX_STREAMS;
  extern __shared__ float part[];
  __shared__ float2 red[32];
  __shared__ float s_mix[SM * SM], s_out[SM], s_in[SM];
  const int S = ST ? ST : p.S, i = blockIdx.x, nt = blockDim.x, H = p.H;
  const long long r = p.rows ? p.rows[i] : i;
  for (int e = threadIdx.x; e < S * S; e += nt) s_mix[e] = p.y ? to_f(static_cast<const T*>(p.mix)[e]) : 0.f;
  for (int e = threadIdx.x; e < S; e += nt) {
    s_out[e] = p.y ? to_f(static_cast<const T*>(p.out)[e]) : 0.f;
    s_in[e] = p.in ? to_f(static_cast<const T*>(p.in)[e]) : 1.f;
  }
  const T* trow = nullptr;
  if (p.ids) {
    long long id = p.ids[r];
    TFB_BOUNDS(id >= 0 && id < p.vocab, 1, id, p.vocab);
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    trow = static_cast<const T*>(p.table) + id * p.ld_table;
  }
  // the streams are on their way while the statistics of y are taken, where the registers hold them
  constexpr bool EARLY = ST > 0 && ST * NV * VEC <= 32;
  float early[EARLY ? NV : 1][SM][VEC];
  auto load_streams = [&](int col, float (&v)[SM][VEC]) {
    if (trow) {
      load_n<VEC>(trow + col, v[0]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[0][e] *= p.scale;
#pragma unroll
      for (int s = 1; s < SM; ++s)
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[s][e] = v[0][e];
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) load_n<VEC>(p.x + (r * S + s) * H + col, v[s]);
    }
  };
  if constexpr (EARLY) {
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int col = (c * nt + threadIdx.x) * VEC;
      if (col < H) load_streams(col, early[c]);
    }
  }
  float y[NV][VEC];
  if (p.y) {
    float y2[NV][VEC];
    float2 ss = make_float2(0.f, 0.f);
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int col = (c * nt + threadIdx.x) * VEC;
      if (col >= H) continue;
      load_n<VEC>(static_cast<const T*>(p.y) + r * p.ldy + col, y[c]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss.x = fmaf(y[c][e], y[c][e], ss.x);
      if (!p.y2) continue;
      load_n<VEC>(static_cast<const T*>(p.y2) + r * p.ldy2 + col, y2[c]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss.y = fmaf(y2[c][e], y2[c][e], ss.y);
    }
    float f = p.share, f2 = p.share;
    if (p.w_post || p.w_post2) {
      ss = block_add2(ss, red);
      if (p.w_post) f *= 1.f / sqrtf(ss.x / H + p.eps);
      if (p.w_post2) f2 *= 1.f / sqrtf(ss.y / H + p.eps);
    }
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int col = (c * nt + threadIdx.x) * VEC;
      if (col >= H) continue;
      float w[VEC];
      if (p.w_post) load_n<VEC>(static_cast<const T*>(p.w_post) + col, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[c][e] *= p.w_post ? f * w[e] : f;
      if (!p.y2) continue;
      if (p.w_post2) load_n<VEC>(static_cast<const T*>(p.w_post2) + col, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[c][e] = fmaf(y2[c][e], p.w_post2 ? f2 * w[e] : f2, y[c][e]);
    }
  }
  __syncthreads();                       // the coefficients are there
  float u[NV][VEC];                      // what the next sublayer reads
#pragma unroll
  for (int c = 0; c < NV; ++c) {
    const int col = (c * nt + threadIdx.x) * VEC;
    if (col >= H) continue;
    float late[SM][VEC];
    float* xr = p.x + r * S * H + col;
    if constexpr (!EARLY) load_streams(col, late);
    float (&v)[SM][VEC] = EARLY ? early[EARLY ? c : 0] : late;
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[c][e] = 0.f;
#pragma unroll
    for (int t = 0; t < SM; ++t) {
      if (t >= S) continue;
      float n[VEC];
      if (p.y) {
        const float o = s_out[t];
#pragma unroll
        for (int e = 0; e < VEC; ++e) n[e] = o * y[c][e];
#pragma unroll
        for (int s = 0; s < SM; ++s) {
          if (s >= S) continue;
          const float m = s_mix[s * S + t];
#pragma unroll
          for (int e = 0; e < VEC; ++e) n[e] = fmaf(m, v[s][e], n[e]);
        }
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) n[e] = v[t][e];
      }
      if (!p.rows && (p.y || trow)) store_n<VEC>(xr + (long long)t * H, n);
      const float g = s_in[t];
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[c][e] = fmaf(g, n[e], u[c][e]);
    }
  }
  if (!p.w) return;
  float f_row = 0.f;
  float* factor = part + H / VEC;        // [groups]
  const int per = H / p.groups;          // a multiple of VEC
  if (p.groups == 1) {
    float2 ss = make_float2(0.f, 0.f);
#pragma unroll
    for (int c = 0; c < NV; ++c)
      if (int((c * nt + threadIdx.x) * VEC) < H) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss.x = fmaf(u[c][e], u[c][e], ss.x);
      }
    f_row = 1.f / sqrtf(block_add2(ss, red).x / H + p.eps);
  } else {
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int q = c * nt + threadIdx.x;
      if (q * VEC >= H) continue;
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(u[c][e], u[c][e], ss);
      part[q] = ss;
    }
    __syncthreads();
    const int lane = threadIdx.x & 31;
    for (int g = threadIdx.x >> 5; g < p.groups; g += nt >> 5) {
      float ss = 0.f;
      for (int q = lane; q < per / VEC; q += 32) ss += part[g * (per / VEC) + q];
      ss = warp_add(ss);
      if (lane == 0) factor[g] = 1.f / sqrtf(ss / per + p.eps);
    }
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < NV; ++c) {
    const int col = (c * nt + threadIdx.x) * VEC;
    if (col >= H) continue;
    const float f = p.groups == 1 ? f_row : factor[col / per];
    float w[VEC];
    load_n<VEC>(static_cast<const T*>(p.w) + col, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[c][e] *= f * w[e];
    store_n<VEC>(static_cast<T*>(p.a) + (long long)i * p.lda + col, u[c]);
  }
}

template <class T, int ST, int VEC>
static int launch_streams(const StreamArgs& p, int n, cudaStream_t st) {
  const int items = (p.H + VEC - 1) / VEC;
  int nt = (items + 31) / 32 * 32;
  const int cap = VEC == 1 ? 512 : 256;
  if (nt > cap) nt = cap;
  const int nv = (items + nt - 1) / nt;
  const size_t sm = p.groups > 1 ? (size_t(items) + p.groups) * 4 : 0;
  if (sm > 40 * 1024) return TFB_ERR_LIMIT;
  if (nv <= 1) launch_k(stream_norm_kernel<T, ST, VEC, 1>, n, nt, sm, st, p);
  else if (nv <= 2) launch_k(stream_norm_kernel<T, ST, VEC, 2>, n, nt, sm, st, p);
  else if (nv <= 4) launch_k(stream_norm_kernel<T, ST, VEC, 4>, n, nt, sm, st, p);
  else if (nv <= 8) launch_k(stream_norm_kernel<T, ST, VEC, 8>, n, nt, sm, st, p);
  else if (VEC == 1 && nv <= 16) launch_k(stream_norm_kernel<T, ST, VEC, VEC == 1 ? 16 : 8>, n, nt, sm, st, p);
  else return TFB_ERR_LIMIT;
  return int(cudaGetLastError());
}

template <class T, int VEC>
static int launch_by_streams(const StreamArgs& p, int n, cudaStream_t st) {
  switch (p.S) {
    case 1: return launch_streams<T, 1, VEC>(p, n, st);
    case 2: return launch_streams<T, 2, VEC>(p, n, st);
    case 3: return launch_streams<T, 3, VEC>(p, n, st);
    case 4: return launch_streams<T, 4, VEC>(p, n, st);
    default: return launch_streams<T, 0, 1>(p, n, st);
  }
}

}  // namespace tfb

// See StreamArgs.  f32 = 1: outputs, table, weights and coefficients are fp32, otherwise bf16; the streams are fp32.
TFB_API int tfb_stream_norm(const long long* ids, const void* table, long long ld_table, float scale, int vocab, float* x, int S, const void* y, long long ldy,
                            const void* y2, long long ldy2, const void* w_post, const void* w_post2, float share, const void* mix, const void* out,
                            const void* in, const void* w, int groups, void* a, long long lda, const int* rows, int n, int H, float eps, int f32,
                            void* stream) {
  using namespace tfb;
  if (n <= 0 || H <= 0 || S <= 0 || groups <= 0 || H % groups || (ids && !table) || (y && (!mix || !out)) || (y2 && !y) || (w_post && !y) ||
      (w_post2 && !y2) || (w && !a))
    return TFB_ERR_ARG;
  if (S > MAX_STREAMS) return TFB_ERR_LIMIT;
  const StreamArgs p{ids, table, ld_table, scale, vocab, x, S, H, y, y2, ldy, ldy2, w_post, w_post2, share, mix, out, in, w, groups, a, lda, rows, eps};
  const int es = f32 ? 4 : 2;
  auto al = [](const void* q, int b) { return (reinterpret_cast<uintptr_t>(q) & (b - 1)) == 0; };
  auto ok = [&](int vec) {
    bool v = H % vec == 0 && H / groups % vec == 0 && al(x, 16) && ldy % vec == 0 && ldy2 % vec == 0 && lda % vec == 0 && ld_table % vec == 0;
    for (const void* q : {y, y2, w_post, w_post2, w, table, static_cast<const void*>(a)}) v = v && al(q, vec * es);
    return v;
  };
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) return ok(4) ? launch_by_streams<float, 4>(p, n, st) : launch_streams<float, 0, 1>(p, n, st);
  if (ok(8) && H > 512) return launch_by_streams<__nv_bfloat16, 8>(p, n, st);
  return ok(4) ? launch_by_streams<__nv_bfloat16, 4>(p, n, st) : launch_streams<__nv_bfloat16, 0, 1>(p, n, st);
}
