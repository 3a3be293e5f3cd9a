// Row operators of decoders with a 32-bit residual stream: scaled embedding, norm of a sublayer's output + residual + norm of (or
// rounding for) the next sublayer's input in one pass, activations, norm of the recurrent mixers' head outputs, partial rotary embedding
// (with a norm of the heads in front) fused with the append to the paged cache, gather of cached rows, and a true fp32 matrix product
// (dense, one block per head, or rows grouped by expert).  Every kernel exists for bf16 and for fp32
// activations; the statistics, the residual and the rotation are fp32 in both.
#include "tfb_elem.cuh"
#include "tfb_host.h"

namespace tfb {
TFB_BOUNDS_DEFINE(stack_ops)

// ------------------------------------------------------------------------------------------------
// x <- x + norm(y) [* scale_post] [+ y2], y itself without w_post;  a = norm(x), or x itself without w_pre
// norm: NORM_CENTRED: v / rms(v) * (1 + w); NORM_PLAIN: v / rms(v) * w; NORM_LAYER: (v - mean) / sqrt(mean squared deviation + eps) * w + b.
// ids != null: x starts as scale * table[id] (normed with w_post if there is no y) instead of being read.  rows != null: output row i is computed from row
// rows[i] of x and y, and x is left alone (the last norm of a step, for the positions whose logits are wanted).
// One block per row; the row lives in registers between the two statistics.
// ------------------------------------------------------------------------------------------------
struct ResNormArgs {
  const long long* ids;
  const void* table;
  long long ld_table;
  float scale;
  int vocab;
  float* x;
  long long ldx;
  const void* y;
  long long ldy;
  const void* y2;
  long long ldy2;
  const void *w_post, *b_post, *scale_post, *w_pre, *b_pre;
  void* a;
  long long lda;
  const int* rows;
  int H;
  float eps;
};

enum { NORM_CENTRED = 0, NORM_LAYER = 1, NORM_PLAIN = 2 };

// statistics of a row held in the block's registers: the mean to subtract (0 unless NORM_LAYER) and the factor
template <int NORM, int VEC, int NV>
__device__ __forceinline__ float2 row_stats(const float (&v)[NV][VEC], int H, float eps, float* red) {
  constexpr bool LAYER = NORM == NORM_LAYER;
  const int nt = blockDim.x;
  float mean = 0.f;
  if constexpr (LAYER) {
    float s = 0.f;
#pragma unroll
    for (int c = 0; c < NV; ++c)
      if (int((c * nt + threadIdx.x) * VEC) < H) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) s += v[c][e];
      }
    mean = block_add(s, red) / H;
  }
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NV; ++c)
    if (int((c * nt + threadIdx.x) * VEC) < H) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float d = LAYER ? v[c][e] - mean : v[c][e];
        ss = fmaf(d, d, ss);
      }
    }
  return make_float2(mean, 1.f / sqrtf(block_add(ss, red) / H + eps));
}

template <class T, int NORM, int VEC>
__device__ __forceinline__ void apply_norm(float (&v)[VEC], float2 st, const void* w, const void* b, int col) {
  float wv[VEC];
  load_n<VEC>(static_cast<const T*>(w) + col, wv);
  if constexpr (NORM == NORM_LAYER) {
    float bv[VEC];
    load_n<VEC>(static_cast<const T*>(b) + col, bv);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = (v[e] - st.x) * st.y * wv[e] + bv[e];
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = v[e] * st.y * (NORM == NORM_PLAIN ? wv[e] : 1.f + wv[e]);
  }
}

template <class T, int NORM, int VEC, int NV>
__global__ void res_norm_kernel(const ResNormArgs p) {
  tfb::pdl_sync();
  __shared__ float red[32];
  const int i = blockIdx.x, nt = blockDim.x;
  const long long r = p.rows ? p.rows[i] : i;
  float v[NV][VEC];
  const T* trow = nullptr;
  if (p.ids) {
    long long id = p.ids[r];
    TFB_BOUNDS(id >= 0 && id < p.vocab, 1, id, p.vocab);
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    trow = static_cast<const T*>(p.table) + id * p.ld_table;
  }
#pragma unroll
  for (int c = 0; c < NV; ++c) {
    const int col = (c * nt + threadIdx.x) * VEC;
    if (col >= p.H) continue;
    if (trow) {
      load_n<VEC>(trow + col, v[c]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[c][e] *= p.scale;
    } else {
      load_n<VEC>(p.x + r * p.ldx + col, v[c]);
    }
  }
  if (p.y) {
    float yv[NV][VEC];
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int col = (c * nt + threadIdx.x) * VEC;
      if (col < p.H) load_n<VEC>(static_cast<const T*>(p.y) + r * p.ldy + col, yv[c]);
    }
    float2 st = make_float2(0.f, 1.f);
    if (p.w_post) st = row_stats<NORM, VEC, NV>(yv, p.H, p.eps, red);
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int col = (c * nt + threadIdx.x) * VEC;
      if (col >= p.H) continue;
      if (p.w_post) apply_norm<T, NORM, VEC>(yv[c], st, p.w_post, p.b_post, col);
      if (p.scale_post) {
        float s[VEC];
        load_n<VEC>(static_cast<const T*>(p.scale_post) + col, s);
#pragma unroll
        for (int e = 0; e < VEC; ++e) yv[c][e] *= s[e];
      }
      if (p.y2) {
        float z[VEC];
        load_n<VEC>(static_cast<const T*>(p.y2) + r * p.ldy2 + col, z);
#pragma unroll
        for (int e = 0; e < VEC; ++e) yv[c][e] += z[e];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[c][e] += yv[c][e];
    }
  } else if (p.w_post) {                 // the embedding's own norm
    const float2 st = row_stats<NORM, VEC, NV>(v, p.H, p.eps, red);
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int col = (c * nt + threadIdx.x) * VEC;
      if (col < p.H) apply_norm<T, NORM, VEC>(v[c], st, p.w_post, p.b_post, col);
    }
  }
  if (!p.rows && (p.y || p.ids)) {
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const int col = (c * nt + threadIdx.x) * VEC;
      if (col < p.H) store_n<VEC>(p.x + r * p.ldx + col, v[c]);
    }
  }
  if (!p.a) return;
  float2 st = make_float2(0.f, 1.f);
  if (p.w_pre) st = row_stats<NORM, VEC, NV>(v, p.H, p.eps, red);
#pragma unroll
  for (int c = 0; c < NV; ++c) {
    const int col = (c * nt + threadIdx.x) * VEC;
    if (col >= p.H) continue;
    if (p.w_pre) apply_norm<T, NORM, VEC>(v[c], st, p.w_pre, p.b_pre, col);
    store_n<VEC>(static_cast<T*>(p.a) + (long long)i * p.lda + col, v[c]);
  }
}

template <class T, int NORM, int VEC>
static int launch_res_norm(const ResNormArgs& p, int n, cudaStream_t st) {
  const int items = (p.H + VEC - 1) / VEC;
  int nt = (items + 31) / 32 * 32;
  const int cap = VEC == 1 ? 512 : 256;
  if (nt > cap) nt = cap;
  const int nv = (items + nt - 1) / nt;
  if (nv <= 1) launch_k(res_norm_kernel<T, NORM, VEC, 1>, n, nt, 0, st, p);
  else if (nv <= 2) launch_k(res_norm_kernel<T, NORM, VEC, 2>, n, nt, 0, st, p);
  else if (nv <= 4) launch_k(res_norm_kernel<T, NORM, VEC, 4>, n, nt, 0, st, p);
  else if (nv <= 8) launch_k(res_norm_kernel<T, NORM, VEC, 8>, n, nt, 0, st, p);
  else return TFB_ERR_LIMIT;
  return int(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------
// act of every entry (codes of the product epilogue: 4 = squared relu)
// ------------------------------------------------------------------------------------------------
__device__ __forceinline__ float act_f32(float v, int act) {
  if (act == 4) {
    v = fmaxf(v, 0.f);
    return v * v;
  }
  return v;
}

template <class T>
__global__ void __launch_bounds__(256) act_rows_kernel(const T* __restrict__ in, long long ldi, T* __restrict__ out, long long ldo, int M, int N, int act) {
  tfb::pdl_sync();
  const long long n = (long long)M * N;
  for (long long t = blockIdx.x * (long long)blockDim.x + threadIdx.x; t < n; t += (long long)gridDim.x * blockDim.x)
    out[t / N * ldo + t % N] = from_f<T>(act_f32(to_f(in[t / N * ldi + t % N]), act));
}

// ------------------------------------------------------------------------------------------------
// [gate | up] -> act(gate) * up; act: see glu_value (tfb_elem.cuh)
// ------------------------------------------------------------------------------------------------
template <class T, int VEC, int ACT>
__global__ void __launch_bounds__(256) glu_kernel(const T* __restrict__ in, long long ldi, T* __restrict__ out, long long ldo, int M, int F,
                                                  float limit) {
  tfb::pdl_sync();
  const int per = F / VEC;
  const long long n = (long long)M * per;
  for (long long t = blockIdx.x * (long long)blockDim.x + threadIdx.x; t < n; t += (long long)gridDim.x * blockDim.x) {
    const long long m = t / per;
    const int c = int(t % per) * VEC;
    float g[VEC], u[VEC];
    load_n<VEC>(in + m * ldi + c, g);
    load_n<VEC>(in + m * ldi + F + c, u);
#pragma unroll
    for (int e = 0; e < VEC; ++e) g[e] = glu_value<ACT>(g[e], u[e], limit);
    store_n<VEC>(out + m * ldo + c, g);
  }
}

// ------------------------------------------------------------------------------------------------
// norm of the head outputs of a recurrent mixer:  o / rms(o) [* w] [* silu(gate)]
// ------------------------------------------------------------------------------------------------
template <class T, int VEC>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long ldg,
                                                         const T* __restrict__ w, T* __restrict__ out, long long ldo, int rows, int H, int V,
                                                         float eps) {
  tfb::pdl_sync();
  const int lane = threadIdx.x & 31;
  const long long nwarps = (long long)gridDim.x * (blockDim.x >> 5), n = (long long)rows * H;
  for (long long i = blockIdx.x * (long long)(blockDim.x >> 5) + (threadIdx.x >> 5); i < n; i += nwarps) {
    const long long r = i / H;
    const int h = int(i % H);
    const float* src = o + i * V;
    const T* gt = gate ? gate + r * ldg + h * V : nullptr;
    T* dst = out + r * ldo + h * V;
    float x0[VEC], g0[VEC], x[VEC], g[VEC], wv[VEC];
    float ss = 0.f;
    for (int j = lane * VEC; j < V; j += 32 * VEC) {
      load_n<VEC>(src + j, x);
      if (j == lane * VEC) {
        if (gt) load_n<VEC>(gt + j, g0);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x0[e] = x[e];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(x[e], x[e], ss);
    }
    const float rs = 1.f / sqrtf(warp_add(ss) / V + eps);
    for (int j = lane * VEC; j < V; j += 32 * VEC) {
      if (w) load_n<VEC>(w + j, wv);
      if (j == lane * VEC) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) { x[e] = x0[e]; g[e] = g0[e]; }
      } else {
        load_n<VEC>(src + j, x);
        if (gt) load_n<VEC>(gt + j, g);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] *= rs * (w ? wv[e] : 1.f) * (gt ? silu_exact(g[e]) : 1.f);
      store_n<VEC>(dst + j, x);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// Rotary embedding of the first `dims` entries of every q and k head, in place, and append of k and v to the paged pools.
// Rows: [nq heads of D | nk heads of D | v_cols].  Pools are [slots][nk * D] and [slots][v_cols]; a negative slot (padding,
// or a position no later query can see) is not cached.  nk = 0: the layer has queries only.
// ------------------------------------------------------------------------------------------------
template <class T, int VEC>
__global__ void __launch_bounds__(256) rope_append_kernel(T* __restrict__ qkv, long long ld, const float* __restrict__ cos_t,
                                                          const float* __restrict__ sin_t, int max_pos, const int* __restrict__ positions,
                                                          const long long* __restrict__ slots, T* __restrict__ kpool,
                                                          T* __restrict__ vpool, long long nslots, int rows, int nq, int nk, int D,
                                                          int dims, int v_cols) {
  tfb::pdl_sync();
  const int half = dims >> 1, hv = half / VEC, pv = (D - dims) / VEC, vv = v_cols / VEC;
  const int per_rot = (nq + nk) * hv, per_pass = nk * pv;
  const int per = per_rot + per_pass + vv;          // work items of one row: rotated pairs, k entries that pass, v entries
  const long long n = (long long)rows * per;
  for (long long t = blockIdx.x * (long long)blockDim.x + threadIdx.x; t < n; t += (long long)gridDim.x * blockDim.x) {
    const long long r = t / per;
    int w = int(t % per);
    T* row = qkv + r * ld;
    long long slot = (slots && nk) ? slots[r] : -1;
    TFB_BOUNDS(slot < nslots, 51, slot, nslots);
    if (slot >= nslots) slot = -1;
    if (w < per_rot) {
      int pos = positions[r];
      TFB_BOUNDS(pos >= 0 && pos < max_pos, 61, pos, max_pos);
      pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
      const int head = w / hv, i = (w % hv) * VEC;
      float u[VEC], v[VEC], c[VEC], s[VEC], a[VEC], b[VEC];
      load_n<VEC>(row + head * D + i, u);
      load_n<VEC>(row + head * D + half + i, v);
      load_n<VEC>(cos_t + (long long)pos * half + i, c);
      load_n<VEC>(sin_t + (long long)pos * half + i, s);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        a[e] = u[e] * c[e] - v[e] * s[e];
        b[e] = v[e] * c[e] + u[e] * s[e];
      }
      store_n<VEC>(row + head * D + i, a);
      store_n<VEC>(row + head * D + half + i, b);
      if (head >= nq && slot >= 0) {
        T* kp = kpool + (slot * nk + (head - nq)) * D;
        store_n<VEC>(kp + i, a);
        store_n<VEC>(kp + half + i, b);
      }
    } else if (slot >= 0) {
      w -= per_rot;
      float u[VEC];
      if (w < per_pass) {
        const int head = w / pv, i = dims + (w % pv) * VEC;
        load_n<VEC>(row + (nq + head) * D + i, u);
        store_n<VEC>(kpool + (slot * nk + head) * D + i, u);
      } else {
        const int i = (w - per_pass) * VEC;
        load_n<VEC>(row + (long long)(nq + nk) * D + i, u);
        store_n<VEC>(vpool + slot * v_cols + i, u);
      }
    }
  }
}

// The same with an RMS norm of every q and k head (weights wq, wk; null: none) in front of the rotation and, behind it, a factor per query
// head (qf, or null).  L lanes share a head, each with two pieces
// of four entries in registers: for rotated entries, four of the first half and their partners in the second (L a power of two,
// 8 L >= D; D, v_cols and the rotated entries are multiples of eight).  Units of a row: nq + nk heads, then pieces of 8 L entries of v; a
// group of L lanes takes NRA_UNITS of them, all loads ahead of the reductions.
constexpr int NRA_UNITS = 2;
template <class T, int L>
__global__ void __launch_bounds__(256, 4) norm_rope_append_kernel(T* __restrict__ qkv, long long ld, const T* __restrict__ wq, const T* __restrict__ wk,
                                                                  const T* __restrict__ qf, float eps, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                                                  int max_pos, const int* __restrict__ positions, const long long* __restrict__ slots,
                                                                  T* __restrict__ kpool, T* __restrict__ vpool, long long nslots, int rows, int nq,
                                                                  int nk, int D, int dims, int v_cols) {
  tfb::pdl_sync();
  const int l = threadIdx.x % L, heads = nq + nk, units = heads + (v_cols + 8 * L - 1) / (8 * L), per = (units + NRA_UNITS - 1) / NRA_UNITS;
  const int id = (blockIdx.x * 256 + threadIdx.x) / L, r = min(id / per, rows - 1), u0 = id - id / per * per;
  const bool on = id < rows * per, turns = l * 8 < dims;
  const int c0 = turns ? l * 4 : l * 8, c1 = turns ? dims / 2 + l * 4 : l * 8 + 4;     // this lane's entries of a head
  T* row = qkv + r * ld;
  float x[NRA_UNITS][2][4], w[NRA_UNITS][2][4], c[4], s[4];
  int at[NRA_UNITS];                               // first entry of the unit in the row; negative: none for this lane
#pragma unroll
  for (int i = 0; i < NRA_UNITS; ++i) {
    const int u = u0 + i * per;
    at[i] = u < heads ? u * D : heads * D + (u - heads) * 8 * L;
    if (!on || u >= units || (u < heads ? l * 8 >= D : at[i] + l * 8 >= heads * D + v_cols)) at[i] = -1;
#pragma unroll
    for (int e = 0; e < 4; ++e) x[i][0][e] = x[i][1][e] = 0.f;
    if (at[i] < 0) continue;
    const int a = u < heads ? c0 : l * 8, b = u < heads ? c1 : l * 8 + 4;
    load_n<4>(row + at[i] + a, x[i][0]);
    load_n<4>(row + at[i] + b, x[i][1]);
    if (u < heads && wq) {
      load_n<4>((u < nq ? wq : wk) + c0, w[i][0]);
      load_n<4>((u < nq ? wq : wk) + c1, w[i][1]);
    }
  }
  if (turns) {
    int pos = positions[r];
    TFB_BOUNDS(pos >= 0 && pos < max_pos, 61, pos, max_pos);
    pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
    load_n<4>(cos_t + (long long)pos * (dims / 2) + c0, c);
    load_n<4>(sin_t + (long long)pos * (dims / 2) + c0, s);
  }
  long long slot = slots ? slots[r] : -1;
  TFB_BOUNDS(slot < nslots, 51, slot, nslots);
  if (slot >= nslots) slot = -1;
  float ss[NRA_UNITS];
#pragma unroll
  for (int i = 0; i < NRA_UNITS; ++i) {
    ss[i] = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) ss[i] = fmaf(x[i][0][e], x[i][0][e], fmaf(x[i][1][e], x[i][1][e], ss[i]));
  }
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1)
#pragma unroll
    for (int i = 0; i < NRA_UNITS; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
  const float inv = 1.f / D;
#pragma unroll
  for (int i = 0; i < NRA_UNITS; ++i) {
    if (at[i] < 0) continue;
    const int u = u0 + i * per;
    if (u >= heads) {
      if (slot >= 0) {
        T* vp = vpool + slot * v_cols + (u - heads) * 8 * L + l * 8;
        store_n<4>(vp, x[i][0]);
        store_n<4>(vp + 4, x[i][1]);
      }
      continue;
    }
    const float f = rsqrtf(fmaf(ss[i], inv, eps)) * (qf && u < nq ? to_f(qf[u]) : 1.f);
    float a[4], b[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      a[e] = x[i][0][e] * f * (wq ? w[i][0][e] : 1.f);
      b[e] = x[i][1][e] * f * (wq ? w[i][1][e] : 1.f);
      if (turns) {
        const float p = a[e] * c[e] - b[e] * s[e];
        b[e] = b[e] * c[e] + a[e] * s[e];
        a[e] = p;
      }
    }
    store_n<4>(row + at[i] + c0, a);
    store_n<4>(row + at[i] + c1, b);
    if (u >= nq && slot >= 0) {
      T* kp = kpool + (slot * nk + (u - nq)) * D;
      store_n<4>(kp + c0, a);
      store_n<4>(kp + c1, b);
    }
  }
}

// any sizes: one warp per head (or per 64 entries of v)
template <class T>
__global__ void __launch_bounds__(256) norm_rope_append_any_kernel(T* __restrict__ qkv, long long ld, const T* __restrict__ wq, const T* __restrict__ wk,
                                                                   const T* __restrict__ qf, float eps, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                                                   int max_pos, const int* __restrict__ positions, const long long* __restrict__ slots,
                                                                   T* __restrict__ kpool, T* __restrict__ vpool, long long nslots, int rows, int nq,
                                                                   int nk, int D, int dims, int v_cols) {
  tfb::pdl_sync();
  const int lane = threadIdx.x & 31, units = nq + nk + (v_cols + 63) / 64, half = dims / 2;
  const long long id = (blockIdx.x * 256ll + threadIdx.x) / 32;
  if (id >= (long long)rows * units) return;
  const long long r = id / units;
  const int u = int(id % units);
  long long slot = slots ? slots[r] : -1;
  TFB_BOUNDS(slot < nslots, 51, slot, nslots);
  if (slot >= nslots) slot = -1;
  T* row = qkv + r * ld;
  if (u >= nq + nk) {
    for (int c = (u - nq - nk) * 64 + lane; slot >= 0 && c < min(v_cols, (u - nq - nk + 1) * 64); c += 32)
      vpool[slot * v_cols + c] = row[(long long)(nq + nk) * D + c];
    return;
  }
  T* x = row + u * D;
  const T* w = u < nq ? wq : wk;
  T* kp = u >= nq && slot >= 0 ? kpool + (slot * nk + (u - nq)) * D : nullptr;
  float ss = 0.f;
  for (int d = lane; d < D; d += 32) ss = fmaf(to_f(x[d]), to_f(x[d]), ss);
  const float f = 1.f / sqrtf(warp_add(ss) / D + eps) * (qf && u < nq ? to_f(qf[u]) : 1.f);     // its shuffles also order the reads before the writes below
  int pos = dims ? positions[r] : 0;
  TFB_BOUNDS(dims == 0 || (pos >= 0 && pos < max_pos), 61, pos, max_pos);
  pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
  for (int d = lane; d < D; d += 32) {
    if (d >= half && d < dims) continue;
    const float a = to_f(x[d]) * f * (w ? to_f(w[d]) : 1.f);
    if (d >= dims) {
      x[d] = from_f<T>(a);
      if (kp) kp[d] = from_f<T>(a);
      continue;
    }
    const float b = to_f(x[d + half]) * f * (w ? to_f(w[d + half]) : 1.f);
    const float c = cos_t[(long long)pos * half + d], s = sin_t[(long long)pos * half + d];
    const T p = from_f<T>(a * c - b * s), q = from_f<T>(b * c + a * s);
    x[d] = p;
    x[d + half] = q;
    if (kp) {
      kp[d] = p;
      kp[d + half] = q;
    }
  }
}

// rows lo .. lo + n - 1 of one sequence (its page list) out of a pool [slots][width], contiguous
template <class T, int VEC>
__global__ void __launch_bounds__(256) gather_rows_kernel(const T* __restrict__ pool, long long nslots, const int* __restrict__ pages,
                                                          int page, int lo, int n, T* __restrict__ out, int width) {
  tfb::pdl_sync();
  const int per = width / VEC;
  const long long total = (long long)n * per;
  for (long long t = blockIdx.x * (long long)blockDim.x + threadIdx.x; t < total; t += (long long)gridDim.x * blockDim.x) {
    const int r = int(t / per), c = int(t % per) * VEC, pos = lo + r;
    const long long slot = (long long)pages[pos / page] * page + pos % page;
    TFB_BOUNDS(slot >= 0 && slot < nslots, 53, slot, nslots);
    float u[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[e] = 0.f;
    if (slot >= 0 && slot < nslots) load_n<VEC>(pool + slot * width + c, u);
    store_n<VEC>(out + (long long)r * width + c, u);
  }
}

// ------------------------------------------------------------------------------------------------
// C[M, N] = act(A[M, K] . B^T) in true fp32 (FFMA), 64 x 64 tiles, any sizes and pitches.
// B is [N, K], or [K, N] with b_kn.  Products of several heads (grid z): A, B, C advance by a_head, b_head, c_head entries per
// head, and row m of head h may be multiplied by sigmoid(gate[m, h]).  Rows grouped by expert: B of a row tile is that of
// expert_of_tile[first row / 128] (negative: the tile is left out).
// ------------------------------------------------------------------------------------------------
struct GemmF32 {
  const float *A, *B;
  float* C;
  long long lda, ldb, ldc;
  int M, N, K, b_kn, act;
  long long a_head, b_head, c_head;
  const float* gate;
  long long ldg;
  const int* expert_of_tile;
  int experts;
  const float* bias;          // [N], added ahead of the activation, or null
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32 p) {
  tfb::pdl_sync();
  __shared__ float sA[16][68], sB[16][68];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, h = blockIdx.z, tid = threadIdx.x;
  const int ty = tid >> 4, tx = tid & 15;
  const float *A = p.A + h * p.a_head, *B = p.B + h * p.b_head;
  float* C = p.C + h * p.c_head;
  if (p.expert_of_tile) {
    const int e = p.expert_of_tile[m0 / 128];
    if (e < 0) return;
    TFB_BOUNDS(e < p.experts, 12, e, p.experts);
    if (e >= p.experts) return;
    B += e * p.b_head;
  }
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + 256 * i, r = e >> 4, k = e & 15;
      sA[k][r] = (m0 + r < p.M && k0 + k < p.K) ? A[(long long)(m0 + r) * p.lda + k0 + k] : 0.f;
      if (p.b_kn) {
        const int kk = e >> 6, n = e & 63;
        sB[kk][n] = (n0 + n < p.N && k0 + kk < p.K) ? B[(long long)(k0 + kk) * p.ldb + n0 + n] : 0.f;
      } else {
        sB[k][r] = (n0 + r < p.N && k0 + k < p.K) ? B[(long long)(n0 + r) * p.ldb + k0 + k] : 0.f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sA[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sB[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= p.M) continue;
    const float f = p.gate ? 1.f / (1.f + expf(-p.gate[m * p.ldg + h])) : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < p.N) C[(long long)m * p.ldc + n] = act_f32(acc[i][j] + (p.bias ? p.bias[n] : 0.f), p.act) * f;
    }
  }
}

static int launch_gemm_f32(const GemmF32& p, int heads, void* stream) {
  if (p.M <= 0 || p.N <= 0 || p.K <= 0 || heads <= 0 || heads > 65535 || (p.M + 63) / 64 > 65535) return TFB_ERR_ARG;
  launch_k(gemm_f32_kernel, dim3((p.N + 63) / 64, (p.M + 63) / 64, heads), 256, 0, static_cast<cudaStream_t>(stream), p);
  return int(cudaGetLastError());
}

static bool aligned(const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }
static int grid_for(long long items) {
  const long long b = (items + 255) / 256, cap = 148ll * 16;
  return int(b < 1 ? 1 : (b < cap ? b : cap));
}

}  // namespace tfb

using bf16 = __nv_bfloat16;

// f32 = 1: activations, table and norm weights are fp32, otherwise bf16.  norm: its kind (NORM_*).  See ResNormArgs.
TFB_API int tfb_res_norm(const long long* ids, const void* table, long long ld_table, float scale, int vocab, float* x, long long ldx,
                         const void* y, long long ldy, const void* y2, long long ldy2, const void* w_post, const void* b_post,
                         const void* scale_post, const void* w_pre, const void* b_pre, void* a, long long lda, const int* rows, int n, int H,
                         float eps, int norm, int f32, void* stream) {
  using namespace tfb;
  const bool layer = norm == NORM_LAYER;
  if (n <= 0 || H <= 0 || (w_post && (!(y || ids) || (layer && !b_post))) || (w_pre && (!a || (layer && !b_pre))) || (ids && !table) || (y2 && !y) ||
      norm < 0 || norm > NORM_PLAIN)
    return TFB_ERR_ARG;
  ResNormArgs p{ids, table, ld_table, scale, vocab, x, ldx, y, ldy, y2, ldy2, w_post, b_post, scale_post, w_pre, b_pre, a, lda, rows, H, eps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int es = f32 ? 4 : 2;
  auto ok = [&](int vec) {
    for (const void* q : {w_post, b_post, scale_post, w_pre, b_pre})
      if (q && !aligned(q, vec * es)) return false;
    return H % vec == 0 && ldx % vec == 0 && aligned(x, 16) && (!y || (ldy % vec == 0 && aligned(y, vec * es))) &&
           (!y2 || (ldy2 % vec == 0 && aligned(y2, vec * es))) &&
           (!a || (lda % vec == 0 && aligned(a, vec * es))) && (!ids || (ld_table % vec == 0 && aligned(table, vec * es)));
  };
#define TFB_RN(T, VEC)                                        \
  (layer ? launch_res_norm<T, NORM_LAYER, VEC>(p, n, st)      \
         : norm == NORM_PLAIN ? launch_res_norm<T, NORM_PLAIN, VEC>(p, n, st) : launch_res_norm<T, NORM_CENTRED, VEC>(p, n, st))
  if (f32) return ok(4) ? TFB_RN(float, 4) : TFB_RN(float, 1);
  if (ok(8)) return TFB_RN(bf16, 8);
  return ok(4) ? TFB_RN(bf16, 4) : TFB_RN(bf16, 1);
#undef TFB_RN
}

TFB_API int tfb_act_rows(const void* in, long long ldi, void* out, long long ldo, int M, int N, int act, int f32, void* stream) {
  using namespace tfb;
  if (M <= 0 || N <= 0) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int grid = grid_for((long long)M * N);
  if (f32) launch_k(act_rows_kernel<float>, grid, 256, 0, st, static_cast<const float*>(in), ldi, static_cast<float*>(out), ldo, M, N, act);
  else launch_k(act_rows_kernel<bf16>, grid, 256, 0, st, static_cast<const bf16*>(in), ldi, static_cast<bf16*>(out), ldo, M, N, act);
  return int(cudaGetLastError());
}

// act, limit: see glu_value
TFB_API int tfb_glu(const void* in, long long ldi, void* out, long long ldo, int M, int F, int act, float limit, int f32, void* stream) {
  using namespace tfb;
  if (M <= 0 || F <= 0 || act < 0 || act > GLU_CLAMPED) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vec = f32 ? 4 : 8;
  const bool v = F % vec == 0 && ldi % vec == 0 && ldo % vec == 0 && aligned(in, 16) && aligned(out, 16);
  const int grid = grid_for((long long)M * (v ? F / vec : F));
#define TFB_GLU1(T, VEC, ACT) launch_k(glu_kernel<T, VEC, ACT>, grid, 256, 0, st, static_cast<const T*>(in), ldi, static_cast<T*>(out), ldo, M, F, limit)
#define TFB_GLU(T, VEC)                                   \
  do {                                                    \
    if (act == GLU_CLAMPED) TFB_GLU1(T, VEC, GLU_CLAMPED); \
    else if (act == GLU_GELU) TFB_GLU1(T, VEC, GLU_GELU); \
    else TFB_GLU1(T, VEC, GLU_SILU);                      \
  } while (0)
  if (f32) { if (v) TFB_GLU(float, 4); else TFB_GLU(float, 1); }
  else { if (v) TFB_GLU(bf16, 8); else TFB_GLU(bf16, 1); }
#undef TFB_GLU
#undef TFB_GLU1
  return int(cudaGetLastError());
}

// o [rows, H, V] fp32; gate [rows, ldg] and w [V] may be null
TFB_API int tfb_gated_norm(const float* o, const void* gate, long long ldg, const void* w, void* out, long long ldo, int rows, int H, int V,
                           float eps, int f32, void* stream) {
  using namespace tfb;
  if (rows <= 0 || H <= 0 || V <= 0) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long blocks = ((long long)rows * H + 7) / 8;
  const int grid = int(blocks < 148ll * 32 ? blocks : 148ll * 32);
  auto al = [](const void* x, int n) { return (reinterpret_cast<uintptr_t>(x) & (n - 1)) == 0; };
  const int es = f32 ? 4 : 2;
  const bool v4 = V % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && al(o, 16) && (!gate || al(gate, 4 * es)) && (!w || al(w, 4 * es)) && al(out, 4 * es);
#define TFB_GN(T, VEC) launch_k(gated_norm_kernel<T, VEC>, grid, 256, 0, st, o, static_cast<const T*>(gate), ldg, static_cast<const T*>(w), \
                                static_cast<T*>(out), ldo, rows, H, V, eps)
  if (f32) { if (v4) TFB_GN(float, 4); else TFB_GN(float, 1); }
  else { if (v4) TFB_GN(bf16, 4); else TFB_GN(bf16, 1); }
#undef TFB_GN
  return int(cudaGetLastError());
}

// As tfb_rope_append behind an RMS norm (weights wq, wk of D entries, or none) of every q and k head; qf: a factor per query head, or
// null; dims may be 0.
TFB_API int tfb_norm_rope_append(void* qkv, long long ld, const void* wq, const void* wk, const void* qf, float eps, const float* cos_t, const float* sin_t,
                                 int max_pos, const int* positions, const long long* slots, void* kpool, void* vpool, long long nslots, int rows,
                                 int nq, int nk, int D, int dims, int v_cols, int f32, void* stream) {
  using namespace tfb;
  if (rows <= 0 || nq <= 0 || nk <= 0 || D <= 0 || dims < 0 || (dims & 1) || dims > D || (dims && (!cos_t || !sin_t || max_pos <= 0)) || !wq != !wk)
    return TFB_ERR_ARG;
  if (nslots == 0) slots = nullptr;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool v = dims % 8 == 0 && D % 8 == 0 && D <= 256 && v_cols % 8 == 0 && ld % (f32 ? 4 : 8) == 0 && aligned(qkv, 16) && aligned(wq, 16) &&
                 aligned(wk, 16) && (!slots || (aligned(kpool, 16) && aligned(vpool, 16)));
  const int L = !v ? 32 : D <= 64 ? 8 : D <= 128 ? 16 : 32, piece = v ? 8 * L : 64;
  const int units = nq + nk + (v_cols + piece - 1) / piece;
  const long long blocks = ((long long)rows * (v ? (units + NRA_UNITS - 1) / NRA_UNITS : units) * L + 255) / 256;
  if (blocks * 256 > 0x7fffffffll) return TFB_ERR_LIMIT;
#define TFB_NRA(KERN, T) launch_k(KERN, int(blocks), 256, 0, st, static_cast<T*>(qkv), ld, static_cast<const T*>(wq), static_cast<const T*>(wk), static_cast<const T*>(qf), eps, \
                                  cos_t, sin_t, max_pos, positions, slots, static_cast<T*>(kpool), static_cast<T*>(vpool), nslots, rows, nq, nk, D, \
                                  dims, v_cols)
#define TFB_NRL(T)                                                          \
  if (!v) TFB_NRA(norm_rope_append_any_kernel<T>, T);                       \
  else if (L == 8) TFB_NRA((norm_rope_append_kernel<T, 8>), T);             \
  else if (L == 16) TFB_NRA((norm_rope_append_kernel<T, 16>), T);           \
  else TFB_NRA((norm_rope_append_kernel<T, 32>), T);
  if (f32) { TFB_NRL(float) } else { TFB_NRL(bf16) }
#undef TFB_NRL
#undef TFB_NRA
  return int(cudaGetLastError());
}

TFB_API int tfb_rope_append(void* qkv, long long ld, const float* cos_t, const float* sin_t, int max_pos, const int* positions,
                            const long long* slots, void* kpool, void* vpool, long long nslots, int rows, int nq, int nk, int D, int dims,
                            int v_cols, int f32, void* stream) {
  using namespace tfb;
  if (rows <= 0 || nq <= 0 || nk < 0 || dims < 0 || (dims & 1) || dims > D) return TFB_ERR_ARG;
  if (nk == 0) v_cols = 0;
  if (dims == 0 && (nk == 0 || !slots || nslots == 0)) return 0;      // nothing to rotate, nothing to keep
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vec = f32 ? 4 : 8;
  const bool v = (dims / 2) % vec == 0 && D % vec == 0 && v_cols % vec == 0 && ld % vec == 0 && aligned(qkv, 16) &&
                 (!kpool || (aligned(kpool, 16) && aligned(vpool, 16)));
  const int q = v ? vec : 1;
  const int grid = grid_for((long long)rows * ((nq + nk) * (dims / 2 / q) + nk * ((D - dims) / q) + v_cols / q));
#define TFB_RA(T, VEC) launch_k(rope_append_kernel<T, VEC>, grid, 256, 0, st, static_cast<T*>(qkv), ld, cos_t, sin_t, max_pos, positions, \
                                slots, static_cast<T*>(kpool), static_cast<T*>(vpool), nslots, rows, nq, nk, D, dims, v_cols)
  if (f32) { if (v) TFB_RA(float, 4); else TFB_RA(float, 1); }
  else { if (v) TFB_RA(bf16, 8); else TFB_RA(bf16, 1); }
#undef TFB_RA
  return int(cudaGetLastError());
}

TFB_API int tfb_gather_rows(const void* pool, long long nslots, const int* pages, int page, int lo, int n, void* out, int width, int f32,
                            void* stream) {
  using namespace tfb;
  if (n <= 0 || width <= 0 || lo < 0 || page <= 0) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vec = f32 ? 4 : 8;
  const bool v = width % vec == 0 && aligned(pool, 16) && aligned(out, 16);
  const int grid = grid_for((long long)n * (v ? width / vec : width));
#define TFB_GR(T, VEC) launch_k(gather_rows_kernel<T, VEC>, grid, 256, 0, st, static_cast<const T*>(pool), nslots, pages, page, lo, n, \
                                static_cast<T*>(out), width)
  if (f32) { if (v) TFB_GR(float, 4); else TFB_GR(float, 1); }
  else { if (v) TFB_GR(bf16, 8); else TFB_GR(bf16, 1); }
#undef TFB_GR
  return int(cudaGetLastError());
}

TFB_API int tfb_gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc, int M, int N, int K, int act,
                         const float* bias, void* stream) {
  using namespace tfb;
  return launch_gemm_f32(GemmF32{A, B, C, lda, ldb, ldc, M, N, K, 0, act, 0, 0, 0, nullptr, 0, nullptr, 0, bias}, 1, stream);
}

// One product per head: C[:, h * c_head ...] = A[:, h * a_head ...] . B_h^T (B_h: N rows of B, or K rows with b_kn) * sigmoid(gate[:, h]).
TFB_API int tfb_gemm_f32_heads(const float* A, long long lda, int a_head, const float* B, long long ldb, int b_kn, float* C, long long ldc, int c_head,
                               const float* gate, long long ldg, int M, int heads, int N, int K, void* stream) {
  using namespace tfb;
  return launch_gemm_f32(GemmF32{A, B, C, lda, ldb, ldc, M, N, K, b_kn, 0, a_head, (long long)(b_kn ? K : N) * ldb, c_head, gate, ldg, nullptr, 0, nullptr},
                         heads, stream);
}

// Rows grouped by expert (M: rows of the expert buffers), B [experts][N][K] with `stride` entries between experts.
TFB_API int tfb_moe_gemm_f32(const float* A, long long lda, const float* B, long long ldb, long long stride, float* C, long long ldc,
                             const int* expert_of_tile, int experts, int M, int N, int K, void* stream) {
  using namespace tfb;
  if (!expert_of_tile || experts <= 0) return TFB_ERR_ARG;
  return launch_gemm_f32(GemmF32{A, B, C, lda, ldb, ldc, M, N, K, 0, 0, 0, stride, 0, nullptr, 0, expert_of_tile, experts, nullptr}, 1, stream);
}
