// Kernels of composed stacks (fp32 residual stream, grouped output norms, HGRN2 recurrence, latent attention).
//
// This file is compiled WITHOUT fast-math: the 32-bit mode of the engine uses the same kernels, and what a composed
// stack computes in fp32 (norms, gates, recurrence, softmax) must be correctly rounded fp32 there.  Where the 16-bit
// mode can afford the hardware approximations (relative error around 1e-6) the code asks for them by intrinsic.
//
//  * embed_rows     token rows -> fp32 residual stream and its 16-bit copy
//  * norm_add       residual += group norm of a sublayer's output; writes the next sublayer's input (or its final norm); one form
//                  first sums the weighted rows of a token's experts, one starts the stream with normed embeddings
//  * sum_norm       residual = norm(alpha residual + a sublayer's output, weighted expert rows included); writes the next sublayer's input
//                  (or its final norm)
//  * hgrn2_step     one token per sequence: gates, state update, read-out and per-head norm in one pass over the state
//                  (and the same for linear attention whose rows decay by gates of their own, here and in hgrn2_scan)
//  * hgrn2_scan     segments of any length: the state stays in registers while the tokens stream through shared memory
//  * latent_write   norm of the latent projection, scattered into the paged latent cache, with the rotation of the part of queries and
//                  rows that carries positions
//  * latent_attn    CUDA-core attention over paged latent rows (any sizes, fp32 or bf16)
//  * glu, gate_outputs, and a CUDA-core GEMM for fp32 and for shapes that no tensor-core kernel takes
#include "stack_common.cuh"

namespace rb {
namespace stack {

// ------------------------------------------------------------------------------------------------- embedding
template <typename T>
__global__ void embed_rows_kernel(const long long* __restrict__ tok, const T* __restrict__ w, float* __restrict__ res,
                                  T* __restrict__ h, int vocab, int pitch, float scale) {
  const long long t = blockIdx.x;
  const long long id = tok[t];
  const bool ok = id >= 0 && id < vocab;
  for (int c = threadIdx.x * 8; c < pitch; c += blockDim.x * 8) {
    F8 v;
#pragma unroll
    for (int i = 0; i < 8; ++i) v.v[i] = 0.f;
    if (ok) v = ld8(w + id * pitch + c);
#pragma unroll
    for (int i = 0; i < 8; ++i) v.v[i] *= scale;
    st8(res + t * pitch + c, v);
    st8(h + t * pitch + c, v);
  }
}

// ------------------------------------------------------------------------------------------------- group norm + add
// One CTA per row.  `parts` consecutive sets of warps own one group at a time (wpg warps per group), so groups are
// reduced side by side; sums of the warps of a group meet in shared memory.
constexpr int NA_WARPS = 8;
template <typename T, bool kSum> struct YType { typedef T type; };
template <typename T> struct YType<T, true> { typedef float type; };
struct NormAddParams {
  float* res;             // [rows][pitch] fp32, updated in place
  const void* y;          // [rows][ldy]
  const void* w;          // [pitch] weight of the output norm
  const void* next_w;     // [pitch] or null
  void* h;                // [rows][pitch]
  int ldy, pitch, width, groups, wpg;
  float eps;
  // NA_EMBED: y is the embedding table, row `tok[row]` of it is normed, and the stream starts with the result
  const long long* tok;
  int vocab;
  // NA_SUM: y (or nothing, when null) plus the weighted rows of `top` experts per row; ex [sorted rows][ldy], row of a
  // choice = offset[expert] + place
  const void* ex;
  const int* expert;      // [rows][top]
  const int* place;       // [rows][top]
  const int* offset;      // [experts + 1]
  const float* weight;    // [rows][top]
  int top, experts;       // choices from `experts` on are identity experts: their output is the stream itself
};
enum : int { NA_PLAIN = 0, NA_EMBED = 1, NA_SUM = 2 };
constexpr int NA_MAX_TOP = 64;

// Where the rows of a token's experts lie (shared memory, filled by the whole CTA).
template <int MAX>
struct ExpertRows {
  long long at[MAX];      // first element of a choice's row, -1: identity expert
  float w[MAX];
  // returns whether the token took identity experts
  __device__ __forceinline__ bool gather(const int* expert, const int* place, const int* offset, const float* weight, long long row, int n, int experts,
                                          int pitch) {
    bool identity = false;
    if (static_cast<int>(threadIdx.x) < n) {
      const long long i = row * n + threadIdx.x;
      const int e = expert[i];
      identity = e >= experts;
      at[threadIdx.x] = identity ? -1 : (static_cast<long long>(offset[e]) + place[i]) * pitch;
      w[threadIdx.x] = weight[i];
    }
    return __syncthreads_or(identity) != 0;
  }
  // sum of the identity experts' weights
  __device__ __forceinline__ float identity(int n) const {
    float s = 0.f;
    for (int k = 0; k < n; ++k) s += at[k] < 0 ? w[k] : 0.f;
    return s;
  }
  template <int V, bool kIdentity, typename T>
  __device__ __forceinline__ void add(const T* ex, int n, float* a) const {
#pragma unroll 4
    for (int k = 0; k < n; ++k) {
      float b[V];
      const long long i = at[k];
      if constexpr (kIdentity) {
#pragma unroll
        for (int j = 0; j < V; ++j) b[j] = 0.f;
        if (i >= 0) ldv<V>(ex + i, b);
      } else {
        ldv<V>(ex + i, b);
      }
      const float f = w[k];
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] += f * b[j];
    }
  }
};
template <typename T, int V, int MODE>
__global__ void __launch_bounds__(NA_WARPS * 32) norm_add_kernel(const NormAddParams p) {
  __shared__ float red[2][NA_WARPS];
  extern __shared__ __align__(16) float ysum[];      // [width] (NA_SUM)
  const long long row = blockIdx.x;
  using Y = typename YType<T, MODE == NA_SUM>::type;
  const Y* y;
  bool known = true;
  if constexpr (MODE == NA_SUM) {
    __shared__ ExpertRows<NA_MAX_TOP> s;
    const bool some = s.gather(p.expert, p.place, p.offset, p.weight, row, p.top, p.experts, p.ldy);
    const float identity = some ? s.identity(p.top) : 0.f;
    const float* stream = p.res + row * p.pitch;
    const T* base = p.y ? static_cast<const T*>(p.y) + row * p.ldy : nullptr;
    const T* ex = static_cast<const T*>(p.ex);
    for (int c = threadIdx.x * V; c < p.width; c += NA_WARPS * 32 * V) {
      float a[V], x[V];
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] = 0.f;
      if (base) ldv<V>(base + c, a);
      if (some) {
        s.add<V, true>(ex + c, p.top, a);
        ldv<V>(stream + c, x);
#pragma unroll
        for (int i = 0; i < V; ++i) a[i] += identity * x[i];
      } else {
        s.add<V, false>(ex + c, p.top, a);
      }
      stv<V>(ysum + c, a);
    }
    __syncthreads();
    y = ysum;
  } else if constexpr (MODE == NA_EMBED) {
    const long long id = p.tok[row];
    known = id >= 0 && id < p.vocab;
    y = static_cast<const T*>(p.y) + (known ? id : 0) * p.ldy;
  } else {
    y = static_cast<const T*>(p.y) + row * p.ldy;
  }
  const T* w = static_cast<const T*>(p.w);
  const T* nw = static_cast<const T*>(p.next_w);
  float* res = p.res + row * p.pitch;
  T* h = static_cast<T*>(p.h) + row * p.pitch;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int part = p.width / p.groups, wpg = p.wpg, lanes = wpg * 32;
  const int sets = NA_WARPS / wpg, set = warp / wpg, first = set * wpg;
  const int l = (warp - first) * 32 + lane;
  const float inv_n = 1.f / part;
  for (int g0 = 0; g0 < p.groups; g0 += sets) {
    const int g = g0 + set;
    const bool live = g < p.groups;
    const int lo = g * part, hi = live ? lo + part : lo;
    float ss = 0.f;
    for (int c = lo + l * V; c < hi; c += lanes * V) {
      float a[V];
      ldv<V>(y + c, a);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += a[i] * a[i];
    }
    ss = wsum(ss);
    if (wpg > 1) {
      if (lane == 0) red[0][warp] = ss;
      __syncthreads();
      ss = 0.f;
      for (int k = 0; k < wpg; ++k) ss += red[0][first + k];
    }
    const float r = known ? 1.f / sqrtf(ss * inv_n + p.eps) : 0.f;
    float s2 = 0.f;
    for (int c = lo + l * V; c < hi; c += lanes * V) {
      float a[V], b[V], x[V];
      ldv<V>(y + c, a);
      ldv<V>(w + c, b);
      if constexpr (MODE == NA_EMBED) {
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] = 0.f;
      } else {
        ldv<V>(res + c, x);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) {
        x[i] += a[i] * r * b[i];
        s2 += x[i] * x[i];
      }
      stv<V>(res + c, x);
      if (!nw) stv<V>(h + c, x);
    }
    if (nw) {      // the same thread wrote these columns of the stream: no hand-over is needed
      s2 = wsum(s2);
      if (wpg > 1) {
        if (lane == 0) red[1][warp] = s2;
        __syncthreads();
        s2 = 0.f;
        for (int k = 0; k < wpg; ++k) s2 += red[1][first + k];
      }
      const float r2 = 1.f / sqrtf(s2 * inv_n + p.eps);
      for (int c = lo + l * V; c < hi; c += lanes * V) {
        float b[V], x[V];
        ldv<V>(nw + c, b);
        ldv<V>(res + c, x);
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] = x[i] * r2 * b[i];
        stv<V>(h + c, x);
      }
    }
    if (wpg > 1) __syncthreads();      // the next pass rewrites the sums
  }
  for (int c = p.width + threadIdx.x; c < p.pitch; c += blockDim.x) {
    st(h + c, 0.f);
    if constexpr (MODE == NA_EMBED) st(res + c, 0.f);
  }
}

// ------------------------------------------------------------------------------------------------- norm of the sum
// x <- norm(alpha x + y + weighted expert rows) over the whole width.  One CTA per row; the row waits in shared memory between the
// passes, and every thread reads back only what it wrote itself.  Variances are means of squared deviations.
struct SumNormParams {
  float* res;             // [rows][pitch] fp32, updated in place
  const void* y;          // [rows][ldy] or null
  const void* ex;         // weighted expert rows as in NormAddParams, or null
  const int* expert;
  const int* place;
  const int* offset;
  const float* weight;
  int top, experts;
  const void* w;          // [pitch]
  const void* b;          // [pitch] or null
  const void* next_w;     // [pitch] or null: h is the stream itself
  const void* next_b;     // [pitch] or null
  void* h;                // [rows][pitch]
  int ldy, pitch, width, centre;
  float alpha, eps, scale;      // scale: factor on h when next_w is given
};
template <typename T, int V, bool kExperts>
__global__ void __launch_bounds__(NA_WARPS * 32) sum_norm_kernel(const SumNormParams p) {
  extern __shared__ __align__(16) float z[];      // [width]
  __shared__ float red[4][NA_WARPS];
  const long long row = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, step = NA_WARPS * 32 * V;
  float* res = p.res + row * p.pitch;
  const T* y = p.y ? static_cast<const T*>(p.y) + row * p.ldy : nullptr;
  const T* ex = static_cast<const T*>(p.ex);
  __shared__ ExpertRows<kExperts ? NA_MAX_TOP : 1> rows;
  float alpha = p.alpha;
  bool some = false;
  if constexpr (kExperts) {
    some = rows.gather(p.expert, p.place, p.offset, p.weight, row, p.top, p.experts, p.ldy);
    if (some) alpha += rows.identity(p.top);      // their output is the stream
  }
  auto total = [&](float v, int k) {      // over the CTA; every k is used once
    v = wsum(v);
    if (lane == 0) red[k][warp] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NA_WARPS; ++i) s += red[k][i];
    return s;
  };
  float sum = 0.f;
  for (int c = threadIdx.x * V; c < p.width; c += step) {
    float x[V], a[V];
    ldv<V>(res + c, x);
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] *= alpha;
    if (y) {
      ldv<V>(y + c, a);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] += a[i];
    }
    if constexpr (kExperts) {
      if (some) rows.template add<V, true>(ex + c, p.top, x);
      else rows.template add<V, false>(ex + c, p.top, x);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) sum += x[i];
    stv<V>(z + c, x);
  }
  const float inv_n = 1.f / p.width;
  float mean = p.centre ? total(sum, 0) * inv_n : 0.f;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < p.width; c += step) {
    float x[V];
    ldv<V>(z + c, x);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += (x[i] - mean) * (x[i] - mean);
  }
  float r = 1.f / sqrtf(total(ss, 1) * inv_n + p.eps);
  const T* w = static_cast<const T*>(p.w);
  const T* b = static_cast<const T*>(p.b);
  const T* nw = static_cast<const T*>(p.next_w);
  const T* nb = static_cast<const T*>(p.next_b);
  T* h = static_cast<T*>(p.h) + row * p.pitch;
  sum = 0.f;
  for (int c = threadIdx.x * V; c < p.width; c += step) {
    float x[V], f[V], g[V];
    ldv<V>(z + c, x);
    ldv<V>(w + c, f);
    if (b) ldv<V>(b + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      x[i] = (x[i] - mean) * r * f[i];
      if (b) x[i] += g[i];
      sum += x[i];
    }
    stv<V>(res + c, x);
    if (nw) stv<V>(z + c, x);
    else stv<V>(h + c, x);
  }
  if (nw) {
    mean = p.centre ? total(sum, 2) * inv_n : 0.f;
    ss = 0.f;
    for (int c = threadIdx.x * V; c < p.width; c += step) {
      float x[V];
      ldv<V>(z + c, x);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += (x[i] - mean) * (x[i] - mean);
    }
    r = 1.f / sqrtf(total(ss, 3) * inv_n + p.eps);
    for (int c = threadIdx.x * V; c < p.width; c += step) {
      float x[V], f[V], g[V];
      ldv<V>(z + c, x);
      ldv<V>(nw + c, f);
      if (nb) ldv<V>(nb + c, g);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        x[i] = (x[i] - mean) * r * f[i];
        if (nb) x[i] += g[i];
        x[i] *= p.scale;
      }
      stv<V>(h + c, x);
    }
  }
  for (int c = p.width + threadIdx.x; c < p.pitch; c += blockDim.x) st(h + c, 0.f);
}

// ------------------------------------------------------------------------------------------------- HGRN2
struct HgrnParams {
  const void* qfv;        // [T][ld]: q (H*dim) | f (H*dim) | v (H*vdim), raw projections
  const void* f_bias;     // [H*dim]
  const void* lower;      // [H*dim]
  const void* norm_w;     // [vdim]
  float* state;           // [slots][H][dim][vp]
  const int* slot;        // [S]
  const int* ctx;         // [S] tokens of the sequence including this segment
  const int* cu;          // [S + 1] (scan only)
  float* o_raw;           // [T][H][vdim] (scan only)
  void* out;              // [T][ldo]
  int H, dim, vdim, vp, ld, ldo;
  float eps;
  // kGla (linear attention with decaying rows): qfv is q (H*dim) | k (H*dim) | v (H*vdim) and, from column gate_col on, output gates
  // (H*vdim); f_bias joins z, and a row decays by sigmoid(z) ^ inv_root
  const float* z;         // [T][ldz]
  int ldz, gate_col;
  float q_scale, inv_root;
};
// sigmoid(z) ^ r from its logarithm, min(z, 0) - log(1 + exp(-|z|))
__device__ __forceinline__ float decay(float z, float r) { return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * r); }

// One new token per sequence.  CTA = (sequence, head); a thread owns four value columns of every ng-th state row, so a
// warp reads and writes whole rows; eight rows per thread are in flight at a time.
constexpr int HS_THREADS = 256;
template <typename T, bool kGla>
__global__ void __launch_bounds__(HS_THREADS) hgrn2_step_kernel(const HgrnParams p) {
  constexpr bool kExact = IsExact<T>::v;
  extern __shared__ __align__(16) float sm[];
  const int dp = (p.dim + 3) & ~3;      // the rows behind are read four values at a time
  float* sq = sm;                       // [dim]
  float* sg = sq + dp;                  // [dim] forget gate
  float* sk = sg + dp;                  // [dim] 1 - gate
  float* sv = sk + dp;                  // [vp]
  float* red = sv + p.vp;               // [ng][vp]
  __shared__ float wred[HS_THREADS / 32];
  const int s = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x;
  const T* row = static_cast<const T*>(p.qfv) + static_cast<long long>(s) * p.ld;
  const int qd = p.H * p.dim;
  for (int d = tid; d < p.dim; d += HS_THREADS) {
    const int c = hd * p.dim + d;
    if constexpr (kGla) {
      sq[d] = ld(row + c) * p.q_scale;
      sk[d] = ld(row + qd + c);
      sg[d] = decay(p.z[static_cast<long long>(s) * p.ldz + c] + ld(static_cast<const T*>(p.f_bias) + c), p.inv_root);
      continue;
    }
    const float q = ld(row + c), f = ld(row + qd + c) + ld(static_cast<const T*>(p.f_bias) + c);
    const float lo = ld(static_cast<const T*>(p.lower) + c);
    const float sf = sigmoid<kExact>(f), sn = sigmoid<kExact>(-f);
    sq[d] = q * sigmoid<kExact>(q);
    sg[d] = lo + (1.f - lo) * sf;
    sk[d] = (1.f - lo) * sn;             // = 1 - gate without the cancellation
  }
  for (int j = tid; j < p.vp; j += HS_THREADS) sv[j] = j < p.vdim ? ld(row + 2 * qd + hd * p.vdim + j) : 0.f;
  __syncthreads();
  const int lpr = p.vp >> 2, ng = HS_THREADS / lpr;
  const int g = tid / lpr, c4 = (tid - g * lpr) * 4;
  const bool fresh = p.ctx[s] == 1;
  if (g < ng) {
    float* S = p.state + ((static_cast<long long>(p.slot[s]) * p.H + hd) * p.dim) * p.vp + c4;
    const float4 v = *reinterpret_cast<const float4*>(sv + c4);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    constexpr int U = 8;
    for (int d0 = g; d0 < p.dim; d0 += ng * U) {
      float4 x[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int d = d0 + u * ng;
        x[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d < p.dim && !fresh) x[u] = __ldcs(reinterpret_cast<const float4*>(S + static_cast<long long>(d) * p.vp));
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int d = d0 + u * ng;
        if (d < p.dim) {
          const float f = sg[d], k = sk[d], q = sq[d];
          x[u].x = f * x[u].x + k * v.x;
          x[u].y = f * x[u].y + k * v.y;
          x[u].z = f * x[u].z + k * v.z;
          x[u].w = f * x[u].w + k * v.w;
          __stcs(reinterpret_cast<float4*>(S + static_cast<long long>(d) * p.vp), x[u]);
          acc.x += q * x[u].x;
          acc.y += q * x[u].y;
          acc.z += q * x[u].z;
          acc.w += q * x[u].w;
        }
      }
    }
    *reinterpret_cast<float4*>(red + g * p.vp + c4) = acc;
  }
  __syncthreads();
  float ss = 0.f;
  for (int j = tid; j < p.vdim; j += HS_THREADS) {
    float o = 0.f;
    for (int k = 0; k < ng; ++k) o += red[k * p.vp + j];
    red[j] = o;                          // column j of group 0 is read by this thread only
    ss += o * o;
  }
  ss = wsum(ss);
  if ((tid & 31) == 0) wred[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int k = 0; k < HS_THREADS / 32; ++k) ss += wred[k];
  const float r = 1.f / sqrtf(ss / p.vdim + p.eps);
  T* out = static_cast<T*>(p.out) + static_cast<long long>(s) * p.ldo;
  for (int j = tid; j < p.vdim; j += HS_THREADS) {
    float o = red[j] * r * ld(static_cast<const T*>(p.norm_w) + j);
    if constexpr (kGla) {
      const float g = ld(row + p.gate_col + hd * p.vdim + j);
      o *= g * sigmoid<kExact>(g);
    }
    st(out + hd * p.vdim + j, o);
  }
  if (hd == p.H - 1)
    for (int j = p.H * p.vdim + tid; j < p.ldo; j += HS_THREADS) st(out + j, 0.f);
}

// Segments of any length.  CTA = (segment, head, 32 value columns); thread (group, lane) keeps an 8 x 4 block of the
// state in registers as pairs along the rows (packed fp32 pair arithmetic).  Tokens come in chunks: while one chunk is
// processed the next one's raw projections are on their way into registers; the gates are computed once per chunk.  The
// read-outs of a chunk are partial sums per row group, added up once per chunk.
constexpr int SC_V = 32;            // value columns per CTA
constexpr int SC_CH = 16;           // tokens per chunk
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b) {
  unsigned long long d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
union Pair {
  unsigned long long u;
  float2 f;
};
template <typename T> struct Raw8 { uint4 u[sizeof(T) / 2]; };
template <typename T>
__device__ __forceinline__ float raw_get(const Raw8<T>& r, int i) {
  if constexpr (sizeof(T) == 4) return reinterpret_cast<const float*>(&r)[i];
  else {
    const uint32_t w = reinterpret_cast<const uint32_t*>(&r)[i >> 1];
    return __uint_as_float((i & 1) ? (w & 0xffff0000u) : (w << 16));
  }
}
template <typename T, bool kVec>
__device__ __forceinline__ Raw8<T> raw_load(const T* p, int valid) {      // `valid` elements of eight, the others zero
  Raw8<T> r;
#pragma unroll
  for (int i = 0; i < static_cast<int>(sizeof(T) / 2); ++i) r.u[i] = make_uint4(0, 0, 0, 0);
  if constexpr (kVec) {
    if (valid >= 8) {
#pragma unroll
      for (int i = 0; i < static_cast<int>(sizeof(T) / 2); ++i) r.u[i] = __ldg(reinterpret_cast<const uint4*>(p) + i);
    }
  } else {
    T* e = reinterpret_cast<T*>(&r);
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < valid) e[i] = p[i];
  }
  return r;
}

template <typename T, bool kVec, bool kGla>
__global__ void __launch_bounds__(512) hgrn2_scan_kernel(const HgrnParams p, int NG) {
  constexpr bool kExact = IsExact<T>::v;
  extern __shared__ __align__(16) float sm[];
  const int DP = NG * 8;
  float* sg = sm;                               // [CH][DP] forget gate
  float* sk = sg + SC_CH * DP;                  // [CH][DP] 1 - gate
  float* sq = sk + SC_CH * DP;                  // [CH][DP]
  float* sv = sq + SC_CH * DP;                  // [CH][2 * V]: every value twice
  float* part = sv + SC_CH * 2 * SC_V;          // [CH][NG][V]
  const int seg = blockIdx.x, hd = blockIdx.y, v0 = blockIdx.z * SC_V;
  const int tid = threadIdx.x, nthr = blockDim.x;       // nthr = NG * 8
  const int g = tid >> 3, c4 = (tid & 7) * 4;
  const int lo = p.cu[seg], hi = p.cu[seg + 1];
  const int qd = p.H * p.dim;
  const int nv = min(SC_V, p.vdim - v0);
  const T* base = static_cast<const T*>(p.qfv);
  float* S = p.state + ((static_cast<long long>(p.slot[seg]) * p.H + hd) * p.dim) * p.vp + v0 + c4;
  const bool fresh = p.ctx[seg] == hi - lo;
  const bool cols = v0 + c4 < p.vp;
  Pair x[4][4];                                 // [row pair][column]
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int d = g * 8 + r * 2 + e;
      float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && d < p.dim && cols) t = *reinterpret_cast<const float4*>(S + static_cast<long long>(d) * p.vp);
      const float* tf = reinterpret_cast<const float*>(&t);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        if (e == 0) x[r][c].f.x = tf[c];
        else x[r][c].f.y = tf[c];
      }
    }
  // raw data of the next chunk: this thread prepares features dpre .. dpre + 7 of the tokens tpre and tpre + 8
  const int tpre = tid / NG, dpre = (tid - tpre * NG) * 8;
  Raw8<T> rq[2], rf[2], rv;
  Raw8<float> rz[kGla ? 2 : 1];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int t = tpre + 8 * k;
      const int valid = t0 + t < hi ? p.dim - dpre : 0;
      const T* a = base + static_cast<long long>(t0 + t) * p.ld + hd * p.dim + dpre;
      rq[k] = raw_load<T, kVec>(a, valid);
      rf[k] = raw_load<T, kVec>(a + qd, valid);
      if constexpr (kGla) rz[k] = raw_load<float, kVec>(p.z + static_cast<long long>(t0 + t) * p.ldz + hd * p.dim + dpre, valid);
    }
    if (tid < SC_CH * 4) {
      const int t = tid >> 2, j = (tid & 3) * 8;
      rv = raw_load<T, kVec>(base + static_cast<long long>(t0 + t) * p.ld + 2 * qd + hd * p.vdim + v0 + j, t0 + t < hi ? nv - j : 0);
    }
  };
  float fb[8], fl[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const bool in = dpre + i < p.dim;
    fb[i] = in ? ld(static_cast<const T*>(p.f_bias) + hd * p.dim + dpre + i) : 0.f;
    if constexpr (!kGla) fl[i] = in ? ld(static_cast<const T*>(p.lower) + hd * p.dim + dpre + i) : 1.f;       // padding rows: 1 - gate = 0
  }
  fetch(lo);
  for (int t0 = lo; t0 < hi; t0 += SC_CH) {
    const int n = min(SC_CH, hi - t0);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int t = tpre + 8 * k;
      F8 a, b, c;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float q = raw_get<T>(rq[k], i), f = raw_get<T>(rf[k], i) + fb[i];
        if constexpr (kGla) {      // padding rows: k = 0
          a.v[i] = decay(raw_get<float>(rz[k], i) + fb[i], p.inv_root);
          b.v[i] = raw_get<T>(rf[k], i);
          c.v[i] = q * p.q_scale;
          continue;
        }
        if constexpr (kExact) {
          a.v[i] = fl[i] + (1.f - fl[i]) * sigmoid<true>(f);
          b.v[i] = (1.f - fl[i]) * sigmoid<true>(-f);
        } else {      // one exponential of -|f|: both halves of the gate without overflow or cancellation
          const float e = __expf(-fabsf(f)), r = __fdividef(1.f, 1.f + e), er = e * r;
          a.v[i] = fl[i] + (1.f - fl[i]) * (f >= 0.f ? r : er);
          b.v[i] = (1.f - fl[i]) * (f >= 0.f ? er : r);
        }
        c.v[i] = q * sigmoid<kExact>(q);
      }
      st8(sg + t * DP + dpre, a);
      st8(sk + t * DP + dpre, b);
      st8(sq + t * DP + dpre, c);
    }
    if (tid < SC_CH * 4) {
      float* d = sv + (tid >> 2) * 2 * SC_V + (tid & 3) * 16;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float v = raw_get<T>(rv, i);
        d[2 * i] = v;
        d[2 * i + 1] = v;
      }
    }
    __syncthreads();
    if (t0 + SC_CH < hi) fetch(t0 + SC_CH);
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
      const ulonglong2* G = reinterpret_cast<const ulonglong2*>(sg + t * DP + g * 8);
      const ulonglong2* K = reinterpret_cast<const ulonglong2*>(sk + t * DP + g * 8);
      const ulonglong2* Q = reinterpret_cast<const ulonglong2*>(sq + t * DP + g * 8);
      const ulonglong2* V = reinterpret_cast<const ulonglong2*>(sv + t * 2 * SC_V + c4 * 2);
      const ulonglong2 g0 = G[0], g1 = G[1], k0 = K[0], k1 = K[1], q0 = Q[0], q1 = Q[1], va = V[0], vb = V[1];
      const unsigned long long gg[4] = {g0.x, g0.y, g1.x, g1.y}, kk[4] = {k0.x, k0.y, k1.x, k1.y};
      const unsigned long long qq[4] = {q0.x, q0.y, q1.x, q1.y}, vv[4] = {va.x, va.y, vb.x, vb.y};
      float4 o;
      float* of = reinterpret_cast<float*>(&o);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        Pair acc;
        acc.u = 0ull;
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          x[r][c].u = fma2(gg[r], x[r][c].u, mul2(kk[r], vv[c]));
          acc.u = fma2(qq[r], x[r][c].u, acc.u);
        }
        of[c] = acc.f.x + acc.f.y;
      }
      *reinterpret_cast<float4*>(part + (t * NG + g) * SC_V + c4) = o;
    }
    __syncthreads();
    for (int i = tid; i < n * (SC_V / 4); i += nthr) {      // four columns of one token
      const int t = i >> 3, j = (i & 7) * 4;
      const float4* a = reinterpret_cast<const float4*>(part + t * NG * SC_V + j);
      float4 o = a[0];
#pragma unroll 4
      for (int k = 1; k < NG; ++k) {
        const float4 b = a[k * (SC_V / 4)];
        o.x += b.x; o.y += b.y; o.z += b.z; o.w += b.w;
      }
      float* d = p.o_raw + (static_cast<long long>(t0 + t) * p.H + hd) * p.vdim + v0 + j;
      if (p.vdim % 4 == 0) {
        if (j < nv) *reinterpret_cast<float4*>(d) = o;
      } else {
        const float of[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (j + c < nv) d[c] = of[c];
      }
    }
  }
  if (cols) {
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = g * 8 + r * 2 + e;
        float4 t;
        float* tf = reinterpret_cast<float*>(&t);
#pragma unroll
        for (int c = 0; c < 4; ++c) tf[c] = e == 0 ? x[r][c].f.x : x[r][c].f.y;
        if (d < p.dim) *reinterpret_cast<float4*>(S + static_cast<long long>(d) * p.vp) = t;
      }
  }
}

// per-head RMS norm of the scan's read-outs, times silu of a gate per feature when given; one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) head_norm_kernel(const float* __restrict__ o_raw, const T* __restrict__ w, T* __restrict__ out,
                                                        const T* __restrict__ gate, int ld_gate, long long units, int H, int vdim, int ldo, float eps) {
  constexpr bool kExact = IsExact<T>::v;
  const long long u = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (u >= units) return;
  const long long t = u / H;
  const int hd = static_cast<int>(u - t * H);
  const float* o = o_raw + u * vdim;
  float ss = 0.f;
  for (int j = lane; j < vdim; j += 32) ss += o[j] * o[j];
  ss = wsum(ss);
  const float r = 1.f / sqrtf(ss / vdim + eps);
  T* d = out + t * ldo;
  for (int j = lane; j < vdim; j += 32) {
    float x = o[j] * r * ld(w + j);
    if (gate) {
      const float g = ld(gate + t * ld_gate + hd * vdim + j);
      x *= g * sigmoid<kExact>(g);
    }
    st(d + hd * vdim + j, x);
  }
  if (hd == H - 1)
    for (int j = H * vdim + lane; j < ldo; j += 32) st(d + j, 0.f);
}

// ------------------------------------------------------------------------------------------------- latent cache write
// One CTA per row.  With rot > 0 the row's rotated key part follows the latent features in the pool (at `part`), and the rotated
// features of every query head, which start at `dim` of its `dk`, turn in place.  Pairs are neighbours.
struct LatentWriteParams {
  const void* raw;           // [rows][ld]: latent projection
  const void* k_rot;         // [rows][ld]: projection of the rotated key part
  void* q;                   // [rows][ld]: query heads of dk features
  const void* w;             // [rank]
  void* pool;                // [pool rows][pitch]
  const long long* slots;
  const float2* table;       // [rows][rot / 2]
  long long pool_rows;
  int ld, rank, pitch, part, rot, H, dk, dim;
  float eps;
};
template <typename T>
__global__ void __launch_bounds__(128) latent_write_kernel(const LatentWriteParams p) {
  __shared__ float red[4];
  const long long t = blockIdx.x;
  const T* x = static_cast<const T*>(p.raw) + t * p.ld;
  const T* w = static_cast<const T*>(p.w);
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.rank; c += 128) {
    const float v = ld(x + c);
    ss += v * v;
  }
  const float2* cs = p.table + t * (p.rot >> 1);
  if (p.rot) {
    const int half = p.rot >> 1;
    T* q = static_cast<T*>(p.q) + t * p.ld + p.dim;
    for (int i = threadIdx.x; i < p.H * half; i += 128) {
      const int hd = i / half, k = i - hd * half;
      T* a = q + hd * p.dk + 2 * k;
      const float u = ld(a), v = ld(a + 1);
      const float2 f = cs[k];
      st(a, u * f.x - v * f.y);
      st(a + 1, v * f.x + u * f.y);
    }
  }
  ss = wsum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float r = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / p.rank + p.eps);
  const long long s = p.slots[t];
  if (s < 0 || s >= p.pool_rows) return;
  T* d = static_cast<T*>(p.pool) + s * p.pitch;
  const T* kr = static_cast<const T*>(p.k_rot) + t * p.ld;
  for (int c = threadIdx.x; c < p.pitch; c += 128) {
    float v = 0.f;
    if (c < p.rank) {
      v = ld(x + c) * r * ld(w + c);
    } else if (c >= p.part && c - p.part < p.rot) {
      const int i = c - p.part;
      const float2 f = cs[i >> 1];
      const float a = ld(kr + (i & ~1)), b = ld(kr + (i | 1));
      v = (i & 1) ? b * f.x + a * f.y : a * f.x - b * f.y;
    }
    st(d + c, v);
  }
}

// ------------------------------------------------------------------------------------------------- latent attention
// CUDA-core form for any sizes: CTA = (row, head), every warp walks every fourth visible position, a lane holds NR of the
// latent features of query, accumulator and current row; the four running softmaxes are merged at the end.
struct LatentParams {
  const void* q;          // [rows][H][R]
  const void* pool;       // [pool rows][R]; the first Rv features are the values
  const int* block_tables;
  const int* row_seg;     // [rows] or null (row = sequence)
  const int* row_pos;     // [rows] last visible position; null: ctx[row] - 1
  const int* ctx;
  const void* gate;       // [rows][ld_gate] or null
  void* out;              // [rows][H][Rv]
  int H, R, Rv, max_blocks, block_size, ld_gate;
  float scale;
};
template <typename T, int NR>
__global__ void __launch_bounds__(128) latent_attn_kernel(const LatentParams p) {
  extern __shared__ float sm[];                 // [4][Rv] accumulators
  __shared__ float sml[4][2];
  const int row = blockIdx.x, hd = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seg = p.row_seg ? p.row_seg[row] : row;
  const int n = (p.row_pos ? p.row_pos[row] : p.ctx[row] - 1) + 1;
  const int* bt = p.block_tables + static_cast<long long>(seg) * p.max_blocks;
  const T* pool = static_cast<const T*>(p.pool);
  const T* qp = static_cast<const T*>(p.q) + (static_cast<long long>(row) * p.H + hd) * p.R;
  float q[NR], o[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int c = lane + 32 * i;
    q[i] = c < p.R ? ld(qp + c) : 0.f;
    o[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int k = warp; k < n; k += 4) {
    const T* c = pool + (static_cast<long long>(bt[k / p.block_size]) * p.block_size + k % p.block_size) * p.R;
    float x[NR], s = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int j = lane + 32 * i;
      x[i] = j < p.R ? ld(c + j) : 0.f;
      s += q[i] * x[i];
    }
    s = wsum(s) * p.scale;
    const float mn = fmaxf(m, s), a = expf(m - mn), e = expf(s - mn);
    m = mn;
    l = l * a + e;
#pragma unroll
    for (int i = 0; i < NR; ++i) o[i] = o[i] * a + e * x[i];
  }
  if (lane == 0) { sml[warp][0] = m; sml[warp][1] = l; }
#pragma unroll
  for (int i = 0; i < NR; ++i)
    if (lane + 32 * i < p.Rv) sm[warp * p.Rv + lane + 32 * i] = o[i];
  __syncthreads();
  const float M = fmaxf(fmaxf(sml[0][0], sml[1][0]), fmaxf(sml[2][0], sml[3][0]));
  float w[4], L = 0.f;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    w[k] = sml[k][0] == -INFINITY ? 0.f : expf(sml[k][0] - M);
    L += w[k] * sml[k][1];
  }
  float f = L > 0.f ? 1.f / L : 0.f;
  if (p.gate) f *= sigmoid<true>(ld(static_cast<const T*>(p.gate) + static_cast<long long>(row) * p.ld_gate + hd));
  T* out = static_cast<T*>(p.out) + (static_cast<long long>(row) * p.H + hd) * p.Rv;
  for (int c = threadIdx.x; c < p.Rv; c += 128)
    st(out + c, (w[0] * sm[c] + w[1] * sm[p.Rv + c] + w[2] * sm[2 * p.Rv + c] + w[3] * sm[3 * p.Rv + c]) * f);
}

// attention output [T][n] times the sigmoid of a gate per feature, in place
template <typename T>
__global__ void gate_outputs_kernel(T* o, const T* __restrict__ gate, int n, int ld_gate) {
  constexpr bool kExact = IsExact<T>::v;
  const long long t = blockIdx.x;
  for (int c = threadIdx.x * 8; c < n; c += blockDim.x * 8) {
    F8 v = ld8(o + t * n + c);
    const F8 g = ld8(gate + t * ld_gate + c);
#pragma unroll
    for (int k = 0; k < 8; ++k) v.v[k] *= sigmoid<kExact>(g.v[k]);
    st8(o + t * n + c, v);
  }
}

// ------------------------------------------------------------------------------------------------- gated unit
// act 0: silu(g); act 1: tanh form of gelu, 0.5 (1 + tanh(u)) = sigmoid(2 u)
template <bool kExact>
__device__ __forceinline__ float glu_act(float g, int act) {
  const float z = act == 0 ? g : 1.5957691216057308f * (g + 0.044715f * g * g * g);      // 2 sqrt(2 / pi)
  return g * sigmoid<kExact>(z);
}
template <typename T>
__global__ void glu_kernel(const T* __restrict__ in, T* __restrict__ out, long long rows, int F, int ld_in, int act) {
  constexpr bool kExact = IsExact<T>::v;
  const int per = F / 8;
  const long long n = rows * per;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / per;
    const int c = static_cast<int>(i - r * per) * 8;
    F8 g = ld8(in + r * ld_in + c);
    const F8 u = ld8(in + r * ld_in + F + c);
#pragma unroll
    for (int k = 0; k < 8; ++k) g.v[k] = glu_act<kExact>(g.v[k], act) * u.v[k];
    st8(out + r * F + c, g);
  }
}

// ------------------------------------------------------------------------------------------------- CUDA-core GEMM
// C[z] = A[z] * B[z]^T (B [N][K]) or A[z] * B[z] (B [K][N]); fp32 accumulation in k order, any sizes and strides.
struct GemmParams {
  const void* A;
  const void* B;
  void* C;
  int M, N, K, lda, ldb, ldc, b_kn;
  long long sa, sb, sc;
};
template <typename T>
__global__ void __launch_bounds__(256) simt_gemm_kernel(const GemmParams p) {
  __shared__ float sa[16][64 + 4], sb[16][64 + 4];
  const T* A = static_cast<const T*>(p.A) + blockIdx.z * p.sa;
  const T* B = static_cast<const T*>(p.B) + blockIdx.z * p.sb;
  T* C = static_cast<T*>(p.C) + blockIdx.z * p.sc;
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, tid = threadIdx.x;
  const int tm = (tid >> 4) * 4, tn = (tid & 15) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + i * 256;
      const int r = e >> 4, k = e & 15;
      sa[k][r] = (m0 + r < p.M && k0 + k < p.K) ? ld(A + static_cast<long long>(m0 + r) * p.lda + k0 + k) : 0.f;
      if (!p.b_kn) {
        sb[k][r] = (n0 + r < p.N && k0 + k < p.K) ? ld(B + static_cast<long long>(n0 + r) * p.ldb + k0 + k) : 0.f;
      } else {
        const int n = e & 63, kk = e >> 6;
        sb[kk][n] = (n0 + n < p.N && k0 + kk < p.K) ? ld(B + static_cast<long long>(k0 + kk) * p.ldb + n0 + n) : 0.f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sa[k][tm]), b = *reinterpret_cast<const float4*>(&sb[k][tn]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += av[i] * bv[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (m0 + tm + i < p.M && n0 + tn + j < p.N) st(C + static_cast<long long>(m0 + tm + i) * p.ldc + n0 + tn + j, acc[i][j]);
}

template <typename T>
static int launch_latent_attn(const LatentParams& p, int rows, cudaStream_t stm) {
  const size_t smem = 4 * static_cast<size_t>(p.Rv) * 4;
  const dim3 grid(rows, p.H);
  if (p.R <= 128) latent_attn_kernel<T, 4><<<grid, 128, smem, stm>>>(p);
  else if (p.R <= 256) latent_attn_kernel<T, 8><<<grid, 128, smem, stm>>>(p);
  else if (p.R <= 512) latent_attn_kernel<T, 16><<<grid, 128, smem, stm>>>(p);
  else if (p.R <= 1024) latent_attn_kernel<T, 32><<<grid, 128, smem, stm>>>(p);
  else return -2;
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, bool kGla>
static int launch_scan(const HgrnParams& p, int segs, int rows, bool vec, cudaStream_t stm) {
  int NG = (p.dim + 31) / 32 * 4;                 // row groups of 8; whole warps (8 lanes per group)
  if (NG < 8) NG = 8;                             // at least 64 threads: they also fetch the values of a chunk
  if (NG * 8 > 512) return -2;
  const size_t smem = (static_cast<size_t>(SC_CH) * (3 * NG * 8 + 2 * SC_V + NG * SC_V)) * 4;
  if (smem > 227 * 1024) return -2;
  auto k = vec ? hgrn2_scan_kernel<T, true, kGla> : hgrn2_scan_kernel<T, false, kGla>;
  const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  k<<<dim3(segs, p.H, (p.vdim + SC_V - 1) / SC_V), NG * 8, smem, stm>>>(p, NG);
  const long long units = static_cast<long long>(rows) * p.H;
  head_norm_kernel<T><<<static_cast<unsigned>((units + 7) / 8), 256, 0, stm>>>(p.o_raw, static_cast<const T*>(p.norm_w), static_cast<T*>(p.out),
                                                                             kGla ? static_cast<const T*>(p.qfv) + p.gate_col : nullptr, p.ld, units, p.H, p.vdim,
                                                                             p.ldo, p.eps);
  rb_note_launch(2);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace stack
}  // namespace rb

using namespace rb;
using namespace rb::stack;
typedef __nv_bfloat16 bf16;

extern "C" int rb_embed_rows(const long long* tok, const void* w, float* res, void* h, int rows, int vocab, int pitch, float scale, int fp32,
                             cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (pitch % 8) return -2;
  const int thr = pitch / 8 < 256 ? (pitch / 8 + 31) / 32 * 32 : 256;
  if (fp32) embed_rows_kernel<float><<<rows, thr, 0, stm>>>(tok, (const float*)w, res, (float*)h, vocab, pitch, scale);
  else embed_rows_kernel<bf16><<<rows, thr, 0, stm>>>(tok, (const bf16*)w, res, (bf16*)h, vocab, pitch, scale);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

template <int MODE>
static int launch_norm_add(NormAddParams p, int rows, bool vec, int fp32, cudaStream_t stm) {
  while (p.wpg < NA_WARPS && p.groups * p.wpg * 2 <= NA_WARPS) p.wpg *= 2;
  const size_t smem = MODE == NA_SUM ? static_cast<size_t>(p.width) * 4 : 0;
  auto k = fp32 ? (vec ? norm_add_kernel<float, 8, MODE> : norm_add_kernel<float, 1, MODE>)
                : (vec ? norm_add_kernel<bf16, 8, MODE> : norm_add_kernel<bf16, 1, MODE>);
  if (smem > 40 * 1024) {
    if (smem > 200 * 1024) return -2;
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  k<<<rows, NA_WARPS * 32, smem, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_norm_add(float* res, const void* y, const void* w, const void* next_w, void* h, int rows, int ldy, int pitch, int width,
                           int groups, float eps, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (groups < 1 || width % groups || pitch < width || pitch % 8 || ldy % 8) return -2;
  NormAddParams p{res, y, w, next_w, h, ldy, pitch, width, groups, 1, eps};
  return launch_norm_add<NA_PLAIN>(p, rows, (width / groups) % 8 == 0, fp32, stm);
}

// y may be null; ex [sorted rows][ldy] are expert outputs (see NormAddParams), offset has one entry more than there are experts
extern "C" int rb_norm_add_experts(float* res, const void* y, const void* ex, const int* expert, const int* place, const int* offset,
                                   const float* weight, int top, int experts, const void* w, const void* next_w, void* h, int rows, int ldy,
                                   int pitch, int width, int groups, float eps, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (groups < 1 || width % groups || pitch < width || pitch % 8 || ldy % 8 || top < 1 || top > NA_MAX_TOP) return -2;
  NormAddParams p{res, y, w, next_w, h, ldy, pitch, width, groups, 1, eps, nullptr, 0, ex, expert, place, offset, weight, top, experts};
  return launch_norm_add<NA_SUM>(p, rows, (width / groups) % 8 == 0, fp32, stm);
}

template <bool kExperts>
static int launch_sum_norm(const SumNormParams& p, int rows, int fp32, cudaStream_t stm) {
  const bool vec = p.width % 8 == 0;
  const size_t smem = static_cast<size_t>(p.width) * 4;
  auto k = fp32 ? (vec ? sum_norm_kernel<float, 8, kExperts> : sum_norm_kernel<float, 1, kExperts>)
                : (vec ? sum_norm_kernel<bf16, 8, kExperts> : sum_norm_kernel<bf16, 1, kExperts>);
  if (smem > 40 * 1024) {
    if (smem > 200 * 1024) return -2;
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  k<<<rows, NA_WARPS * 32, smem, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

// y may be null, and so may ex (see rb_norm_add_experts), b, next_w and next_b; centre: layer norm, else RMS
extern "C" int rb_sum_norm(float* res, const void* y, const void* ex, const int* expert, const int* place, const int* offset, const float* weight,
                           int top, int experts, const void* w, const void* b, const void* next_w, const void* next_b, void* h, int rows, int ldy,
                           int pitch, int width, int centre, float alpha, float eps, float scale, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (width < 1 || pitch < width || pitch % 8 || ldy % 8 || ldy < width || (!y && !ex) || (ex && (top < 1 || top > NA_MAX_TOP))) return -2;
  SumNormParams p{res, y, ex, expert, place, offset, weight, top, experts, w, b, next_w, next_b, h, ldy, pitch, width, centre, alpha, eps, scale};
  return ex ? launch_sum_norm<true>(p, rows, fp32, stm) : launch_sum_norm<false>(p, rows, fp32, stm);
}

// the stream starts with the normed rows of the embedding table
extern "C" int rb_embed_norm(const long long* tok, const void* table, const void* w, float* res, void* h, int rows, int vocab, int pitch, int width,
                             int groups, float eps, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (groups < 1 || width % groups || pitch < width || pitch % 8) return -2;
  NormAddParams p{res, table, w, nullptr, h, pitch, pitch, width, groups, 1, eps, tok, vocab};
  return launch_norm_add<NA_EMBED>(p, rows, (width / groups) % 8 == 0, fp32, stm);
}

template <typename T, bool kGla>
static int launch_recurrence(const HgrnParams& p, int rows, int segs, cudaStream_t stm) {
  if (p.cu) {
    if (!p.o_raw) return -3;
    const bool vec = p.dim % 8 == 0 && p.vdim % 8 == 0 && p.ld % 8 == 0 && p.ldz % 4 == 0 &&
                     (reinterpret_cast<uintptr_t>(p.qfv) | reinterpret_cast<uintptr_t>(p.z)) % 16 == 0;
    return launch_scan<T, kGla>(p, segs, rows, vec, stm);
  }
  const int lpr = p.vp / 4, ng = HS_THREADS / lpr;
  const size_t smem = (3 * static_cast<size_t>((p.dim + 3) & ~3) + p.vp + static_cast<size_t>(ng) * p.vp) * 4;
  if (smem > 48 * 1024) return -2;
  hgrn2_step_kernel<T, kGla><<<dim3(segs, p.H), HS_THREADS, smem, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

// cu == null: one row per segment.  o_raw: scratch [rows][H][vdim] fp32, needed with cu.
extern "C" int rb_hgrn2(const void* qfv, const void* f_bias, const void* lower, const void* norm_w, float* state, const int* slot, const int* ctx,
                        const int* cu, float* o_raw, void* out, int rows, int segs, int H, int dim, int vdim, int vp, int ld, int ldo, float eps,
                        int fp32, cudaStream_t stm) {
  if (rows <= 0 || segs <= 0) return 0;
  if (vp % 4 || vp < vdim || vp > 4 * HS_THREADS || ld < H * (2 * dim + vdim) || ldo < H * vdim) return -2;
  HgrnParams p{qfv, f_bias, lower, norm_w, state, slot, ctx, cu, o_raw, out, H, dim, vdim, vp, ld, ldo, eps};
  return fp32 ? launch_recurrence<float, false>(p, rows, segs, stm) : launch_recurrence<bf16, false>(p, rows, segs, stm);
}

// rows [T][ld]: q | k | v, from gate_col on output gates; z [T][ldz] fp32, to which z_bias is added; q_scale: factor on q
extern "C" int rb_gla(const void* in, const float* z, int ldz, const void* z_bias, const void* norm_w, float* state, const int* slot, const int* ctx,
                      const int* cu, float* o_raw, void* out, int rows, int segs, int H, int dim, int vdim, int vp, int ld, int ldo, int gate_col, float eps,
                      float q_scale, float inv_root, int fp32, cudaStream_t stm) {
  if (rows <= 0 || segs <= 0) return 0;
  if (vp % 4 || vp < vdim || vp > 4 * HS_THREADS || gate_col < H * (2 * dim + vdim) || ld < gate_col + H * vdim || ldo < H * vdim || ldz < H * dim) return -2;
  HgrnParams p{in, z_bias, nullptr, norm_w, state, slot, ctx, cu, o_raw, out, H, dim, vdim, vp, ld, ldo, eps, z, ldz, gate_col, q_scale, inv_root};
  return fp32 ? launch_recurrence<float, true>(p, rows, segs, stm) : launch_recurrence<bf16, true>(p, rows, segs, stm);
}

// rot > 0: k_rot and q (see LatentWriteParams) share the pitch ld of raw; part: column of the rotated key part in the pool
extern "C" int rb_latent_write(const void* raw, const void* k_rot, void* q, int ld, const void* w, void* pool, const long long* slots,
                               const float* table, long long pool_rows, int rows, int rank, int pitch, int part, int rot, int H, int dk, int dim,
                               float eps, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (rank < 1 || pitch < rank || rot < 0 || rot % 2) return -2;
  if (rot && (!k_rot || !q || !table || part < rank || pitch < part + rot || H < 1 || dim < 0 || dk < dim + rot)) return -2;
  LatentWriteParams p{raw, k_rot, q, w, pool, slots, reinterpret_cast<const float2*>(table), pool_rows, ld, rank, pitch, part, rot, H, dk, dim, eps};
  if (fp32) latent_write_kernel<float><<<rows, 128, 0, stm>>>(p);
  else latent_write_kernel<bf16><<<rows, 128, 0, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_latent_attn(const void* q, const void* pool, const int* block_tables, const int* row_seg, const int* row_pos, const int* ctx,
                              const void* gate, void* out, int rows, int H, int R, int Rv, int max_blocks, int block_size, int ld_gate, float scale,
                              int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (Rv < 1 || Rv > R) return -2;
  LatentParams p{q, pool, block_tables, row_seg, row_pos, ctx, gate, out, H, R, Rv, max_blocks, block_size, ld_gate, scale};
  return fp32 ? launch_latent_attn<float>(p, rows, stm) : launch_latent_attn<bf16>(p, rows, stm);
}

// o [rows][n] *= sigmoid(gate [rows][ld_gate])
extern "C" int rb_gate_outputs(void* o, const void* gate, int ld_gate, int rows, int n, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (n % 8 || ld_gate % 8 || ld_gate < n || (reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate)) % 16) return -2;
  if (fp32) gate_outputs_kernel<float><<<rows, 256, 0, stm>>>((float*)o, (const float*)gate, n, ld_gate);
  else gate_outputs_kernel<bf16><<<rows, 256, 0, stm>>>((bf16*)o, (const bf16*)gate, n, ld_gate);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_glu(const void* in, void* out, long long rows, int F, int ld_in, int act, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (F % 8 || ld_in % 8 || ld_in < 2 * F || act < 0 || act > 1) return -2;
  long long blocks = (rows * (F / 8) + 255) / 256;
  if (blocks > num_sms() * 16LL) blocks = num_sms() * 16LL;
  if (fp32) glu_kernel<float><<<static_cast<unsigned>(blocks), 256, 0, stm>>>((const float*)in, (float*)out, rows, F, ld_in, act);
  else glu_kernel<bf16><<<static_cast<unsigned>(blocks), 256, 0, stm>>>((const bf16*)in, (bf16*)out, rows, F, ld_in, act);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_simt_gemm(const void* A, const void* B, void* C, int M, int N, int K, int lda, int ldb, int ldc, int b_kn, int batch, long long sa,
                            long long sb, long long sc, int fp32, cudaStream_t stm) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  if (batch > 65535 || (M + 63) / 64 > 65535) return -2;
  GemmParams p{A, B, C, M, N, K, lda, ldb, ldc, b_kn, sa, sb, sc};
  const dim3 grid((N + 63) / 64, (M + 63) / 64, batch);
  if (fp32) simt_gemm_kernel<float><<<grid, 256, 0, stm>>>(p);
  else simt_gemm_kernel<bf16><<<grid, 256, 0, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}
