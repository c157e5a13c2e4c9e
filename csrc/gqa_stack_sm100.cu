// Around the attention of composed stacks with cached keys and values: angles, rotation + norm + cache write, and a CUDA-core
// attention for any sizes.  Compiled WITHOUT fast-math: the 32-bit mode of the engine uses these kernels as they are.
//
//  * rope_table        cos / sin of every row's angles, once per forward
//  * attention_inputs  raw projections -> rotated and normed queries; keys and values into their pages (norms head by head, pairs
//                      of neighbours)
//  * projection_inputs the same with weighted norms over the whole query and key projections, and either pairing
//  * conv_inputs       the same with biases, a short causal convolution over time on every channel (the last rows of a sequence wait in a
//                      state slot) and weighted norms head by head
//  * mix_heads         outputs of every head's weights on every group's values -> heads whose weights were mixed
//  * paged_attention   one (row, head) per CTA: 32-bit mode, and head sizes that the tensor-core kernels do not take
#include "stack_common.cuh"

namespace rb {
namespace stack {

__global__ void rope_table_kernel(const int* __restrict__ pos, int offset, const double* __restrict__ freq, float2* __restrict__ out, int rows,
                                  int half) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows * half) return;
  const int t = i / half;
  double s, c;
  sincos(static_cast<double>(pos[t] + offset) * freq[i - t * half], &s, &c);      // late positions keep their low bits
  out[i] = make_float2(static_cast<float>(c), static_cast<float>(s));
}

struct InputParams {
  const void* qkv;           // [T][ld]: H query heads | G key heads | G value heads (keys and values only with k_pool)
  const float2* table;       // [T][rot / 2] or null
  void* q;                   // [T][H][dp]
  void* k_pool;              // [rows][G][dp] or null
  void* v_pool;              // [rows][G][vp]
  const long long* slots;    // [T] pool rows
  long long pool_rows;
  int T, H, G, dim, vdim, dp, vp, rot, ld;
  float eps;                 // <= 0: no norm
};
// One warp per (row, head); lane l holds the feature pairs l, l + 32, ...
template <typename T, int NP, bool kPair>
__global__ void __launch_bounds__(256) attention_inputs_kernel(const InputParams p) {
  const int lane = threadIdx.x & 31;
  const int per = p.H + (p.k_pool ? 2 * p.G : 0);
  const long long u = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (u >= static_cast<long long>(p.T) * per) return;
  const int t = static_cast<int>(u / per), hd = static_cast<int>(u - static_cast<long long>(t) * per);
  const T* src = static_cast<const T*>(p.qkv) + static_cast<long long>(t) * p.ld;
  const bool value = hd >= p.H + p.G;
  const int n = value ? p.vdim : p.dim, pitch = value ? p.vp : p.dp;
  T* dst;
  if (hd < p.H) {
    src += hd * p.dim;
    dst = static_cast<T*>(p.q) + (static_cast<long long>(t) * p.H + hd) * p.dp;
  } else {
    const long long slot = p.slots[t];
    if (slot < 0 || slot >= p.pool_rows) return;
    const int g = hd - p.H - (value ? p.G : 0);
    src += p.H * p.dim + (value ? p.G * p.dim + g * p.vdim : g * p.dim);
    dst = static_cast<T*>(value ? p.v_pool : p.k_pool) + (slot * p.G + g) * pitch;
  }
  float a[NP], b[NP], ss = 0.f;
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int e = 2 * (lane + 32 * i);
    a[i] = b[i] = 0.f;
    if constexpr (kPair) {
      if (e < n) {
        if constexpr (sizeof(T) == 4) {
          const float2 x = *reinterpret_cast<const float2*>(src + e);
          a[i] = x.x;
          b[i] = x.y;
        } else {
          const uint32_t x = *reinterpret_cast<const uint32_t*>(src + e);
          a[i] = __uint_as_float(x << 16);
          b[i] = __uint_as_float(x & 0xffff0000u);
        }
      }
    } else {
      if (e < n) a[i] = ld(src + e);
      if (e + 1 < n) b[i] = ld(src + e + 1);
    }
    if (!value && e < p.rot) {
      const float2 cs = p.table[static_cast<long long>(t) * (p.rot >> 1) + (e >> 1)];
      const float x = a[i] * cs.x - b[i] * cs.y;
      b[i] = b[i] * cs.x + a[i] * cs.y;
      a[i] = x;
    }
    ss += a[i] * a[i] + b[i] * b[i];
  }
  float r = 1.f;
  if (!value && p.eps > 0.f) r = 1.f / sqrtf(wsum(ss) / p.dim + p.eps);
#pragma unroll
  for (int i = 0; i < NP; ++i) {      // columns behind the head's features are written as zeros
    const int e = 2 * (lane + 32 * i);
    if (e >= pitch) continue;
    if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float2*>(dst + e) = make_float2(a[i] * r, b[i] * r);
    } else {
      const __nv_bfloat162 v = __floats2bfloat162_rn(a[i] * r, b[i] * r);
      *reinterpret_cast<__nv_bfloat162*>(dst + e) = v;
    }
  }
}

// Norms over the whole projection: one CTA per row sums the squares of all query and all key columns, then every thread turns and
// stores groups of V columns.  A feature's partner in its pair is `rot / 2` columns away, or its neighbour; it is read again
// (from the cache) instead of being handed over.
struct ProjectionParams {
  const void* qkv;           // [T][ld]: H query heads | G key heads | G value heads (keys and values only with k_pool)
  const void* q_w;           // [H * dim] or null
  const void* k_w;           // [G * dim] or null
  const float2* table;       // [T][rot / 2] or null
  void* q;                   // [T][H][dp]
  void* k_pool;              // [rows][G][dp] or null
  void* v_pool;              // [rows][G][vp]
  const long long* slots;    // [T] pool rows
  long long pool_rows;
  int H, G, dim, vdim, dp, vp, rot, halves, ld;
  float eps;                 // <= 0: no norm
};
constexpr int PI_WARPS = 8;
template <typename T, int V>
__global__ void __launch_bounds__(PI_WARPS * 32) projection_inputs_kernel(const ProjectionParams p) {
  __shared__ float red[2][PI_WARPS];
  const long long t = blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const T* row = static_cast<const T*>(p.qkv) + t * p.ld;
  const int qd = p.H * p.dim, kd = p.k_pool ? p.G * p.dim : 0;
  float r[2] = {1.f, 1.f};
  if (p.eps > 0.f) {
    float ss[2] = {0.f, 0.f};
    for (int c = tid * V; c < qd + kd; c += PI_WARPS * 32 * V) {      // (qd is a multiple of V)
      float a[V];
      ldv<V>(row + c, a);
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < V; ++i) s += a[i] * a[i];
      if (c < qd) ss[0] += s;
      else ss[1] += s;
    }
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      ss[k] = wsum(ss[k]);
      if (lane == 0) red[k][warp] = ss[k];
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < PI_WARPS; ++w) s += red[k][w];
      r[k] = 1.f / sqrtf(s / (k ? max(kd, 1) : qd) + p.eps);
    }
  }
  long long slot = 0;
  int heads = p.H;
  if (p.k_pool) {
    slot = p.slots[t];
    if (slot >= 0 && slot < p.pool_rows) heads += 2 * p.G;
  }
  const int half = p.rot >> 1, per = (max(p.dp, p.k_pool ? p.vp : 0) + V - 1) / V;
  for (int i = tid; i < heads * per; i += PI_WARPS * 32) {
    const int hd = i / per, e = (i - hd * per) * V;
    const int kind = hd < p.H ? 0 : (hd < p.H + p.G ? 1 : 2);
    const int n = kind == 2 ? p.vdim : p.dim, pitch = kind == 2 ? p.vp : p.dp;
    if (e >= pitch) continue;
    const int g = kind == 0 ? hd : hd - p.H - (kind == 2 ? p.G : 0);
    const T* src = row + (kind == 0 ? 0 : (kind == 1 ? qd : qd + p.G * p.dim)) + g * n;
    float x[V];
    if (e < n) {
      ldv<V>(src + e, x);
      if (kind < 2) {
        const T* w = static_cast<const T*>(kind ? p.k_w : p.q_w);
        const float f = r[kind];
        if (w) {
          float b[V];
          ldv<V>(w + g * n + e, b);
#pragma unroll
          for (int k = 0; k < V; ++k) x[k] *= f * b[k];
        } else {
#pragma unroll
          for (int k = 0; k < V; ++k) x[k] *= f;
        }
        if (e < p.rot) {
          const float2* cs = p.table + t * half;
          if (V > 1 && !p.halves) {      // both features of every pair are here
#pragma unroll
            for (int k = 0; k + 1 < V; k += 2) {
              const float2 a = cs[(e + k) >> 1];
              const float u = x[k] * a.x - x[k + 1] * a.y;
              x[k + 1] = x[k + 1] * a.x + x[k] * a.y;
              x[k] = u;
            }
          } else {
            const bool second = p.halves ? e >= half : (e & 1) != 0;
            const int at = p.halves ? (second ? e - half : e + half) : e ^ 1;
            const int pair = p.halves ? (second ? e - half : e) : e >> 1;
            float y[V], b[V];
            ldv<V>(src + at, y);
            if (w) ldv<V>(w + g * n + at, b);
#pragma unroll
            for (int k = 0; k < V; ++k) {
              const float2 a = cs[pair + k];
              const float o = y[k] * (w ? f * b[k] : f);
              x[k] = second ? x[k] * a.x + o * a.y : x[k] * a.x - o * a.y;
            }
          }
        }
      }
    } else {      // columns behind the head's features are written as zeros
#pragma unroll
      for (int k = 0; k < V; ++k) x[k] = 0.f;
    }
    T* dst = kind == 0 ? static_cast<T*>(p.q) + (t * p.H + g) * p.dp : static_cast<T*>(kind == 1 ? p.k_pool : p.v_pool) + (slot * p.G + g) * pitch;
    stv<V>(dst + e, x);
  }
}

// One warp per head and `runs` runs of RUN rows.  Lane l holds 2 NP consecutive features with their weights; a run's raw rows and what is
// known about them are fetched at once, and the rows slide through registers.  With one row per sequence the warp also moves the state on;
// otherwise conv_state_kernel does, afterwards.
struct ConvParams {
  const void* qkv;           // [T][ld]: H query heads | G key heads | G value heads (keys and values only with k_pool)
  const void* bias;          // [C] or null
  const void* taps;          // [C][n], the last one on the row itself; null: none
  void* state;               // [slots][n - 1][C] raw rows before a segment, the newest last
  const void* q_w;           // [dim] weights of the norms (eps > 0)
  const void* k_w;
  const float2* table;       // [T][rot / 2] or null
  void* q;                   // [T][H][dp]
  void* k_pool;              // [rows][G][dp] or null
  void* v_pool;              // [rows][G][vp]
  const long long* slots;    // [T] pool rows
  const int* ctx;            // [segments]
  const int* state_slot;     // [segments]
  const int* cu;             // [segments + 1]; null: one row per segment
  const int* seg_of;         // [T] (with cu)
  const int* pos;            // [T] (with cu)
  long long pool_rows;
  int T, H, G, dim, vdim, dp, vp, rot, ld, n, C, runs;
  float eps;                 // <= 0: no norm
};
// N consecutive elements of which `left` exist (kVec: all or none, N * sizeof(T) aligned)
template <typename T, int N, bool kVec>
struct Run {      // as loaded: 16-bit pairs stay packed until they are used
  static constexpr bool kPacked = kVec && sizeof(T) == 2;
  static constexpr int W = kPacked ? N / 2 : N;
  uint32_t u[W];
  __device__ __forceinline__ void load(const T* p, int left) {
#pragma unroll
    for (int i = 0; i < W; ++i) u[i] = 0u;
    if constexpr (kVec) {
      if (left <= 0) return;
      const uint32_t* w = reinterpret_cast<const uint32_t*>(p);
      if constexpr (W % 4 == 0 && kPacked) {
#pragma unroll
        for (int i = 0; i < W; i += 4) *reinterpret_cast<uint4*>(u + i) = *reinterpret_cast<const uint4*>(w + i);
      } else if constexpr (W % 2 == 0) {
#pragma unroll
        for (int i = 0; i < W; i += 2) *reinterpret_cast<uint2*>(u + i) = *reinterpret_cast<const uint2*>(w + i);
      } else {
        u[0] = *w;
      }
    } else {
#pragma unroll
      for (int i = 0; i < N; ++i)
        if (i < left) u[i] = __float_as_uint(ld(p + i));
    }
  }
  __device__ __forceinline__ float at(int i) const {
    if constexpr (kPacked) return __uint_as_float(i & 1 ? u[i >> 1] & 0xffff0000u : u[i >> 1] << 16);
    else return __uint_as_float(u[i]);
  }
};
template <typename T, int N, bool kVec>
__device__ __forceinline__ void load_run(const T* p, int left, float* v) {
  Run<T, N, kVec> r;
  r.load(p, left);
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = r.at(i);
}
template <typename T, int N, bool kVec>
__device__ __forceinline__ void store_run(T* p, int left, const float* v) {
  if constexpr (kVec) {
    if (left <= 0) return;
    if constexpr (sizeof(T) == 4) {
#pragma unroll
      for (int i = 0; i < N; i += 2) *reinterpret_cast<float2*>(p + i) = *reinterpret_cast<const float2*>(v + i);
    } else {
      uint32_t u[N / 2];
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        u[i] = *reinterpret_cast<const uint32_t*>(&b);
      }
      if constexpr (N % 8 == 0) {
#pragma unroll
        for (int i = 0; i < N / 2; i += 4) *reinterpret_cast<uint4*>(p + 2 * i) = *reinterpret_cast<const uint4*>(u + i);
      } else if constexpr (N == 4) {
        *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(u);
      } else {
#pragma unroll
        for (int i = 0; i < N / 2; ++i) *reinterpret_cast<uint32_t*>(p + 2 * i) = u[i];
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (i < left) st(p + i, v[i]);
  }
}
// kVec: heads, their pitches, rows and the state split into aligned runs of 2 NP features
template <typename T, int NP, int NT, int RUN, bool kVec>
__global__ void __launch_bounds__(256, NP <= 2 && NT <= 4 ? 2 : 1) conv_inputs_kernel(const ConvParams p) {
  constexpr int N = 2 * NP;
  const int lane = threadIdx.x & 31;
  const int per = p.H + (p.k_pool ? 2 * p.G : 0);
  const long long u = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const long long part = u / per;
  const int hd = static_cast<int>(u - part * per);
  if (part * p.runs * RUN >= p.T) return;
  const bool value = hd >= p.H + p.G;
  const int n = value ? p.vdim : p.dim, pitch = value ? p.vp : p.dp;
  const int g = hd - (hd < p.H ? 0 : p.H + (value ? p.G : 0));
  const int ch = (hd < p.H ? 0 : p.H * p.dim + (value ? p.G * p.dim : 0)) + g * n;      // first channel of the head
  const int e = N * lane, left = n - e;
  const T* src = static_cast<const T*>(p.qkv) + ch + e;
  const bool normed = !value && p.eps > 0.f;
  float w[NT][N], bias[N], nw[N];
#pragma unroll
  for (int i = 0; i < N; ++i) {
#pragma unroll
    for (int k = 0; k < NT; ++k) w[k][i] = 0.f;
    w[0][i] = 1.f;
    bias[i] = 0.f;
    nw[i] = 1.f;
  }
  if (p.taps) {
    const T* tp = static_cast<const T*>(p.taps) + static_cast<long long>(ch + e) * p.n;
    if (kVec && NT == 4 && p.n == NT) {
      float v[N * NT];
      load_run<T, N * NT, kVec>(tp, left, v);
#pragma unroll
      for (int i = 0; i < N; ++i)
#pragma unroll
        for (int k = 0; k < NT; ++k) w[k][i] = v[i * NT + NT - 1 - k];
    } else {
#pragma unroll
      for (int i = 0; i < N; ++i)
#pragma unroll
        for (int k = 0; k < NT; ++k)
          if (i < left && k < p.n) w[k][i] = ld(tp + i * p.n + p.n - 1 - k);
    }
  }
  if (p.bias) load_run<T, N, kVec>(static_cast<const T*>(p.bias) + ch + e, left, bias);
  if (normed) load_run<T, N, kVec>(static_cast<const T*>(hd < p.H ? p.q_w : p.k_w) + e, left, nw);
  float past[NT > 1 ? NT - 1 : 1][N];      // rows t - 1, t - 2, .. with their biases, zeros before the sequence's start
  int seg = -1;
  for (int r = 0; r < p.runs; ++r) {
    const int t0 = (static_cast<int>(part) * p.runs + r) * RUN, rows = min(p.T - t0, RUN);
    if (rows <= 0) break;
    // what is known about the rows: lane i holds it for row t0 + i
    int m_seg = 0, m_at = 0, m_first = 0, m_state = 0;
    long long m_slot = 0;
    if (lane < rows) {
      const int t = t0 + lane;
      m_seg = p.cu ? p.seg_of[t] : t;
      m_at = p.cu ? p.pos[t] : p.ctx[t] - 1;
      m_first = p.cu ? p.cu[m_seg] : t;
      m_state = p.state_slot[m_seg];
      if (hd >= p.H) m_slot = p.slots[t];
    }
    Run<T, N, kVec> x[RUN];
    float2 cs[RUN][NP];
#pragma unroll
    for (int k = 0; k < RUN; ++k) {
      if (k < rows) x[k].load(src + static_cast<long long>(t0 + k) * p.ld, left);
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        cs[k][i] = make_float2(1.f, 0.f);
        if (k < rows && !value && e + 2 * i < p.rot) cs[k][i] = p.table[static_cast<long long>(t0 + k) * (p.rot >> 1) + (e >> 1) + i];
      }
    }
#pragma unroll
    for (int k = 0; k < RUN; ++k) {
      if (k >= rows) break;
      const int t = t0 + k;
      const int s = __shfl_sync(0xffffffffu, m_seg, k);
      const long long slot = __shfl_sync(0xffffffffu, m_slot, k);
      if (s != seg) {      // the rows in front of this one
        seg = s;
        const int at = __shfl_sync(0xffffffffu, m_at, k), local = t - __shfl_sync(0xffffffffu, m_first, k);
        const int place = __shfl_sync(0xffffffffu, m_state, k);
        T* state = p.n > 1 ? static_cast<T*>(p.state) + static_cast<long long>(place) * (p.n - 1) * p.C + ch + e : nullptr;
#pragma unroll
        for (int b = 1; b < NT; ++b) {
          const bool there = b < p.n && b <= at;
          const T* from = b <= local ? src + static_cast<long long>(t - b) * p.ld : state + static_cast<long long>(p.n - 1 - (b - local)) * p.C;
          load_run<T, N, kVec>(from, there ? left : 0, past[b - 1]);
        }
        if (!p.cu && p.n > 1) {      // the state moves on by one row
#pragma unroll
          for (int b = NT - 1; b >= 1; --b)
            if (b < p.n) {
              float moved[N];
#pragma unroll
              for (int i = 0; i < N; ++i) moved[i] = b > 1 ? past[b > 1 ? b - 2 : 0][i] : x[k].at(i);
              store_run<T, N, kVec>(state + static_cast<long long>(p.n - 1 - b) * p.C, left, moved);
            }
        }
#pragma unroll
        for (int b = 1; b < NT; ++b)
#pragma unroll
          for (int i = 0; i < N; ++i) past[b - 1][i] += b < p.n && b <= at ? bias[i] : 0.f;
      }
      float y[N], ss = 0.f;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const float now = x[k].at(i) + bias[i];
        float a = w[0][i] * now;
#pragma unroll
        for (int b = 1; b < NT; ++b) a += w[b][i] * past[b - 1][i];      // (taps behind the last one are zero)
#pragma unroll
        for (int b = NT - 1; b > 1; --b) past[b - 1][i] = past[b - 2][i];
        if (NT > 1) past[0][i] = now;
        y[i] = a;
        ss += a * a;
      }
      if (normed) {
        const float f = 1.f / sqrtf(wsum(ss) / p.dim + p.eps);
#pragma unroll
        for (int i = 0; i < N; ++i) y[i] *= f * nw[i];
      }
      T* dst;
      if (hd < p.H) {
        dst = static_cast<T*>(p.q) + (static_cast<long long>(t) * p.H + hd) * p.dp;
      } else {
        if (slot < 0 || slot >= p.pool_rows) continue;
        dst = static_cast<T*>(value ? p.v_pool : p.k_pool) + (slot * p.G + g) * pitch;
      }
#pragma unroll
      for (int i = 0; i < N; i += 2) {
        const float2 f = cs[k][i >> 1];
        const float a = y[i] * f.x - y[i + 1] * f.y;
        y[i + 1] = y[i + 1] * f.x + y[i] * f.y;
        y[i] = a;
      }
      store_run<T, N, kVec>(dst + e, pitch - e, y);      // columns behind the head's features are written as zeros
    }
  }
}

// The last n - 1 raw rows of every segment, or of what was before it and the segment together, become its state.
template <typename T>
__global__ void __launch_bounds__(256) conv_state_kernel(const ConvParams p) {
  const int s = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
  if (c >= p.C) return;
  const int lo = p.cu[s], len = p.cu[s + 1] - lo;
  const bool fresh = p.ctx[s] == len;
  T* state = static_cast<T*>(p.state) + static_cast<long long>(p.state_slot[s]) * (p.n - 1) * p.C + c;
  const T* src = static_cast<const T*>(p.qkv) + c;
  for (int j = 0; j < p.n - 1; ++j) {      // (what is read lies behind what has been written)
    const int i = len + j;
    float v;
    if (i >= p.n - 1) v = ld(src + static_cast<long long>(lo + i - (p.n - 1)) * p.ld);
    else v = fresh ? 0.f : ld(state + static_cast<long long>(i) * p.C);
    st(state + static_cast<long long>(j) * p.C, v);
  }
}

// out[t][h] = sum over g of mix[h][g] wide[t][g][group of h]: `wide` holds what every head's weights make of every group's values.
// Any type: thread = (token, four heads of one group, eight columns).
template <typename T>
__global__ void __launch_bounds__(128) mix_heads_kernel(const T* __restrict__ wide, const T* __restrict__ mix, T* __restrict__ out, long long units, int H,
                                                        int G, int vo) {
  const long long u = static_cast<long long>(blockIdx.x) * 128 + threadIdx.x;
  if (u >= units) return;
  const int cols = vo / 8, rep = H / G, quads = (rep + 3) / 4;
  const int c = static_cast<int>(u % cols) * 8;
  long long r = u / cols;
  const int quad = static_cast<int>(r % quads) * 4;
  r /= quads;
  const int grp = static_cast<int>(r % G);
  const long long t = r / G;
  const T* src = wide + (t * H * G + grp) * vo + c;
  const T* m = mix + static_cast<long long>(grp * rep + quad) * H;
  float acc[4][8];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
#pragma unroll 4
  for (int g = 0; g < H; ++g) {
    float a[8];
    ldv<8>(src + static_cast<long long>(g) * G * vo, a);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float f = quad + i < rep ? ld(m + i * H + g) : 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[i][j] += f * a[j];
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
    if (quad + i < rep) stv<8>(out + (t * H + grp * rep + quad + i) * vo + c, acc[i]);
}

// bf16, up to 16 heads per group: warp = (token, group, 64 columns), one m16n8k16 product per 16 heads g and 8 columns.  This pass is bound by
// reading `wide`, and what its products need of the tensor cores is a few of these per 16-byte load.  A lane fetches 8 consecutive columns of
// the rows g that its fragments hold; which columns form a product's eight is free, so column j of every lane quarter's run goes to product j.
template <int KS>
__global__ void __launch_bounds__(256) mix_heads_mma_kernel(const __nv_bfloat16* __restrict__ wide, const __nv_bfloat16* __restrict__ mix,
                                                            __nv_bfloat16* __restrict__ out, int tokens, int H, int G, int vo) {
  const int lane = threadIdx.x & 31, q = lane >> 2, k2 = (lane & 3) * 2;
  const int runs = (vo + 63) / 64, rep = H / G;
  const int grp = blockIdx.y / runs, c = (blockIdx.y % runs) * 64 + q * 8;
  const long long row = static_cast<long long>(G) * vo;      // elements between two heads g
  uint32_t a[KS][4];                                         // rows: heads of the group, columns: heads g
#pragma unroll
  for (int s = 0; s < KS; ++s)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int h = q + (i & 1) * 8, g = s * 16 + k2 + (i >> 1) * 8;
      const __nv_bfloat16* m = mix + static_cast<long long>(grp * rep + h) * H + g;
      const uint32_t lo = h < rep && g < H ? __bfloat16_as_ushort(m[0]) : 0, hi = h < rep && g + 1 < H ? __bfloat16_as_ushort(m[1]) : 0;
      a[s][i] = lo | hi << 16;
    }
  for (int t = blockIdx.x * 8 + (threadIdx.x >> 5); t < tokens; t += gridDim.x * 8) {
    const __nv_bfloat16* src = wide + static_cast<long long>(t) * H * row + static_cast<long long>(grp) * vo + c;
    uint4 x[KS][4];
#pragma unroll
    for (int s = 0; s < KS; ++s)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int g = s * 16 + k2 + (i & 1) + (i >> 1) * 8;
        x[s][i] = make_uint4(0, 0, 0, 0);
        if (g < H && c < vo) x[s][i] = __ldcs(reinterpret_cast<const uint4*>(src + g * row));
      }
    float d[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e) d[j][e] = 0.f;
#pragma unroll
      for (int s = 0; s < KS; ++s) {
        const uint32_t* w0 = reinterpret_cast<const uint32_t*>(&x[s][0]) + (j >> 1);
        uint32_t b[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {      // heads g and g + 1 of column j
          const uint32_t lo = w0[i * 8], hi = w0[i * 8 + 4];
          b[i] = (j & 1) ? __byte_perm(lo, hi, 0x7632) : __byte_perm(lo, hi, 0x5410);
        }
        asm volatile(
            "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
            : "+f"(d[j][0]), "+f"(d[j][1]), "+f"(d[j][2]), "+f"(d[j][3])
            : "r"(a[s][0]), "r"(a[s][1]), "r"(a[s][2]), "r"(a[s][3]), "r"(b[0]), "r"(b[1]));
      }
    }
    // d[j][e]: head q + (e / 2) 8, column j of the run of lane quarter k2 + (e & 1)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = q + (e >> 1) * 8, col = (blockIdx.y % runs) * 64 + (k2 + (e & 1)) * 8;
      if (h < rep && col < vo) {
        F8 o;
#pragma unroll
        for (int j = 0; j < 8; ++j) o.v[j] = d[j][e];
        st8(out + (static_cast<long long>(t) * H + grp * rep + h) * vo + col, o);
      }
    }
  }
}

// CTA = (row, head), every warp walks every fourth visible position, a lane holds NR features of query, accumulator, key and
// value; the four running softmaxes and the sink are merged at the end.
struct GqaParams {
  const void* q;            // [rows][H][dp]
  const void* k_pool;       // [pool rows][G][dp]
  const void* v_pool;       // [pool rows][G][vp]
  const int* block_tables;
  const int* row_seg;       // [rows] or null (row = segment)
  const int* row_pos;       // [rows] last visible position; null: ctx[row] - 1
  const int* ctx;
  const void* sink;         // [H] or null
  const void* gate;         // [rows][ld_gate]: sigmoid(gate) of every output feature, head h's at h * vo, or null
  void* out;                // [rows][H][vo]
  int H, G, dp, vp, vo, max_blocks, block_size, ld_gate;
  int window;               // positions a row sees, its own included (0: all)
  int keep;                 // with a window: the first positions that stay visible
  int chunk;                // > 0: a row sees its own chunk of this many positions
  int wide;                 // the head's weights meet the values of every group (blockIdx.z): out [rows][H][G][vo], no gate
  float scale;
  float cap;                // > 0: scores s become cap tanh(s / cap)
};
template <typename T, int NR>
__global__ void __launch_bounds__(128) gqa_attn_kernel(const GqaParams p) {
  extern __shared__ float sm[];                 // [4][vp] accumulators
  __shared__ float sml[4][2];
  const int row = blockIdx.x, hd = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = hd / (p.H / p.G);
  const int seg = p.row_seg ? p.row_seg[row] : row;
  const int n = (p.row_pos ? p.row_pos[row] : p.ctx[row] - 1) + 1;
  const int* bt = p.block_tables + static_cast<long long>(seg) * p.max_blocks;
  const T* qp = static_cast<const T*>(p.q) + (static_cast<long long>(row) * p.H + hd) * p.dp;
  float q[NR], o[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int c = lane + 32 * i;
    q[i] = c < p.dp ? ld(qp + c) : 0.f;
    o[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int first = p.chunk ? (n - 1) / p.chunk * p.chunk : (p.window && n > p.window ? n - p.window : 0);
  const int kept = min(p.keep, first);          // positions 0 .. kept - 1, then first .. n - 1
  for (int i = warp; i < kept + n - first; i += 4) {
    const int k = i < kept ? i : first + i - kept;
    const long long row_at = (static_cast<long long>(bt[k / p.block_size]) * p.block_size + k % p.block_size) * p.G;
    const T* kp = static_cast<const T*>(p.k_pool) + (row_at + g) * p.dp;
    const T* vp = static_cast<const T*>(p.v_pool) + (row_at + (p.wide ? blockIdx.z : g)) * p.vp;
    float x[NR], s = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int c = lane + 32 * i;
      if (c < p.dp) s += q[i] * ld(kp + c);
      x[i] = c < p.vp ? ld(vp + c) : 0.f;
    }
    s = wsum(s) * p.scale;
    if (p.cap > 0.f) s = p.cap * tanhf(s / p.cap);
    const float mn = fmaxf(m, s), a = expf(m - mn), e = expf(s - mn);
    m = mn;
    l = l * a + e;
#pragma unroll
    for (int i = 0; i < NR; ++i) o[i] = o[i] * a + e * x[i];
  }
  if (lane == 0) { sml[warp][0] = m; sml[warp][1] = l; }
#pragma unroll
  for (int i = 0; i < NR; ++i)
    if (lane + 32 * i < p.vp) sm[warp * p.vp + lane + 32 * i] = o[i];
  __syncthreads();
  float M = fmaxf(fmaxf(sml[0][0], sml[1][0]), fmaxf(sml[2][0], sml[3][0]));
  const float sink = p.sink ? ld(static_cast<const T*>(p.sink) + hd) : 0.f;
  if (p.sink) M = fmaxf(M, sink);
  float w[4], L = p.sink ? expf(sink - M) : 0.f;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    w[k] = sml[k][0] == -INFINITY ? 0.f : expf(sml[k][0] - M);
    L += w[k] * sml[k][1];
  }
  const float f = L > 0.f ? 1.f / L : 0.f;
  T* out = static_cast<T*>(p.out) + ((static_cast<long long>(row) * p.H + hd) * gridDim.z + blockIdx.z) * p.vo;
  const T* gate = p.gate ? static_cast<const T*>(p.gate) + static_cast<long long>(row) * p.ld_gate + hd * p.vo : nullptr;
  for (int c = threadIdx.x; c < p.vo; c += 128) {
    float o = (w[0] * sm[c] + w[1] * sm[p.vp + c] + w[2] * sm[2 * p.vp + c] + w[3] * sm[3 * p.vp + c]) * f;
    if (gate) o *= sigmoid<true>(ld(gate + c));
    st(out + c, o);
  }
}

template <typename T, bool kPair>
static int launch_inputs(const InputParams& p, cudaStream_t stm) {
  const long long units = static_cast<long long>(p.T) * (p.H + (p.k_pool ? 2 * p.G : 0));
  const unsigned grid = static_cast<unsigned>((units + 7) / 8);
  const int w = p.k_pool ? (p.dp > p.vp ? p.dp : p.vp) : p.dp;
  if (w <= 128) attention_inputs_kernel<T, 2, kPair><<<grid, 256, 0, stm>>>(p);
  else if (w <= 256) attention_inputs_kernel<T, 4, kPair><<<grid, 256, 0, stm>>>(p);
  else if (w <= 512) attention_inputs_kernel<T, 8, kPair><<<grid, 256, 0, stm>>>(p);
  else return -2;
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int NP, int NT>
static int launch_conv_np(ConvParams p, int segs, cudaStream_t stm) {
  constexpr int N = 2 * NP, bytes = sizeof(T) == 4 ? 8 : (N % 8 == 0 ? 16 : 2 * N);      // what a lane loads at once
  const bool pair = p.dim % N == 0 && p.dp % N == 0 && p.ld * sizeof(T) % bytes == 0 && p.C * sizeof(T) % bytes == 0 &&
                    (!p.k_pool || (p.vdim % N == 0 && p.vp % N == 0)) &&
                    (reinterpret_cast<uintptr_t>(p.qkv) | reinterpret_cast<uintptr_t>(p.state) | reinterpret_cast<uintptr_t>(p.q) |
                     reinterpret_cast<uintptr_t>(p.k_pool) | reinterpret_cast<uintptr_t>(p.v_pool) | reinterpret_cast<uintptr_t>(p.bias) |
                     reinterpret_cast<uintptr_t>(p.taps) | reinterpret_cast<uintptr_t>(p.q_w) | reinterpret_cast<uintptr_t>(p.k_w)) % 16 == 0;
  constexpr int RUN = NP <= 4 ? 4 : 2;
  p.runs = p.cu ? (p.T >= 2048 ? 32 : 8) / RUN : 1;      // (fewer rows: more warps instead)
  const int run = p.cu ? RUN * p.runs : 1;
  const long long units = static_cast<long long>((p.T + run - 1) / run) * (p.H + (p.k_pool ? 2 * p.G : 0));
  const unsigned grid = static_cast<unsigned>((units + 7) / 8);
  if (p.cu) {
    if (pair) conv_inputs_kernel<T, NP, NT, RUN, true><<<grid, 256, 0, stm>>>(p);
    else conv_inputs_kernel<T, NP, NT, RUN, false><<<grid, 256, 0, stm>>>(p);
    if (p.n > 1) conv_state_kernel<T><<<dim3(segs, (p.C + 255) / 256), 256, 0, stm>>>(p);
    rb_note_launch(p.n > 1 ? 2 : 1);
  } else {
    if (pair) conv_inputs_kernel<T, NP, NT, 1, true><<<grid, 256, 0, stm>>>(p);
    else conv_inputs_kernel<T, NP, NT, 1, false><<<grid, 256, 0, stm>>>(p);
    rb_note_launch(1);
  }
  return static_cast<int>(cudaGetLastError());
}
template <typename T, int NT>
static int launch_conv(const ConvParams& p, int segs, cudaStream_t stm) {
  const int w = p.k_pool ? (p.dp > p.vp ? p.dp : p.vp) : p.dp;
  if (w <= 64) return launch_conv_np<T, 1, NT>(p, segs, stm);
  if (w <= 128) return launch_conv_np<T, 2, NT>(p, segs, stm);
  if (w <= 256) return launch_conv_np<T, 4, NT>(p, segs, stm);
  if (w <= 512) return launch_conv_np<T, 8, NT>(p, segs, stm);
  return -2;
}

template <typename T>
static int launch_gqa(const GqaParams& p, int rows, cudaStream_t stm) {
  const size_t smem = 4 * static_cast<size_t>(p.vp) * 4;
  const dim3 grid(rows, p.H, p.wide ? p.G : 1);
  const int w = p.dp > p.vp ? p.dp : p.vp;
  if (w <= 64) gqa_attn_kernel<T, 2><<<grid, 128, smem, stm>>>(p);
  else if (w <= 128) gqa_attn_kernel<T, 4><<<grid, 128, smem, stm>>>(p);
  else if (w <= 256) gqa_attn_kernel<T, 8><<<grid, 128, smem, stm>>>(p);
  else if (w <= 512) gqa_attn_kernel<T, 16><<<grid, 128, smem, stm>>>(p);
  else return -2;
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace stack
}  // namespace rb

using namespace rb;
using namespace rb::stack;
typedef __nv_bfloat16 bf16;

// out [rows][half] (cos, sin) of (pos + offset) * freq
extern "C" int rb_rope_table(const int* pos, int offset, const double* freq, float* out, int rows, int half, cudaStream_t stm) {
  if (rows <= 0 || half <= 0) return 0;
  const long long n = static_cast<long long>(rows) * half;
  if (n > (1ll << 30)) return -2;
  rope_table_kernel<<<static_cast<unsigned>((n + 127) / 128), 128, 0, stm>>>(pos, offset, freq, reinterpret_cast<float2*>(out), rows, half);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_attention_inputs(const void* qkv, int ld, const float* table, void* q, void* k_pool, void* v_pool, const long long* slots,
                                   long long pool_rows, int T, int H, int G, int dim, int vdim, int dp, int vp, int rot, float eps, int fp32,
                                   cudaStream_t stm) {
  if (T <= 0) return 0;
  if (H < 1 || dim < 1 || dp < dim || dp % 2 || rot % 2 || rot < 0 || rot > dim || (rot && !table)) return -2;
  if (ld < H * dim + (k_pool ? G * (dim + vdim) : 0) || (k_pool && (!v_pool || !slots || G < 1 || vdim < 1 || vp < vdim || vp % 2))) return -2;
  InputParams p{qkv, reinterpret_cast<const float2*>(table), q, k_pool, v_pool, slots, pool_rows, T, H, G, dim, vdim, dp, vp, rot, ld, eps};
  const bool pair = dim % 2 == 0 && (!k_pool || vdim % 2 == 0) && ld % 2 == 0 && reinterpret_cast<uintptr_t>(qkv) % 8 == 0;
  if (fp32) return pair ? launch_inputs<float, true>(p, stm) : launch_inputs<float, false>(p, stm);
  return pair ? launch_inputs<bf16, true>(p, stm) : launch_inputs<bf16, false>(p, stm);
}

// q_w, k_w: weights of the norms over all query / key columns (null: none); eps <= 0: no norms; halves: pairs are rot / 2 apart
extern "C" int rb_projection_inputs(const void* qkv, int ld, const void* q_w, const void* k_w, const float* table, void* q, void* k_pool, void* v_pool,
                                    const long long* slots, long long pool_rows, int T, int H, int G, int dim, int vdim, int dp, int vp, int rot,
                                    int halves, float eps, int fp32, cudaStream_t stm) {
  if (T <= 0) return 0;
  if (H < 1 || dim < 1 || dp < dim || rot % 2 || rot < 0 || rot > dim || (rot && !table)) return -2;
  if (ld < H * dim + (k_pool ? G * (dim + vdim) : 0) || (k_pool && (!v_pool || !slots || G < 1 || vdim < 1 || vp < vdim))) return -2;
  ProjectionParams p{qkv, q_w, k_w, reinterpret_cast<const float2*>(table), q, k_pool, v_pool, slots, pool_rows, H, G, dim, vdim, dp, vp, rot, halves, ld,
                     eps};
  const uintptr_t bases = reinterpret_cast<uintptr_t>(qkv) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(q_w) |
                          reinterpret_cast<uintptr_t>(k_w) | reinterpret_cast<uintptr_t>(k_pool) | reinterpret_cast<uintptr_t>(v_pool);
  const bool vec = dim % 8 == 0 && dp % 8 == 0 && ld % 8 == 0 && rot % (halves ? 16 : 8) == 0 && bases % 16 == 0 &&
                   (!k_pool || (vdim % 8 == 0 && vp % 8 == 0));
  if (fp32) {
    if (vec) projection_inputs_kernel<float, 8><<<T, PI_WARPS * 32, 0, stm>>>(p);
    else projection_inputs_kernel<float, 1><<<T, PI_WARPS * 32, 0, stm>>>(p);
  } else {
    if (vec) projection_inputs_kernel<bf16, 8><<<T, PI_WARPS * 32, 0, stm>>>(p);
    else projection_inputs_kernel<bf16, 1><<<T, PI_WARPS * 32, 0, stm>>>(p);
  }
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

// C = H dim (+ G (dim + vdim) with k_pool) channels; taps [C][n] (n up to 8) or null; state [slots][n - 1][C] (n > 1); cu, seg_of, pos: segments of any
// length, or null: one row per segment.  q_w, k_w: weights of the norms (eps > 0)
extern "C" int rb_conv_inputs(const void* qkv, int ld, const void* bias, const void* taps, int n, void* state, const void* q_w, const void* k_w,
                              const float* table, void* q, void* k_pool, void* v_pool, const long long* slots, const int* ctx, const int* state_slot,
                              const int* cu, const int* seg_of, const int* pos, long long pool_rows, int T, int segs, int H, int G, int dim, int vdim,
                              int dp, int vp, int rot, float eps, int fp32, cudaStream_t stm) {
  if (T <= 0) return 0;
  if (H < 1 || dim < 1 || dp < dim || dp % 2 || rot % 2 || rot < 0 || rot > dim || (rot && !table) || n < 1 || n > 8 || (n > 1 && (!taps || !state))) return -2;
  const int C = H * dim + (k_pool ? G * (dim + vdim) : 0);
  if (ld < C || (k_pool && (!v_pool || !slots || G < 1 || vdim < 1 || vp < vdim || vp % 2)) || (cu && (!seg_of || !pos)) || !ctx || !state_slot) return -2;
  if (eps > 0.f && (!q_w || (k_pool && !k_w))) return -2;
  ConvParams p{qkv, bias, taps, state, q_w, k_w, reinterpret_cast<const float2*>(table), q, k_pool, v_pool, slots, ctx, state_slot, cu, seg_of, pos,
               pool_rows, T, H, G, dim, vdim, dp, vp, rot, ld, n, C, 1, eps};
  if (fp32) return n <= 4 ? launch_conv<float, 4>(p, segs, stm) : launch_conv<float, 8>(p, segs, stm);
  return n <= 4 ? launch_conv<bf16, 4>(p, segs, stm) : launch_conv<bf16, 8>(p, segs, stm);
}

// wide [rows][H][G][vo], mix [H][H], out [rows][H][vo]
extern "C" int rb_mix_heads(const void* wide, const void* mix, void* out, int rows, int H, int G, int vo, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (G < 1 || H % G || vo % 8 || vo < 8) return -2;
  const int ks = (H + 15) / 16, groups = G * ((vo + 63) / 64);
  if (!fp32 && H / G <= 16 && ks <= 4 && groups <= 65535) {
    const int blocks = (rows + 7) / 8, most = (num_sms() * 16 + groups - 1) / groups;
    const dim3 grid(blocks < most ? blocks : most, groups);
    auto k = ks == 1 ? mix_heads_mma_kernel<1> : ks == 2 ? mix_heads_mma_kernel<2> : ks == 3 ? mix_heads_mma_kernel<3> : mix_heads_mma_kernel<4>;
    k<<<grid, 256, 0, stm>>>((const bf16*)wide, (const bf16*)mix, (bf16*)out, rows, H, G, vo);
    rb_note_launch(1);
    return static_cast<int>(cudaGetLastError());
  }
  const long long units = static_cast<long long>(rows) * G * ((H / G + 3) / 4) * (vo / 8);
  const unsigned grid = static_cast<unsigned>((units + 127) / 128);
  if (fp32) mix_heads_kernel<float><<<grid, 128, 0, stm>>>((const float*)wide, (const float*)mix, (float*)out, units, H, G, vo);
  else mix_heads_kernel<bf16><<<grid, 128, 0, stm>>>((const bf16*)wide, (const bf16*)mix, (bf16*)out, units, H, G, vo);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_gqa_attn(const void* q, const void* k_pool, const void* v_pool, const int* block_tables, const int* row_seg, const int* row_pos,
                           const int* ctx, const void* sink, const void* gate, int ld_gate, void* out, int rows, int H, int G, int dp, int vp, int vo,
                           int max_blocks, int block_size, int window, int keep, int chunk, int wide, float scale, float cap, int fp32,
                           cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (G < 1 || G > 65535 || H % G || vo > vp || H > 65535 || window < 0 || keep < 0 || chunk < 0 || (gate && (wide || ld_gate < H * vo))) return -2;
  GqaParams p{q, k_pool, v_pool, block_tables, row_seg, row_pos, ctx, sink, gate, out, H, G, dp, vp, vo, max_blocks, block_size, ld_gate, window, keep,
              chunk, wide, scale, cap};
  return fp32 ? launch_gqa<float>(p, rows, stm) : launch_gqa<bf16>(p, rows, stm);
}
