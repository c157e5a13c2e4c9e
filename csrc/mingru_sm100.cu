// Gated running means (minGRU): S <- (1 - z) S + z c per channel, with gates and candidates that read the current token only, read out
// through silu(g).  Compiled WITHOUT fast-math: the recurrence and all that enters it are fp32.
//
//  * mingru_step   one row per sequence
//  * mingru_scan   segments of any length, every row read once: a CTA follows a few channels through a segment in blocks of time.  A thread
//                  owns two channels and eight consecutive rows of a block: it composes the rows' maps S -> (1 - z) S + z c into one, one
//                  warp chains the maps of the block's threads, and every thread runs its rows again from its own start.  The next
//                  block's rows are fetched meanwhile.
#include "stack_common.cuh"

namespace rb {
namespace stack {

struct MinGruParams {
  const void* rows;          // [T][ld]: z | x | g, each `pitch` columns
  const void* z_b;           // [pitch]
  const void* x_b;
  float* state;              // [slots][sp]
  const int* slot;           // [segments]
  const int* ctx;
  const int* cu;             // [segments + 1]; null: one row per segment
  void* out;                 // [T][pitch]
  int ld, pitch, width, sp;
};

template <typename T> struct Two;      // two neighbouring elements
template <> struct Two<float> { typedef float2 raw; };
template <> struct Two<__nv_bfloat16> { typedef uint32_t raw; };
__device__ __forceinline__ float2 open2(float2 v) { return v; }
__device__ __forceinline__ float2 open2(uint32_t u) { return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u)); }
__device__ __forceinline__ void st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }

// z c and 1 - z of raw projections that already carry their biases.  1 - z comes from the side on which it is known; in 16-bit mode the two
// denominators, which lie in [1, 2], share one reciprocal.
template <bool kExact>
__device__ __forceinline__ void gates(float a, float u, float& add, float& keep) {
  if constexpr (kExact) {
    keep = sigmoid<true>(-a);
    add = sigmoid<true>(a) * (u >= 0.f ? u + 0.5f : sigmoid<true>(u));
  } else {
    const float e = __expf(-fabsf(a)), f = __expf(-fabsf(u)), both = __fdividef(1.f, (1.f + e) * (1.f + f));
    const float r = both * (1.f + f);                              // 1 / (1 + e)
    const float z = a >= 0.f ? r : e * r;
    keep = a >= 0.f ? e * r : r;
    add = z * (u >= 0.f ? u + 0.5f : f * both * (1.f + e));
  }
}
template <bool kExact>
__device__ __forceinline__ float silu(float x) { return x * sigmoid<kExact>(x); }

template <typename T>
__global__ void __launch_bounds__(64) mingru_step_kernel(const MinGruParams p) {
  constexpr bool kExact = IsExact<T>::v;
  using R = typename Two<T>::raw;
  const int c = (blockIdx.y * 64 + threadIdx.x) * 2, s = blockIdx.x;
  if (c >= p.pitch) return;
  const T* src = static_cast<const T*>(p.rows) + static_cast<long long>(s) * p.ld + c;
  const float2 z = open2(*reinterpret_cast<const R*>(src)), x = open2(*reinterpret_cast<const R*>(src + p.pitch)),
               g = open2(*reinterpret_cast<const R*>(src + 2 * p.pitch));
  const float2 zb = open2(*reinterpret_cast<const R*>(static_cast<const T*>(p.z_b) + c)), xb = open2(*reinterpret_cast<const R*>(static_cast<const T*>(p.x_b) + c));
  float2 S = make_float2(0.f, 0.f), o = S;
  if (c < p.width) {
    float2* at = reinterpret_cast<float2*>(p.state + static_cast<long long>(p.slot[s]) * p.sp + c);
    if (p.ctx[s] != 1) S = *at;
    float2 add, keep;
    gates<kExact>(z.x + zb.x, x.x + xb.x, add.x, keep.x);
    gates<kExact>(z.y + zb.y, x.y + xb.y, add.y, keep.y);
    S.x = keep.x * S.x + add.x;
    S.y = keep.y * S.y + add.y;
    *at = S;      // (the slot has room for the second channel of an odd width)
    o = make_float2(S.x * silu<kExact>(g.x), c + 1 < p.width ? S.y * silu<kExact>(g.y) : 0.f);
  }
  st2(static_cast<T*>(p.out) + static_cast<long long>(s) * p.pitch + c, o);
}

// PAIRS channel pairs and 512 / PAIRS runs of time per CTA
constexpr int MG_THREADS = 512, MG_RUN = 8;
template <typename T, int PAIRS>
__global__ void __launch_bounds__(MG_THREADS) mingru_scan_kernel(const MinGruParams p) {
  constexpr bool kExact = IsExact<T>::v;
  constexpr int RUNS = MG_THREADS / PAIRS, BLOCK = RUNS * MG_RUN;
  using R = typename Two<T>::raw;
  __shared__ float2 map[RUNS][PAIRS * 2 + 1];      // per channel: factor and summand of a run, then factor unused and its start
  const int pr = threadIdx.x % PAIRS, run = threadIdx.x / PAIRS;
  const int c = (blockIdx.y * PAIRS + pr) * 2, k = blockIdx.x;
  const int lo = p.cu[k], hi = p.cu[k + 1];
  const bool live = c < p.pitch;
  const T* src = static_cast<const T*>(p.rows) + (live ? c : 0);
  float2 zb = make_float2(0.f, 0.f), xb = zb;
  if (live) {
    zb = open2(*reinterpret_cast<const R*>(static_cast<const T*>(p.z_b) + c));
    xb = open2(*reinterpret_cast<const R*>(static_cast<const T*>(p.x_b) + c));
  }
  // the chaining threads: one channel each
  const int chain = (blockIdx.y * PAIRS) * 2 + threadIdx.x;
  const bool chains = threadIdx.x < 2 * PAIRS && chain < p.width;
  float* state = chains ? p.state + static_cast<long long>(p.slot[k]) * p.sp + chain : nullptr;
  float carry = chains && p.ctx[k] != hi - lo ? *state : 0.f;
  R z[MG_RUN], x[MG_RUN], g[MG_RUN];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < MG_RUN; ++i) {
      const int t = t0 + run * MG_RUN + i;
      if (live && t < hi) {
        const T* r = src + static_cast<long long>(t) * p.ld;
        z[i] = *reinterpret_cast<const R*>(r);
        x[i] = *reinterpret_cast<const R*>(r + p.pitch);
        g[i] = *reinterpret_cast<const R*>(r + 2 * p.pitch);
      }
    }
  };
  fetch(lo);
  for (int t0 = lo; t0 < hi; t0 += BLOCK) {
    const int t = t0 + run * MG_RUN, n = min(MG_RUN, hi - t);
    float2 add[MG_RUN], keep[MG_RUN], A = make_float2(1.f, 1.f), B = make_float2(0.f, 0.f);
    R gate[MG_RUN];
#pragma unroll
    for (int i = 0; i < MG_RUN; ++i) {
      add[i] = make_float2(0.f, 0.f);
      keep[i] = make_float2(1.f, 1.f);
      if (live && i < n) {
        const float2 a = open2(z[i]), u = open2(x[i]);
        gates<kExact>(a.x + zb.x, u.x + xb.x, add[i].x, keep[i].x);
        gates<kExact>(a.y + zb.y, u.y + xb.y, add[i].y, keep[i].y);
        gate[i] = g[i];
      }
      A.x *= keep[i].x;
      A.y *= keep[i].y;
      B.x = keep[i].x * B.x + add[i].x;
      B.y = keep[i].y * B.y + add[i].y;
    }
    map[run][2 * pr] = make_float2(A.x, B.x);
    map[run][2 * pr + 1] = make_float2(A.y, B.y);
    if (t0 + BLOCK < hi) fetch(t0 + BLOCK);
    __syncthreads();
    if (threadIdx.x < 2 * PAIRS) {
#pragma unroll 8
      for (int r = 0; r < RUNS; ++r) {
        const float2 m = map[r][threadIdx.x];
        map[r][threadIdx.x].y = carry;
        carry = m.x * carry + m.y;
      }
    }
    __syncthreads();
    float2 S = make_float2(map[run][2 * pr].y, map[run][2 * pr + 1].y);
#pragma unroll
    for (int i = 0; i < MG_RUN; ++i)
      if (live && i < n) {
        S.x = keep[i].x * S.x + add[i].x;
        S.y = keep[i].y * S.y + add[i].y;
        const float2 v = open2(gate[i]);
        st2(static_cast<T*>(p.out) + static_cast<long long>(t + i) * p.pitch + c,
            make_float2(c < p.width ? S.x * silu<kExact>(v.x) : 0.f, c + 1 < p.width ? S.y * silu<kExact>(v.y) : 0.f));
      }
    // (a thread's next maps are written to cells that only the chaining threads and itself have read)
  }
  if (chains) *state = carry;
}

template <typename T>
static int launch_mingru(const MinGruParams& p, int segs, cudaStream_t stm) {
  if (!p.cu) {
    mingru_step_kernel<T><<<dim3(segs, (p.pitch / 2 + 63) / 64), 64, 0, stm>>>(p);
  } else if (static_cast<long long>(segs) * ((p.pitch + 31) / 32) >= num_sms() / 2) {
    mingru_scan_kernel<T, 16><<<dim3(segs, (p.pitch + 31) / 32), MG_THREADS, 0, stm>>>(p);
  } else {
    mingru_scan_kernel<T, 8><<<dim3(segs, (p.pitch + 15) / 16), MG_THREADS, 0, stm>>>(p);
  }
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace stack
}  // namespace rb

// rows [T][ld]: z | x | g of `pitch` columns each (width rounded up to 8), out [T][pitch]; state [slots][sp], sp even and at least the width
// rounded up to 2; cu: segments of any length, or null: one row per segment
extern "C" int rb_mingru(const void* rows, const void* z_b, const void* x_b, float* state, const int* slot, const int* ctx, const int* cu, void* out,
                         int segs, int width, int ld, int sp, int fp32, cudaStream_t stm) {
  using namespace rb::stack;
  if (segs <= 0) return 0;
  const int pitch = (width + 7) / 8 * 8;
  if (width < 1 || ld < 3 * pitch || ld % 2 || sp % 2 || sp < width || pitch / 16 >= 65535) return -2;
  MinGruParams p{rows, z_b, x_b, state, slot, ctx, cu, out, ld, pitch, width, sp};
  return fp32 ? launch_mingru<float>(p, segs, stm) : launch_mingru<__nv_bfloat16>(p, segs, stm);
}
