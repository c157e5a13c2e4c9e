// Gated running means (minGRU): S <- (1 - z) S + z c per channel, with gates and candidates that read the current token only, read out
// through silu(g).  Compiled WITHOUT fast-math: the recurrence and all that enters it are fp32.
//
// A thread follows two neighbouring channels.  Long segments are cut into SPANS that run side by side: the first pass computes what a
// span adds to a state of zero and the product of its 1 - z, one kernel chains the spans of a segment, and the last pass computes the
// outputs from the chained states.
#include "stack_common.cuh"

namespace rb {
namespace stack {

enum GruMode { kWhole = 0, kStates = 1, kFromScratch = 2 };
struct MinGruParams {
  const void* rows;          // [T][ld]: z | x | g, each `pitch` columns
  const void* z_b;           // [pitch]
  const void* x_b;
  float* state;              // [slots][sp]
  const int* slot;           // [segments]
  const int* ctx;
  const int* cu;             // [segments + 1]; null: one row per segment
  const int* spans;          // [n][2] rows (not kWhole)
  float2* span_sum;          // [n][pitch / 2]: kStates: sum of the span; kFromScratch: state at its start
  float2* span_keep;         // [n][pitch / 2] product of 1 - z
  void* out;                 // [T][pitch]
  int ld, pitch, width, sp;
};

__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ld2(const __nv_bfloat16* p) {
  const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
}
__device__ __forceinline__ void st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }

// z and 1 - z from the side on which the small one is known
template <bool kExact>
__device__ __forceinline__ void gate_of(float a, float& z, float& keep) {
  if constexpr (kExact) {
    z = sigmoid<true>(a);
    keep = sigmoid<true>(-a);
  } else {
    const float e = __expf(-fabsf(a)), r = __fdividef(1.f, 1.f + e);
    z = a >= 0.f ? r : e * r;
    keep = a >= 0.f ? e * r : r;
  }
}
template <bool kExact>
__device__ __forceinline__ float candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoid<kExact>(u); }

template <typename T, int kMode>
__global__ void __launch_bounds__(64) mingru_kernel(const MinGruParams p) {
  constexpr bool kExact = IsExact<T>::v;
  constexpr int U = 8;       // rows in flight
  const int c = (blockIdx.y * 64 + threadIdx.x) * 2;
  if (c >= p.pitch) return;
  const int k = blockIdx.x;
  int lo, hi;
  if (kMode == kWhole) {
    lo = p.cu ? p.cu[k] : k;
    hi = p.cu ? p.cu[k + 1] : k + 1;
  } else {
    lo = p.spans[2 * k];
    hi = p.spans[2 * k + 1];
  }
  const T* src = static_cast<const T*>(p.rows) + c;
  const float2 zb = ld2(static_cast<const T*>(p.z_b) + c), xb = ld2(static_cast<const T*>(p.x_b) + c);
  float* state = kMode == kWhole ? p.state + static_cast<long long>(p.slot[k]) * p.sp + c : nullptr;
  const bool live = c < p.width;
  float2 S = make_float2(0.f, 0.f), keep = make_float2(1.f, 1.f);
  if (kMode == kWhole) {
    if (live && p.ctx[k] != hi - lo) S = ld2(state);
  } else if (kMode == kFromScratch) {
    S = p.span_sum[static_cast<long long>(k) * (p.pitch >> 1) + (c >> 1)];
  }
  for (int t0 = lo; t0 < hi; t0 += U) {
    float2 z[U], x[U], g[U];
#pragma unroll
    for (int i = 0; i < U; ++i)
      if (t0 + i < hi) {
        const T* r = src + static_cast<long long>(t0 + i) * p.ld;
        z[i] = ld2(r);
        x[i] = ld2(r + p.pitch);
        if (kMode != kStates) g[i] = ld2(r + 2 * p.pitch);
      }
#pragma unroll
    for (int i = 0; i < U; ++i)
      if (t0 + i < hi) {
        float za, ka, zc, kc;
        gate_of<kExact>(z[i].x + zb.x, za, ka);
        gate_of<kExact>(z[i].y + zb.y, zc, kc);
        S.x = ka * S.x + za * candidate<kExact>(x[i].x + xb.x);
        S.y = kc * S.y + zc * candidate<kExact>(x[i].y + xb.y);
        if (kMode == kStates) {
          keep.x *= ka;
          keep.y *= kc;
        } else {
          float2 o = make_float2(S.x * g[i].x * sigmoid<kExact>(g[i].x), S.y * g[i].y * sigmoid<kExact>(g[i].y));
          if (c >= p.width) o.x = 0.f;
          if (c + 1 >= p.width) o.y = 0.f;
          st2(static_cast<T*>(p.out) + static_cast<long long>(t0 + i) * p.pitch + c, o);
        }
      }
  }
  if (kMode == kWhole && live) st2(state, S);      // (sp leaves room for the second channel)
  if (kMode == kStates) {
    const long long i = static_cast<long long>(k) * (p.pitch >> 1) + (c >> 1);
    p.span_sum[i] = S;
    p.span_keep[i] = keep;
  }
}

// chains the spans of a segment: what kStates left in span_sum[i] becomes the state at the start of span i
__global__ void __launch_bounds__(64) mingru_chain_kernel(const MinGruParams p, const int* __restrict__ first) {
  const int c = (blockIdx.y * 64 + threadIdx.x) * 2;
  if (c >= p.width) return;
  const int seg = blockIdx.x, a = first[seg], b = first[seg + 1];
  const bool fresh = p.ctx[seg] == p.spans[2 * b - 1] - p.spans[2 * a];
  float* state = p.state + static_cast<long long>(p.slot[seg]) * p.sp + c;
  float2 S = fresh ? make_float2(0.f, 0.f) : ld2(state);
  for (int k0 = a; k0 < b; k0 += 8) {
    float2 sum[8], keep[8];
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (k0 + i < b) {
        const long long at = static_cast<long long>(k0 + i) * (p.pitch >> 1) + (c >> 1);
        sum[i] = p.span_sum[at];
        keep[i] = p.span_keep[at];
      }
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (k0 + i < b) {
        p.span_sum[static_cast<long long>(k0 + i) * (p.pitch >> 1) + (c >> 1)] = S;
        S.x = keep[i].x * S.x + sum[i].x;
        S.y = keep[i].y * S.y + sum[i].y;
      }
  }
  st2(state, S);
}

template <typename T>
static int launch_mingru(const MinGruParams& p, int segs, int n_spans, const int* first, cudaStream_t stm) {
  const unsigned y = static_cast<unsigned>((p.pitch / 2 + 63) / 64);
  if (!n_spans) {
    mingru_kernel<T, kWhole><<<dim3(segs, y), 64, 0, stm>>>(p);
    rb_note_launch(1);
  } else {
    mingru_kernel<T, kStates><<<dim3(n_spans, y), 64, 0, stm>>>(p);
    mingru_chain_kernel<<<dim3(segs, y), 64, 0, stm>>>(p, first);
    mingru_kernel<T, kFromScratch><<<dim3(n_spans, y), 64, 0, stm>>>(p);
    rb_note_launch(3);
  }
  return static_cast<int>(cudaGetLastError());
}

}  // namespace stack
}  // namespace rb

// rows [T][ld]: z | x | g of `pitch` columns each (width rounded up to 8), out [T][pitch]; state [slots][sp], sp even and at least the width
// rounded up to 2.  n_spans > 0: spans [n_spans][2] rows, those of segment s being first[s] .. first[s + 1], with scratch [n_spans][pitch] for
// their sums and for the products of their 1 - z.
extern "C" int rb_mingru(const void* rows, const void* z_b, const void* x_b, float* state, const int* slot, const int* ctx, const int* cu, const int* spans,
                         const int* first, float* span_sum, float* span_keep, void* out, int segs, int n_spans, int width, int ld, int sp, int fp32,
                         cudaStream_t stm) {
  using namespace rb::stack;
  if (segs <= 0) return 0;
  const int pitch = (width + 7) / 8 * 8;
  if (width < 1 || ld < 3 * pitch || ld % 2 || sp % 2 || sp < width || (n_spans && (!spans || !first || !span_sum || !span_keep))) return -2;
  MinGruParams p{rows, z_b, x_b, state, slot, ctx, cu, spans, reinterpret_cast<float2*>(span_sum), reinterpret_cast<float2*>(span_keep), out, ld, pitch, width, sp};
  return fp32 ? launch_mingru<float>(p, segs, n_spans, first, stm) : launch_mingru<__nv_bfloat16>(p, segs, n_spans, first, stm);
}
