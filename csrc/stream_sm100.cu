// The residual stream of composed stacks whose sublayers read norms of it.  Compiled WITHOUT fast-math: the 32-bit mode uses the same
// kernels, and the stream and its norms are fp32 in both modes.
//
//  * stream_step   stream += mean of one or two sublayer outputs (each RMS-normed first, or plain) + the weighted rows of a token's
//                  experts; then the layer norms that the next layer reads, or a copy in the operands' type.  With one row per sequence
//                  the first norm also moves towards the sequence's row before (token shift), which a state slot keeps
//  * token_shift   the same move for segments of several rows
//  * side_gate     gelu(z) times a layer's own features of the tokens in a second embedding table
//  * softcap       cap * tanh(z / cap) on fp32 logits, in place
#include "stack_common.cuh"

namespace rb {
namespace stack {

constexpr int SS_WARPS = 8, SS_MAX_TOP = 64;
struct StreamStepParams {
  float* res;                // [rows][pitch], updated in place when there is anything to add
  const void* y[2];          // [rows][ldy] sublayer outputs, or null
  const void* yw[2];         // [pitch] weights of their RMS norms, or null: plain
  const void* ex;            // [sorted rows][ldx] expert outputs, row of a choice = offset[expert] + place; or null
  const int* expert;         // [rows][top]
  const int* place;
  const int* offset;
  const float* weight;
  const void* nw[2];         // [pitch] weights of the layer norms, or null
  void* out[2];              // [rows][pitch]
  const void* mu;            // [pitch] token shift of out[0] (one row per sequence), or null
  void* state;               // [slots][pitch]
  const int* slot;           // [rows]
  const int* ctx;            // [rows] 1: the sequence's first token
  int ldy[2], ldx, top, pitch, width, n_y, n_out;
  float eps;
};

template <typename T, int V>
__global__ void __launch_bounds__(SS_WARPS * 32) stream_step_kernel(const StreamStepParams p) {
  extern __shared__ __align__(16) float z[];      // [width]; every thread reads back only what it wrote itself
  __shared__ float red[4][SS_WARPS];
  __shared__ long long ex_at[SS_MAX_TOP];
  __shared__ float ex_w[SS_MAX_TOP];
  const long long row = blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, step = SS_WARPS * 32 * V;
  float* res = p.res + row * p.pitch;
  const float inv_n = 1.f / p.width;
  auto total = [&](float v, int k) {      // over the CTA; every k is used once
    v = wsum(v);
    if (lane == 0) red[k][warp] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < SS_WARPS; ++i) s += red[k][i];
    return s;
  };
  if (p.ex && tid < p.top) {
    const long long i = row * p.top + tid;
    ex_at[tid] = (static_cast<long long>(p.offset[p.expert[i]]) + p.place[i]) * p.ldx;
    ex_w[tid] = p.weight[i];
  }
  const T* y0 = p.n_y > 0 ? static_cast<const T*>(p.y[0]) + row * p.ldy[0] : nullptr;
  const T* y1 = p.n_y > 1 ? static_cast<const T*>(p.y[1]) + row * p.ldy[1] : nullptr;
  const T* w0 = static_cast<const T*>(p.yw[0]);
  const T* w1 = static_cast<const T*>(p.yw[1]);
  float f0 = p.n_y > 1 ? 0.5f : 1.f, f1 = 0.5f;
  if (w0) {
    float s0 = 0.f, s1 = 0.f;
    for (int c = tid * V; c < p.width; c += step) {
      float a[V];
      ldv<V>(y0 + c, a);
#pragma unroll
      for (int i = 0; i < V; ++i) s0 += a[i] * a[i];
      if (y1) {
        ldv<V>(y1 + c, a);
#pragma unroll
        for (int i = 0; i < V; ++i) s1 += a[i] * a[i];
      }
    }
    s1 = wsum(s1);
    if (lane == 0) red[1][warp] = s1;
    f0 /= sqrtf(total(s0, 0) * inv_n + p.eps);
    s1 = 0.f;
#pragma unroll
    for (int i = 0; i < SS_WARPS; ++i) s1 += red[1][i];
    f1 /= sqrtf(s1 * inv_n + p.eps);
  } else {
    __syncthreads();      // the experts' places
  }
  T* out0 = static_cast<T*>(p.out[0]) + row * p.pitch;
  const bool norms = p.nw[0] != nullptr;
  float sum = 0.f;
  for (int c = tid * V; c < p.width; c += step) {
    float x[V], a[V], b[V];
    ldv<V>(res + c, x);
    if (y0) {
      ldv<V>(y0 + c, a);
      if (w0) ldv<V>(w0 + c, b);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] += a[i] * (w0 ? f0 * b[i] : f0);
    }
    if (y1) {
      ldv<V>(y1 + c, a);
      if (w1) ldv<V>(w1 + c, b);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] += a[i] * (w1 ? f1 * b[i] : f1);
    }
    if (p.ex) {
      const T* ex = static_cast<const T*>(p.ex) + c;
#pragma unroll 4
      for (int k = 0; k < p.top; ++k) {
        ldv<V>(ex + ex_at[k], a);
        const float f = ex_w[k];
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] += f * a[i];
      }
    }
    if (y0 || p.ex) stv<V>(res + c, x);
    if (norms) {
      stv<V>(z + c, x);
#pragma unroll
      for (int i = 0; i < V; ++i) sum += x[i];
    } else {
      stv<V>(out0 + c, x);
    }
  }
  if (norms) {
    const float mean = total(sum, 2) * inv_n;
    float ss = 0.f;
    for (int c = tid * V; c < p.width; c += step) {
      float x[V];
      ldv<V>(z + c, x);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += (x[i] - mean) * (x[i] - mean);
    }
    const float r = 1.f / sqrtf(total(ss, 3) * inv_n + p.eps);
    const T* mu = static_cast<const T*>(p.mu);
    T* state = mu ? static_cast<T*>(p.state) + static_cast<long long>(p.slot[row]) * p.pitch : nullptr;
    const bool fresh = mu && p.ctx[row] == 1;
    for (int c = tid * V; c < p.width; c += step) {
      float x[V], w[V], o[V];
      ldv<V>(z + c, x);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] = (x[i] - mean) * r;
      ldv<V>(static_cast<const T*>(p.nw[0]) + c, w);
#pragma unroll
      for (int i = 0; i < V; ++i) o[i] = x[i] * w[i];
      if (mu) {
        float before[V], m[V];
#pragma unroll
        for (int i = 0; i < V; ++i) before[i] = 0.f;
        if (!fresh) ldv<V>(state + c, before);
        ldv<V>(mu + c, m);
        stv<V>(state + c, o);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          const float n = round_to<T>(o[i]);
          o[i] = n + (before[i] - n) * m[i];
        }
      }
      stv<V>(out0 + c, o);
      if (p.n_out > 1) {
        ldv<V>(static_cast<const T*>(p.nw[1]) + c, w);
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] *= w[i];
        stv<V>(static_cast<T*>(p.out[1]) + row * p.pitch + c, x);
      }
    }
  }
  for (int c = p.width + tid; c < p.pitch; c += SS_WARPS * 32)
    for (int k = 0; k < p.n_out; ++k) st(static_cast<T*>(p.out[k]) + row * p.pitch + c, 0.f);
}

// One CTA per row.  The CTA of a segment's first row reads the state and then replaces it by the segment's last row.
struct TokenShiftParams {
  const void* n;             // [rows][pitch]
  const void* mu;            // [pitch]
  void* state;               // [slots][pitch]
  void* out;                 // [rows][pitch]
  const int* slot;           // [segments]
  const int* ctx;
  const int* cu;
  const int* seg_of;         // [rows]
  int pitch;
};
template <typename T>
__global__ void __launch_bounds__(256) token_shift_kernel(const TokenShiftParams p) {
  const long long t = blockIdx.x;
  const int s = p.seg_of[t], lo = p.cu[s], hi = p.cu[s + 1];
  const bool first = t == lo, fresh = first && p.ctx[s] == hi - lo;
  const T* n = static_cast<const T*>(p.n);
  T* state = static_cast<T*>(p.state) + static_cast<long long>(p.slot[s]) * p.pitch;
  for (int c = threadIdx.x * 8; c < p.pitch; c += blockDim.x * 8) {
    F8 x = ld8(n + t * p.pitch + c), before;
    const F8 mu = ld8(static_cast<const T*>(p.mu) + c);
    if (first) {
#pragma unroll
      for (int i = 0; i < 8; ++i) before.v[i] = 0.f;
      if (!fresh) before = ld8(state + c);
      st8(state + c, hi - lo == 1 ? x : ld8(n + static_cast<long long>(hi - 1) * p.pitch + c));
    } else {
      before = ld8(n + (t - 1) * p.pitch + c);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) x.v[i] += (before.v[i] - x.v[i]) * mu.v[i];
    st8(static_cast<T*>(p.out) + t * p.pitch + c, x);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) side_gate_kernel(const T* __restrict__ z, int ldz, const T* __restrict__ embed, long long lde, const long long* __restrict__ tok,
                                                        int vocab, T* __restrict__ out, int rows, int dim, int pitch) {
  constexpr bool kExact = IsExact<T>::v;
  const long long i = (static_cast<long long>(blockIdx.x) * 256 + threadIdx.x) * V;
  if (i >= static_cast<long long>(rows) * pitch) return;
  const long long t = i / pitch;
  const int c = static_cast<int>(i - t * pitch);
  const long long id = tok[t];
  float v[V];
#pragma unroll
  for (int k = 0; k < V; ++k) v[k] = 0.f;
  if (c < dim && id >= 0 && id < vocab) {
    float g[V], e[V];
    ldv<V>(z + t * ldz + c, g);
    ldv<V>(embed + id * lde + c, e);
#pragma unroll
    for (int k = 0; k < V; ++k)      // 0.5 (1 + tanh(u)) = sigmoid(2 u); 2 sqrt(2 / pi)
      v[k] = g[k] * sigmoid<kExact>(1.5957691216057308f * (g[k] + 0.044715f * g[k] * g[k] * g[k])) * e[k];
  }
  stv<V>(out + i, v);
}

__global__ void softcap_kernel(float* __restrict__ z, long long n4, float cap) {
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n4; i += static_cast<long long>(gridDim.x) * blockDim.x) {
    float4 v = reinterpret_cast<float4*>(z)[i];
    v.x = cap * tanhf(v.x / cap);
    v.y = cap * tanhf(v.y / cap);
    v.z = cap * tanhf(v.z / cap);
    v.w = cap * tanhf(v.w / cap);
    reinterpret_cast<float4*>(z)[i] = v;
  }
}

}  // namespace stack
}  // namespace rb

using namespace rb;
using namespace rb::stack;
typedef __nv_bfloat16 bf16;

// y0 / y1 may be null (y1 only with y0), and so may their norms' weights (both or none), ex, n0 / n1 (h0 is then a copy of the stream) and
// mu (see StreamStepParams)
extern "C" int rb_stream_step(float* res, const void* y0, int ldy0, const void* y1, int ldy1, const void* w0, const void* w1, const void* ex, int ldx,
                              const int* expert, const int* place, const int* offset, const float* weight, int top, const void* n0, const void* n1,
                              void* h0, void* h1, const void* mu, void* state, const int* slot, const int* ctx, int rows, int pitch, int width, float eps,
                              int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (width < 1 || pitch < width || pitch % 8 || !h0 || (y1 && !y0) || (w0 && !y0) || (y1 && !w0 != !w1) || (n1 && (!n0 || !h1))) return -2;
  if ((y0 && (ldy0 % 8 || ldy0 < width)) || (y1 && (ldy1 % 8 || ldy1 < width)) || (ex && (ldx % 8 || ldx < width || top < 1 || top > SS_MAX_TOP))) return -2;
  if (mu && (!n0 || !state || !slot || !ctx)) return -2;
  StreamStepParams p{res, {y0, y1}, {w0, w1}, ex, expert, place, offset, weight, {n0, n1}, {h0, h1}, mu, state, slot, ctx, {ldy0, ldy1}, ldx, top, pitch, width,
                     y0 ? (y1 ? 2 : 1) : 0, n1 ? 2 : 1, eps};
  const bool vec = width % 8 == 0;
  const size_t smem = n0 ? static_cast<size_t>(width) * 4 : 0;
  auto k = fp32 ? (vec ? stream_step_kernel<float, 8> : stream_step_kernel<float, 1>) : (vec ? stream_step_kernel<bf16, 8> : stream_step_kernel<bf16, 1>);
  if (smem > 40 * 1024) {
    if (smem > 200 * 1024) return -2;
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  k<<<rows, SS_WARPS * 32, smem, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_token_shift(const void* n, const void* mu, void* state, void* out, const int* slot, const int* ctx, const int* cu, const int* seg_of,
                              int rows, int pitch, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (pitch % 8) return -2;
  TokenShiftParams p{n, mu, state, out, slot, ctx, cu, seg_of, pitch};
  const int thr = pitch / 8 < 256 ? (pitch / 8 + 31) / 32 * 32 : 256;
  if (fp32) token_shift_kernel<float><<<rows, thr, 0, stm>>>(p);
  else token_shift_kernel<bf16><<<rows, thr, 0, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

// embed points at the layer's first feature; out [rows][pitch], columns behind dim are zero
extern "C" int rb_side_gate(const void* z, int ldz, const void* embed, long long lde, const long long* tok, int vocab, void* out, int rows, int dim,
                            int pitch, int fp32, cudaStream_t stm) {
  if (rows <= 0) return 0;
  if (dim < 1 || pitch < dim || ldz < dim || lde < dim) return -2;
  const bool vec = dim % 8 == 0 && ldz % 8 == 0 && lde % 8 == 0 &&
                   (reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(embed) | reinterpret_cast<uintptr_t>(out)) % 16 == 0;
  const long long n = static_cast<long long>(rows) * pitch / (vec ? 8 : 1);
  const unsigned grid = static_cast<unsigned>((n + 255) / 256);
  auto run = [&](auto kernel, auto type) {
    using T = decltype(type);
    kernel<<<grid, 256, 0, stm>>>((const T*)z, ldz, (const T*)embed, lde, tok, vocab, (T*)out, rows, dim, pitch);
  };
  if (fp32) vec ? run(side_gate_kernel<float, 8>, float()) : run(side_gate_kernel<float, 1>, float());
  else vec ? run(side_gate_kernel<bf16, 8>, bf16()) : run(side_gate_kernel<bf16, 1>, bf16());
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_softcap(float* z, long long n, float cap, cudaStream_t stm) {
  if (n <= 0) return 0;
  if (n % 4 || cap <= 0.f || reinterpret_cast<uintptr_t>(z) % 16) return -2;
  long long blocks = (n / 4 + 255) / 256;
  if (blocks > num_sms() * 16LL) blocks = num_sms() * 16LL;
  softcap_kernel<<<static_cast<unsigned>(blocks), 256, 0, stm>>>(z, n / 4, cap);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}
