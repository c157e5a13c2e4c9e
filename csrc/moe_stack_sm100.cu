// Routing of composed stacks' expert layers, their ungated activation, and a CUDA-core grouped GEMM for the 32-bit mode (ungated or gated
// experts).
// Compiled WITHOUT fast-math: scores are correctly rounded fp32 in both modes.
#include <limits.h>

#include "stack_common.cuh"

namespace rb {
namespace stack {

struct RouteParams {
  const float* logits;      // [T][ld]: E experts, then N - E identity experts (chosen and weighted alike, but without rows)
  const void* correction;   // [N] offsets of the scores for the choice, or null
  int corr_fp32;
  int* expert;              // [T][top]
  float* weight;            // [T][top]
  int* place;               // [T][top] row of the choice among its expert's rows
  int* row_token;           // [E][T] token of an expert's rows
  int* count;               // [E + 1] zeros: rows per expert, then the number of finished CTAs
  int* offset;              // [E + 1] first sorted row of every expert
  int4* tiles;              // [cap]: expert, first sorted row, rows, number inside the expert
  int* n_tiles;
  int T, ld, E, N, groups, keep, group_best, top, tile_rows, cap, renormalize, softmax;
  float weight_scale;
};
constexpr int RT_WARPS = 8;

// Integers that order like the floats they stand for; kTaken is below all of them.
constexpr int kTaken = INT_MIN;
__device__ __forceinline__ int order_key(float x) {
  const int b = __float_as_int(x);
  return b >= 0 ? b : b ^ 0x7fffffff;
}
// index of the largest of x[0 .. n), the first one among equals (0 when all are taken); every lane returns it
__device__ __forceinline__ int warp_argmax(const int* x, int n, int lane) {
  int best = kTaken, at = n;
  for (int i = lane; i < n; i += 32) {
    const int b = x[i];
    if (b > best) { best = b; at = i; }
  }
  const int top = __reduce_max_sync(0xffffffffu, best);
  at = __reduce_min_sync(0xffffffffu, best == top ? at : n);
  return at < n ? at : 0;
}

// One warp per row chooses its experts; the last CTA to finish lays the experts' rows out and writes the tile list.
__global__ void __launch_bounds__(RT_WARPS * 32) moe_route_kernel(const RouteParams p) {
  extern __shared__ float sm[];                 // [warps][2 N + groups]: scores, keys of the choice, keys of the groups
  __shared__ int s_last;
  __shared__ int s_sum[2][RT_WARPS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long t = static_cast<long long>(blockIdx.x) * RT_WARPS + warp;
  float* sc = sm + warp * (2 * p.N + p.groups);
  int* key = reinterpret_cast<int*>(sc + p.N);
  int* gs = key + p.N;
  if (t < p.T) {
    const float* z = p.logits + t * p.ld;
    if (p.softmax) {
      float m = -INFINITY, sum = 0.f;
      for (int e = lane; e < p.N; e += 32) m = fmaxf(m, z[e]);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      for (int e = lane; e < p.N; e += 32) {
        sc[e] = expf(z[e] - m);
        sum += sc[e];
      }
      sum = wsum(sum);
      for (int e = lane; e < p.N; e += 32) sc[e] /= sum;
    } else {
      for (int e = lane; e < p.N; e += 32) sc[e] = sigmoid<true>(z[e]);
    }
    for (int e = lane; e < p.N; e += 32) {      // (the lane's own scores)
      float s = sc[e] >= 0.f ? sc[e] : 0.f;     // a NaN counts as zero
      sc[e] = s;
      if (p.correction) s += p.corr_fp32 ? static_cast<const float*>(p.correction)[e] : ld(static_cast<const __nv_bfloat16*>(p.correction) + e);
      key[e] = order_key(s);
    }
    __syncwarp();
    const int n = p.N / p.groups;
    if (p.keep < p.groups) {
      for (int g = lane; g < p.groups; g += 32) {      // a group counts with its best score, or with the sum of its two best
        int a = kTaken, b = kTaken;
#pragma unroll 4
        for (int i = 0; i < n; ++i) {
          const int s = key[g * n + i];
          if (s > a) { b = a; a = s; }
          else if (s > b) b = s;
        }
        if (p.group_best == 2 && n > 1) {
          const float x = __int_as_float(a >= 0 ? a : a ^ 0x7fffffff), y = __int_as_float(b >= 0 ? b : b ^ 0x7fffffff);
          a = order_key(x + y);
        }
        gs[g] = a;
      }
      __syncwarp();
      for (int k = 0; k < p.keep; ++k) {
        const int g = warp_argmax(gs, p.groups, lane);
        __syncwarp();
        if (lane == 0) gs[g] = kTaken;
        __syncwarp();
      }
      for (int e = lane; e < p.N; e += 32)
        if (gs[e / n] != kTaken) key[e] = kTaken;
      __syncwarp();
    }
    float mine[2] = {0.f, 0.f}, sum = 0.f;       // choices lane and lane + 32 (top <= 64)
    int id[2] = {0, 0};
    for (int k = 0; k < p.top; ++k) {
      const int e = warp_argmax(key, p.N, lane);
      const float s = sc[e];
      __syncwarp();
      if (lane == 0) key[e] = kTaken;
      __syncwarp();
      sum += s;
      if (lane == (k & 31)) { mine[k >> 5] = s; id[k >> 5] = e; }
    }
    const float f = p.weight_scale / (p.renormalize ? sum + 1e-20f : 1.f);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int k = lane + 32 * j;
      if (k < p.top) {
        const bool rows = id[j] < p.E;           // identity experts have none
        const int at = rows ? atomicAdd(p.count + id[j], 1) : 0;
        const long long i = t * p.top + k;
        p.expert[i] = id[j];
        p.weight[i] = mine[j] * f;
        p.place[i] = at;
        if (rows && at < p.T) p.row_token[static_cast<long long>(id[j]) * p.T + at] = static_cast<int>(t);
      }
    }
    __threadfence();
  }
  __syncthreads();
  if (gridDim.x > 1) {
    if (threadIdx.x == 0) {
      __threadfence();
      s_last = atomicAdd(p.count + p.E, 1) == static_cast<int>(gridDim.x) - 1;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
  }
  // ---- rows and tiles in front of every expert: each thread takes a run of experts
  const int per = (p.E + RT_WARPS * 32 - 1) / (RT_WARPS * 32);
  const int e0 = min(p.E, static_cast<int>(threadIdx.x) * per), e1 = min(p.E, e0 + per);
  int rows = 0, tiles = 0;
  for (int e = e0; e < e1; ++e) {
    const int c = __ldcg(p.count + e);
    rows += c;
    tiles += (c + p.tile_rows - 1) / p.tile_rows;
  }
  int row = rows, tile = tiles;                  // inclusive sums over the warp, then over the warps
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int a = __shfl_up_sync(0xffffffffu, row, o), b = __shfl_up_sync(0xffffffffu, tile, o);
    if (lane >= o) { row += a; tile += b; }
  }
  if (lane == 31) { s_sum[0][warp] = row; s_sum[1][warp] = tile; }
  __syncthreads();
  for (int w = 0; w < warp; ++w) { row += s_sum[0][w]; tile += s_sum[1][w]; }
  if (threadIdx.x == RT_WARPS * 32 - 1) {
    p.offset[p.E] = row;
    *p.n_tiles = tile;
  }
  row -= rows;
  tile -= tiles;
  for (int e = e0; e < e1; ++e) {
    const int c = __ldcg(p.count + e);
    p.offset[e] = row;
    for (int i = 0; i * p.tile_rows < c; ++i, ++tile)
      if (tile < p.cap) p.tiles[tile] = make_int4(e, row + i * p.tile_rows, min(p.tile_rows, c - i * p.tile_rows), i);
    row += c;
  }
}

template <typename T>
__global__ void relu2_kernel(T* __restrict__ x, long long n8) {
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n8; i += static_cast<long long>(gridDim.x) * blockDim.x) {
    F8 v = ld8(x + i * 8);
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const float a = fmaxf(v.v[k], 0.f);
      v.v[k] = a * a;
    }
    st8(x + i * 8, v);
  }
}

// C[sorted row] = act(A[token or sorted row] * B[expert]^T); one tile of the list (up to 64 rows) x 64 columns per CTA.  act 0: none,
// 1: squared relu, 2 and 3: gated (columns of B alternate between 32 gates and the 32 units they belong to; C has half as many)
struct MoeSimtParams {
  const void* A;
  const void* B;             // [E][N][K]
  void* C;                   // [sorted rows][N]
  const int4* tiles;
  const int* n_tiles;
  const int* row_token;      // [E][capacity] or null
  int capacity, cap, N, K, act;
  float limit;               // act 2: g = min(gate, limit), u = unit clamped to +- limit, g sigmoid(1.702 g) (u + 1); act 3: silu(gate) unit
};
template <typename T>
__global__ void __launch_bounds__(256) moe_simt_kernel(const MoeSimtParams p) {
  __shared__ float sa[16][64 + 4], sb[16][64 + 4];
  __shared__ long long s_src[64];
  if (static_cast<int>(blockIdx.y) >= min(*p.n_tiles, p.cap)) return;
  const int4 tile = p.tiles[blockIdx.y];
  const int tid = threadIdx.x, n0 = blockIdx.x * 64;
  if (tid < 64) {
    long long r = tile.y + tid;
    if (p.row_token && tid < tile.z) r = p.row_token[static_cast<long long>(tile.x) * p.capacity + tile.w * 64 + tid];
    s_src[tid] = r * p.K;
  }
  __syncthreads();
  const T* A = static_cast<const T*>(p.A);
  const T* B = static_cast<const T*>(p.B) + static_cast<long long>(tile.x) * p.N * p.K;
  const int tm = (tid >> 4) * 4, tn = (tid & 15) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + i * 256, r = e >> 4, k = e & 15;
      sa[k][r] = (r < tile.z && k0 + k < p.K) ? ld(A + s_src[r] + k0 + k) : 0.f;
      sb[k][r] = (n0 + r < p.N && k0 + k < p.K) ? ld(B + static_cast<long long>(n0 + r) * p.K + k0 + k) : 0.f;
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
  T* C = static_cast<T*>(p.C);
  if (p.act >= 2) {
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {      // the thread eight lanes on holds the units of this thread's gates
        float u = __shfl_down_sync(0xffffffffu, acc[i][j], 8), g = acc[i][j];
        if (p.act == 2) {
          u = fminf(fmaxf(u, -p.limit), p.limit) + 1.f;
          g = fminf(g, p.limit);
          g *= sigmoid<true>(1.702f * g);
        } else {
          g *= sigmoid<true>(g);
        }
        if (tn < 32 && tm + i < tile.z) st(C + static_cast<long long>(tile.y + tm + i) * (p.N >> 1) + (n0 >> 1) + tn + j, g * u);
      }
    return;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (tm + i < tile.z && n0 + tn + j < p.N) {
        float v = acc[i][j];
        if (p.act) {
          v = fmaxf(v, 0.f);
          v *= v;
        }
        st(C + static_cast<long long>(tile.y + tm + i) * p.N + n0 + tn + j, v);
      }
}

}  // namespace stack
}  // namespace rb

using namespace rb;
using namespace rb::stack;
typedef __nv_bfloat16 bf16;

// count [E + 1] must be zero and is left used.  cap: room in `tiles`, at least min(T top, E) + T top / tile_rows.  N outputs: E experts and
// N - E identity experts; correction [N] or null; softmax: scores over all N outputs, else sigmoids; group_best: 1 or 2
extern "C" int rb_moe_route(const float* logits, int ld, const void* correction, int corr_fp32, int* expert, float* weight, int* place, int* row_token,
                            int* count, int* offset, int* tiles, int* n_tiles, int T, int E, int N, int groups, int keep, int group_best, int top,
                            int tile_rows, int cap, int renormalize, int softmax, float weight_scale, cudaStream_t stm) {
  if (T <= 0) return 0;
  if (E < 1 || N < E || ld < N || groups < 1 || N % groups || keep < 1 || keep > groups || top < 1 || top > 64 || top > N / groups * keep ||
      tile_rows < 1 || group_best < 1 || group_best > 2)
    return -2;
  const size_t smem = static_cast<size_t>(RT_WARPS) * (2 * N + groups) * 4;
  if (smem > 200 * 1024) return -2;
  if (smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  RouteParams p{logits, correction, corr_fp32, expert, weight, place, row_token, count, offset, reinterpret_cast<int4*>(tiles), n_tiles, T, ld, E, N,
                groups, keep, group_best, top, tile_rows, cap, renormalize, softmax, weight_scale};
  moe_route_kernel<<<(T + RT_WARPS - 1) / RT_WARPS, RT_WARPS * 32, smem, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int rb_relu2(void* x, long long n, int fp32, cudaStream_t stm) {
  if (n <= 0) return 0;
  if (n % 8) return -2;
  long long blocks = (n / 8 + 255) / 256;
  if (blocks > num_sms() * 16LL) blocks = num_sms() * 16LL;
  if (fp32) relu2_kernel<float><<<static_cast<unsigned>(blocks), 256, 0, stm>>>((float*)x, n / 8);
  else relu2_kernel<bf16><<<static_cast<unsigned>(blocks), 256, 0, stm>>>((bf16*)x, n / 8);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

// the tile list must have been made with 64 rows per tile
extern "C" int rb_moe_simt(const void* A, const void* B, void* C, const int* tiles, const int* n_tiles, const int* row_token, int capacity, int cap,
                           int N, int K, int act, float limit, int fp32, cudaStream_t stm) {
  if (cap <= 0) return 0;
  if (cap > 65535 || N < 1 || K < 1 || act < 0 || act > 3 || (act >= 2 && N % 64)) return -2;
  MoeSimtParams p{A, B, C, reinterpret_cast<const int4*>(tiles), n_tiles, row_token, capacity, cap, N, K, act, limit};
  const dim3 grid((N + 63) / 64, cap);
  if (fp32) moe_simt_kernel<float><<<grid, 256, 0, stm>>>(p);
  else moe_simt_kernel<bf16><<<grid, 256, 0, stm>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}
