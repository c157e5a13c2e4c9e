// One small GEMM per head on the tensor cores: out[t][h][:] = x[t][h][:] * W_h, for all tokens and heads in one launch.
//
// This folds a latent up-projection into the queries (W_h [K][N], read MN-major in place) and applies one to attended
// latent rows (W_h [N][K]).  CTA = (128 output features, head, 128 tokens): TMA warp (64-deep stages, A through a
// 3-D map so that x may be a strided slice of a wider projection), MMA warp, four epilogue warps that write rows of the
// output directly, multiplied by the sigmoid of a gate per output feature when one is given.  The reductions are short (one to eight stages), so CTAs are small and several share an SM.
#include "common.cuh"
#include "host_utils.h"

namespace rb {
namespace hg {

constexpr int STAGES = 3;
constexpr int A_BYTES = 128 * 128;        // 128 tokens x 64 k
constexpr int STAGE = 2 * A_BYTES;
constexpr int THREADS = 192;
constexpr int BAR = STAGES * STAGE;
constexpr int TOTAL = BAR + 256;

struct Params {
  __nv_bfloat16* out;      // [T][H][N]
  const __nv_bfloat16* gate;      // [T][ld_gate], head h's features at h * N, or null
  int T, H, N, K, kn, ld_gate;
  int* err;
};

__global__ void __launch_bounds__(THREADS, 2)
head_gemm_kernel(const __grid_constant__ CUtensorMap tma_x, const __grid_constant__ CUtensorMap tma_w, const Params p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + BAR);
  uint64_t* empty = full + STAGES;
  uint64_t* done = empty + STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * 128, h = blockIdx.y, t0 = blockIdx.z * 128;
  const int steps = (p.K + 63) / 64;
  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    mbar_init(done, 1);
    *abort_flag = 0;
    if ((smem_u32(smem) & 1023u) != 0) {
      *abort_flag = 1;
      if (p.err) atomicCAS(p.err, kOk, kErrBadArgument);
    }
    fence_barrier_init();
  }
  if (warp == 5) {
    tmem_alloc<128>(tmem_slot);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const bool dead = (*abort_flag != 0);
  if (warp == 4) {
    if (lane == 0 && !dead) {
      for (int k = 0; k < steps; ++k) {
        const int s = k % STAGES;
        if (!mbar_wait(&empty[s], (static_cast<uint32_t>(k / STAGES) & 1) ^ 1, abort_flag, p.err)) break;
        uint8_t* a = smem + s * STAGE;
        uint8_t* b = a + A_BYTES;
        mbar_expect_tx(&full[s], STAGE);
        tma_load_3d(a, &tma_x, &full[s], k * 64, h, t0);      // features behind K and tokens behind T come in as zeros
        if (!p.kn) {
          tma_load_2d(b, &tma_w, &full[s], k * 64, h * p.N + n0);
        } else {      // rows behind this head's K meet zero features of x
          tma_load_2d(b, &tma_w, &full[s], n0, h * p.K + k * 64);
          tma_load_2d(b + 8192, &tma_w, &full[s], n0 + 64, h * p.K + k * 64);
        }
      }
    }
  } else if (warp == 5) {
    if (lane == 0 && !dead) {
      const uint32_t idesc = make_idesc_f16(128, 128, true, false, p.kn != 0);
      bool ok = true;
      for (int k = 0; k < steps && ok; ++k) {
        const int s = k % STAGES;
        ok = mbar_wait(&full[s], static_cast<uint32_t>(k / STAGES) & 1, abort_flag, p.err);
        if (!ok) break;
        tc_fence_after();
        const uint32_t a = smem_u32(smem + s * STAGE), b = a + A_BYTES;
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          const uint64_t da = make_smem_desc(a + kk * 32, 16, 1024, kSwizzle128B);
          const uint64_t db = p.kn ? make_smem_desc(b + kk * 2048, 8192, 1024, kSwizzle128B) : make_smem_desc(b + kk * 32, 16, 1024, kSwizzle128B);
          umma_f16(tmem_base, da, db, idesc, (k > 0 || kk > 0) ? 1u : 0u);
        }
        umma_commit(&empty[s]);
      }
      if (ok) umma_commit(done);
    }
  } else {
    const int t = t0 + warp * 32 + lane;
    // gates of 32 columns at a time are fetched ahead of their use
    const __nv_bfloat16* gate = p.gate && t < p.T ? p.gate + static_cast<size_t>(t) * p.ld_gate + h * p.N + n0 : nullptr;
    uint4 g[4];
    auto fetch = [&](int c) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (gate && c < 128 && n0 + c + i * 8 < p.N) g[i] = *reinterpret_cast<const uint4*>(gate + c + i * 8);
    };
    fetch(0);
    const bool ok = !dead && mbar_wait(done, 0, abort_flag, p.err);
    __syncwarp();
    tc_fence_after();
    __nv_bfloat16* out = p.out + (static_cast<size_t>(t) * p.H + h) * p.N + n0;
#pragma unroll 1
    for (int c = 0; c < 128; c += 32) {
      if (n0 + c >= p.N) break;
      uint32_t r[32];
      tmem_ld_32x32b_x32(tmem_base + c + (static_cast<uint32_t>(warp * 32) << 16), r);
      tmem_wait_ld();
      if (ok && t < p.T) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (n0 + c + i * 8 < p.N) {      // N is a multiple of 8
            if (gate) {
              const uint32_t w[4] = {g[i].x, g[i].y, g[i].z, g[i].w};
#pragma unroll
              for (int k = 0; k < 4; ++k) {
                r[8 * i + 2 * k] = __float_as_uint(__fdividef(__uint_as_float(r[8 * i + 2 * k]), 1.f + __expf(-__uint_as_float(w[k] << 16))));
                r[8 * i + 2 * k + 1] = __float_as_uint(__fdividef(__uint_as_float(r[8 * i + 2 * k + 1]), 1.f + __expf(-__uint_as_float(w[k] & 0xffff0000u))));
              }
            }
            uint4 v;
            v.x = pack_bf16(__uint_as_float(r[8 * i]), __uint_as_float(r[8 * i + 1]));
            v.y = pack_bf16(__uint_as_float(r[8 * i + 2]), __uint_as_float(r[8 * i + 3]));
            v.z = pack_bf16(__uint_as_float(r[8 * i + 4]), __uint_as_float(r[8 * i + 5]));
            v.w = pack_bf16(__uint_as_float(r[8 * i + 6]), __uint_as_float(r[8 * i + 7]));
            *reinterpret_cast<uint4*>(out + c + i * 8) = v;
          }
        }
      }
      fetch(c + 32);
    }
  }
  if (*abort_flag) __nanosleep(50000);
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc<128>(tmem_base);
  }
}

}  // namespace hg
}  // namespace rb

// x [T][H][K] bf16 with strides x_tok, x_head (elements, multiples of 8); w [H][N][K] (kn = 0) or [H][K][N] (kn = 1),
// contiguous; out [T][H][N] contiguous.  gate [T][ld_gate >= H N] or null.  N and K are multiples of 8; returns -20 otherwise.
extern "C" int rb_head_gemm(const void* x, const void* w, const void* gate, int ld_gate, void* out, int T, int H, int N, int K, long long x_tok,
                            long long x_head, int kn, int* err, cudaStream_t st) {
  using namespace rb;
  using namespace rb::hg;
  if (T <= 0 || H <= 0) return 0;
  if (N % 8 || K % 8 || x_tok % 8 || x_head % 8 || N < 8 || K < 8 || H > 65535 || (T + 127) / 128 > 65535) return -20;
  if ((reinterpret_cast<uintptr_t>(x) % 16) || (reinterpret_cast<uintptr_t>(w) % 16) || (reinterpret_cast<uintptr_t>(out) % 16)) return -20;
  if (gate && (ld_gate % 8 || ld_gate < H * N || reinterpret_cast<uintptr_t>(gate) % 16)) return -2;
  CUtensorMap tx, tw;
  int rc = encode_tma_3d_16bit(&tx, x, K, H, T, x_head, x_tok, 64, 1, 128);
  if (rc) return rc;
  rc = kn ? encode_tma_2d_bf16(&tw, w, N, static_cast<uint64_t>(H) * K, N, 64, 64) : encode_tma_2d_bf16(&tw, w, K, static_cast<uint64_t>(H) * N, K, 64, 128);
  if (rc) return rc;
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(head_gemm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, TOTAL);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr = true;
  }
  Params p{static_cast<__nv_bfloat16*>(out), static_cast<const __nv_bfloat16*>(gate), T, H, N, K, kn, ld_gate, err};
  head_gemm_kernel<<<dim3((N + 127) / 128, H, (T + 127) / 128), THREADS, TOTAL, st>>>(tx, tw, p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}
