// Grouped GEMM of routed experts for serving on sm_100a: Y[row] = act(X[source(row)] * W[expert(row)]^T), ONE launch for all experts.
//
// Rows of one expert lie side by side in the sorted order; the tile list (expert, first sorted row, rows, tile number inside the
// expert) was written by the routing kernel, so nothing about the routing is known on the host: the grid is persistent and walks
// the list.  The first product GATHERS its rows: the token indices of an expert's rows are read from the routing kernel's table and
// fetched with TMA gather4 (four rows per instruction, all 32 lanes of the producer warp issue), so no sorted copy of the
// activations is ever made and padding rows cost no traffic.  The second product reads the sorted rows of the first.  The
// activation is applied in the epilogue; for gated experts the weight rows alternate between 32 gates and the 32 units they belong
// to, so both accumulators of an output are columns of the same tile.
//
// Tiles of 128 rows x BN columns (64: decode, so that few experts still fill the machine; 128; 256: prompts); fp32 accumulators in
// TMEM, double buffered.  Warp 0 = TMA, warp 1 = MMA and TMEM, warps 2..5 = epilogue.  Every wait is bounded; no load uses
// cluster multicast.
#include "common.cuh"
#include "host_utils.h"

namespace rb {
namespace mg {

constexpr int BM = 128;
constexpr int BK = 64;
constexpr int THREADS = 192;
constexpr int COPIERS = 128;                   // threads of the row copies (kCopy)
constexpr int LAG = 2;                         // stages whose row copies are in flight behind the newest one
constexpr int kABytes = BM * BK * 2;
enum : int { kSorted = 0, kGather4 = 1, kCopy = 2 };      // source of the A rows

template <int BN>
struct Cfg {
  static constexpr int kStages = BN == 256 ? 4 : 6;
  static_assert(kStages > LAG, "the copiers arrive LAG stages late");
  static constexpr int kBBytes = BN * BK * 2;
  static constexpr int kStage = kABytes + kBBytes;
  static constexpr int kBar = kStages * kStage;
  static constexpr int kTotal = kBar + 256 + 1024;
  static constexpr int kTmemCols = 2 * BN;
};

struct Params {
  const int4* tiles;         // [cap]: expert, first sorted row, rows (1 .. 128), number of the tile inside its expert
  const int* n_tiles;        // device counter
  const int* row_token;      // [E][capacity] token of an expert's rows; null: the sorted rows themselves
  int capacity, cap, N, K, act;
  float limit;               // act 2 (gated): g = min(gate, limit), u = unit clamped to +- limit, g sigmoid(1.702 g) (u + 1); act 3: silu(gate) unit
  const __nv_bfloat16* x;    // [x_rows][K] (kCopy)
  __nv_bfloat16* out;        // [sorted rows][N], act 2: [N / 2]
  int* err;
};

__device__ __forceinline__ void tma_gather4(void* dst, const CUtensorMap* m, uint64_t* bar, int x, const int4& r) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile::gather4.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6, %7}], [%2];"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(r.x), "r"(r.y), "r"(r.z), "r"(r.w)
      : "memory");
}

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

template <int BN, int SRC>
__global__ void __launch_bounds__(SRC == kCopy ? THREADS + COPIERS : THREADS, 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap tma_a, const __grid_constant__ CUtensorMap tma_b, const Params p) {
  using C = Cfg<BN>;
  constexpr int kStages = C::kStages;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + C::kBar);
  uint64_t* empty_bar = full_bar + kStages;
  uint64_t* tfull_bar = empty_bar + kStages;   // [2]
  uint64_t* tempty_bar = tfull_bar + 2;        // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tempty_bar + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  const int tiles_n = (p.N + BN - 1) / BN;
  const int total = min(*p.n_tiles, p.cap) * tiles_n;
  const int k_iters = p.K / BK;

  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) { mbar_init(&full_bar[s], SRC == kCopy ? 1 + COPIERS : 1); mbar_init(&empty_bar[s], 1); }
    for (int a = 0; a < 2; ++a) { mbar_init(&tfull_bar[a], 1); mbar_init(&tempty_bar[a], 4); }
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc<C::kTmemCols>(tmem_slot);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer (gather4: the whole warp)
    if (lane == 0) {
      if constexpr (SRC != kCopy) tma_prefetch_desc(&tma_a);
      tma_prefetch_desc(&tma_b);
    }
    int s = 0;
    uint32_t ph = 0;
    bool ok = true;
    for (int t = blockIdx.x; t < total && ok; t += gridDim.x) {
      const int m = t / tiles_n, n0 = (t - m * tiles_n) * BN;
      const int4 tile = p.tiles[m];
      int4 src = make_int4(0, 0, 0, 0);
      const int quads = (tile.z + 3) >> 2;
      if constexpr (SRC == kGather4) {
        // lane l brings rows 4 l .. 4 l + 3; behind the last row of the tile its token is repeated
        const int* tok = p.row_token + static_cast<long long>(tile.x) * p.capacity + tile.w * BM;
        const int last = tile.z - 1;
        if (lane < quads) src = make_int4(tok[min(4 * lane, last)], tok[min(4 * lane + 1, last)], tok[min(4 * lane + 2, last)], tok[min(4 * lane + 3, last)]);
      }
      for (int k = 0; k < k_iters; ++k) {
        if (ok) ok = mbar_wait(&empty_bar[s], ph ^ 1, abort_flag, p.err);
        if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
        uint8_t* sa = smem + s * C::kStage;
        if (lane == 0) {
          mbar_expect_tx(&full_bar[s], (SRC == kGather4 ? quads * 512 : (SRC == kSorted ? kABytes : 0)) + C::kBBytes);
          tma_load_2d(sa + kABytes, &tma_b, &full_bar[s], k * BK, tile.x * p.N + n0);
          if constexpr (SRC == kSorted) tma_load_2d(sa, &tma_a, &full_bar[s], k * BK, tile.y);
        }
        if constexpr (SRC == kGather4) {
          __syncwarp();
          if (lane < quads) tma_gather4(sa + lane * 512, &tma_a, &full_bar[s], k * BK, src);
        }
        if (++s == kStages) { s = 0; ph ^= 1; }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      const uint32_t idesc = make_idesc_f16(BM, BN, true, false, false);
      int s = 0, acc = 0;
      uint32_t ph = 0, acc_ph = 0;
      bool ok = true;
      for (int t = blockIdx.x; t < total && ok; t += gridDim.x) {
        if (!mbar_wait(&tempty_bar[acc], acc_ph ^ 1, abort_flag, p.err)) break;
        tc_fence_after();
        const uint32_t d_tmem = tmem_base + acc * BN;
        for (int k = 0; k < k_iters; ++k) {
          if (!mbar_wait(&full_bar[s], ph, abort_flag, p.err)) { ok = false; break; }
          tc_fence_after();
          const uint32_t sa = smem_u32(smem + s * C::kStage);
          const uint32_t sb = sa + kABytes;
#pragma unroll
          for (int kk = 0; kk < BK / 16; ++kk)
            umma_f16(d_tmem, make_smem_desc(sa + kk * 32, 16, 1024, kSwizzle128B), make_smem_desc(sb + kk * 32, 16, 1024, kSwizzle128B), idesc,
                     (k > 0 || kk > 0) ? 1u : 0u);
          umma_commit(&empty_bar[s]);
          if (++s == kStages) { s = 0; ph ^= 1; }
        }
        if (!ok) break;
        umma_commit(&tfull_bar[acc]);
        acc ^= 1;
        if (acc == 0) acc_ph ^= 1;
      }
    }
  } else if (SRC == kCopy && warp >= 6) {
    // ------------------------------------------------------------------ row copies: eight threads bring 128 bytes of one row
    const int i = threadIdx.x - THREADS, c = i & 7, r0 = i >> 3;
    const uint32_t sbase = smem_u32(smem);
    int s = 0, done = 0;
    uint32_t ph = 0;
    int pending = 0;
    bool ok = true;
    for (int t = blockIdx.x; t < total && ok; t += gridDim.x) {
      const int4 tile = p.tiles[t / tiles_n];
      const int* tok = p.row_token + static_cast<long long>(tile.x) * p.capacity + tile.w * BM;
      const __nv_bfloat16* src[BM / 16];
#pragma unroll
      for (int j = 0; j < BM / 16; ++j) {
        const int r = r0 + 16 * j;
        src[j] = r < tile.z ? p.x + static_cast<long long>(tok[r]) * p.K + c * 8 : nullptr;
      }
      for (int k = 0; k < k_iters; ++k) {
        if (!mbar_wait(&empty_bar[s], ph ^ 1, abort_flag, p.err)) { ok = false; break; }
        const uint32_t sa = sbase + s * C::kStage + ((c ^ (r0 & 7)) << 4);      // rows 16 apart share the swizzle
#pragma unroll
        for (int j = 0; j < BM / 16; ++j)
          if (src[j]) cp_async16(sa + (r0 + 16 * j) * 128, src[j] + k * BK);
        cp_async_commit();
        if (pending == LAG) {          // the stage LAG behind has landed: hand it to the tensor core's proxy
          cp_async_wait<LAG>();
          fence_proxy_async();
          mbar_arrive(&full_bar[done]);
          if (++done == kStages) done = 0;
        } else {
          ++pending;
        }
        if (++s == kStages) { s = 0; ph ^= 1; }
      }
    }
    cp_async_wait<0>();
    fence_proxy_async();
    for (; pending > 0; --pending) {
      mbar_arrive(&full_bar[done]);
      if (++done == kStages) done = 0;
    }
  } else {
    // ------------------------------------------------------------------ epilogue (warps 2..5)
    const int grp = warp & 3;
    int acc = 0;
    uint32_t acc_ph = 0;
    bool ok = true;
    for (int t = blockIdx.x; t < total; t += gridDim.x) {
      const int m = t / tiles_n, n0 = (t - m * tiles_n) * BN;
      const int4 tile = p.tiles[m];
      ok = mbar_wait(&tfull_bar[acc], acc_ph, abort_flag, p.err);
      if (!__all_sync(0xffffffffu, ok)) break;
      tc_fence_after();
      const int row = grp * 32 + lane;
      const bool live = row < tile.z;
      if (grp * 32 < tile.z) {
        const uint32_t taddr = tmem_base + acc * BN + (static_cast<uint32_t>(grp * 32) << 16);
        const bool gated = p.act >= 2;
        const int shift = gated ? 1 : 0, step = 1 + shift;
        __nv_bfloat16* out = p.out + static_cast<size_t>(tile.y + row) * (p.N >> shift) + (n0 >> shift);
#pragma unroll 1
        for (int c = 0; c < BN / 32; c += step) {
          if (n0 + c * 32 >= p.N) break;             // N is a multiple of 64
          uint32_t r[32];
          tmem_ld_32x32b_x32(taddr + c * 32, r);
          if (gated) {
            uint32_t v[32];
            tmem_ld_32x32b_x32(taddr + c * 32 + 32, v);
            tmem_wait_ld();
            if (p.act == 3) {
#pragma unroll
              for (int i = 0; i < 32; ++i) {
                const float g = __uint_as_float(r[i]);
                r[i] = __float_as_uint(__fdividef(g, 1.f + __expf(-g)) * __uint_as_float(v[i]));
              }
            } else {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const float g = fminf(__uint_as_float(r[i]), p.limit), u = fminf(fmaxf(__uint_as_float(v[i]), -p.limit), p.limit);
              r[i] = __float_as_uint(__fdividef(g, 1.f + __expf(-1.702f * g)) * (u + 1.f));
            }
            }
          } else {
            tmem_wait_ld();
          }
          if (p.act == 1) {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const float v = fmaxf(__uint_as_float(r[i]), 0.f);
              r[i] = __float_as_uint(v * v);
            }
          }
          if (live) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              uint4 o;
              o.x = pack_bf16(__uint_as_float(r[8 * i]), __uint_as_float(r[8 * i + 1]));
              o.y = pack_bf16(__uint_as_float(r[8 * i + 2]), __uint_as_float(r[8 * i + 3]));
              o.z = pack_bf16(__uint_as_float(r[8 * i + 4]), __uint_as_float(r[8 * i + 5]));
              o.w = pack_bf16(__uint_as_float(r[8 * i + 6]), __uint_as_float(r[8 * i + 7]));
              reinterpret_cast<uint4*>(out + (c >> shift) * 32)[i] = o;
            }
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tempty_bar[acc]);
      acc ^= 1;
      if (acc == 0) acc_ph ^= 1;
    }
  }

  if (*abort_flag) __nanosleep(50000);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc<C::kTmemCols>(tmem_base);
  }
}

template <int BN, int SRC>
static int launch(const void* X, int x_rows, const void* W, int E, const Params& p, cudaStream_t st) {
  using C = Cfg<BN>;
  CUtensorMap ta, tb;
  int rc = encode_tma_2d_bf16(&ta, X, p.K, x_rows, p.K, BK, SRC == kGather4 ? 1 : BM);
  if (rc) return rc;
  rc = encode_tma_2d_bf16(&tb, W, p.K, static_cast<uint64_t>(E) * p.N, p.K, BK, BN);
  if (rc) return rc;
  auto kern = moe_gemm_kernel<BN, SRC>;
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kTotal);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr = true;
  }
  const long long work = static_cast<long long>(p.cap) * ((p.N + BN - 1) / BN);
  kern<<<static_cast<unsigned>(work < num_sms() ? work : num_sms()), SRC == kCopy ? THREADS + COPIERS : THREADS, C::kTotal, st>>>(ta, tb, p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace mg
}  // namespace rb

// X [x_rows][K] (token rows with row_token [E][capacity], else sorted rows), W [E][N][K] -> out [sorted rows][N]; tiles hold at most
// `cap` entries.  act: 0 none, 1 squared relu, 2 and 3 gated (see Params::limit; out [sorted rows][N / 2]).  bn: 128 or 256 columns per tile.  full: most tiles have many rows (choice of the
// gather only).  N and K are multiples of 64.
extern "C" int rb_moe_gemm(const void* X, const void* W, void* out, const int* tiles, const int* n_tiles, const int* row_token, int x_rows,
                           int capacity, int cap, int E, int N, int K, int act, float limit, int bn, int full, int* err, cudaStream_t st) {
  using namespace rb;
  using namespace rb::mg;
  if (x_rows <= 0 || cap <= 0) return 0;
  if (E < 1 || N < 64 || K < 64 || N % 64 || K % 64 || act < 0 || act > 3 || (act >= 2 && N % 128) || reinterpret_cast<uintptr_t>(X) % 16) return -2;
  Params p{reinterpret_cast<const int4*>(tiles), n_tiles, row_token, capacity, cap, N, K, act, limit, (const __nv_bfloat16*)X, (__nv_bfloat16*)out, err};
  if (row_token && full) return bn == 256 ? launch<256, kCopy>(X, x_rows, W, E, p, st) : launch<128, kCopy>(X, x_rows, W, E, p, st);
  if (row_token) return bn == 256 ? launch<256, kGather4>(X, x_rows, W, E, p, st) : launch<128, kGather4>(X, x_rows, W, E, p, st);
  return bn == 256 ? launch<256, kSorted>(X, x_rows, W, E, p, st) : launch<128, kSorted>(X, x_rows, W, E, p, st);
}
