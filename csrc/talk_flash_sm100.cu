// Flash attention of prompt portions whose heads' weights are mixed afterwards, over paged keys and values: every head's weights meet the
// values of every group (see talk_decode_sm100.cu), out [rows][H][G][out_d].
//
// Tiles are those of paged_flash_sm100.cu (128 (token, head) rows of one key group, blocks of 64 positions straight from the pages), but a CTA
// keeps the accumulators of several groups' values (up to 384 columns of TMEM), so scores and softmax are computed once for all of
// them.  Scores are capped: the softmax has a fixed reference and nothing is rescaled; what a score costs is a polynomial and one
// exponential.  Two sets of eight warps (two threads per row) take the blocks in turn, so one set's latencies hide behind the other's
// arithmetic.  The CTAs are persistent: their blocks form one sequence across tiles, and the scores of the next tile are on their way
// while the last one's accumulators are read.  Warps 0-15: softmax and epilogue, warp 16: TMA, warp 17: MMA.  Every wait is bounded; no load
// uses cluster multicast.
#include <limits.h>

#include "common.cuh"
#include "host_utils.h"

namespace rb {
namespace tf {

constexpr int BQ = 128;
constexpr int BKV = 64;
constexpr int SOFT = 512;                 // softmax threads: two sets of two per row
constexpr int THREADS = SOFT + 64;
constexpr int kTmemCols = 512;
constexpr int T_S = 0;                    // two buffers of 64 columns
constexpr int T_O = 128;
constexpr int kQHalf = BQ * 128, kKVHalf = BKV * 128;      // bytes of 64 columns
constexpr int kPBytes = BQ * BKV * 2;

struct Params {
  const int* blocks;         // [n][4]: segment, first row, rows, position of the first row; null: row i is segment i, at ctx[i] - 1
  const int* ctx;            // [S]
  const int* block_tables;   // [S][max_blocks]
  const __nv_bfloat16* sink; // [H] or null
  __nv_bfloat16* out;        // [rows][H][Hkv][out_d]
  int H, Hkv, G, tokens, max_blocks, page, out_d, nv;      // G: heads per group; nv: value groups per item
  int n_items, slices;       // items: query tile, key group, slice of value groups (the last one fastest)
  int window, keep, chunk;   // as in paged_flash
  int v_at, p_at, bar_at;    // bytes into shared memory
  float cap_in;              // s = cap_log2 tanh(cap_in q . k), in log2 units
  float cap_log2;
  int* err;
};

// tanh(x) = x (t0 + t1 u + .. + t6 u^6), u = x^2, for |x| <= 1 up to 5e-8: interpolation of tanh(sqrt u) / sqrt u at Chebyshev points of [0, 1]
__device__ constexpr float kTanh[7] = {0.99999994865f, -0.33332827979f, 0.13325076146f, -0.05345164637f, 0.02027970829f, -0.00619432483f, 0.00103802510f};

__device__ __forceinline__ unsigned long long pair2(float a, float b) {
  unsigned long long d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(a), "f"(b));
  return d;
}
__device__ __forceinline__ void split2(unsigned long long v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
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

// One unit of work: a query tile, the group of its keys, and the value groups v0 .. v0 + nv - 1.
struct Item {
  int seg, row0, ntok, pos0, kvh, v0, nv, block0, n_kept, n_blocks;
  __device__ __forceinline__ Item(const Params& p, int i) {
    const int z = i % p.slices;
    i /= p.slices;
    kvh = i % p.Hkv;
    i /= p.Hkv;
    v0 = z * p.nv;
    nv = min(p.nv, p.Hkv - v0);
    if (p.blocks) {
      const int4 b = reinterpret_cast<const int4*>(p.blocks)[i];
      seg = b.x; row0 = b.y; ntok = b.z; pos0 = b.w;
    } else {
      seg = row0 = i;
      ntok = 1;
      pos0 = p.ctx[seg] - 1;
    }
    block0 = (p.chunk ? pos0 / p.chunk * p.chunk : max(0, pos0 - p.window + 1)) / BKV;
    n_kept = min((p.keep + BKV - 1) / BKV, block0);
    n_blocks = n_kept + (pos0 + ntok + BKV - 1) / BKV - block0;
  }
  __device__ __forceinline__ int first_position(int j) const { return (j < n_kept ? j : block0 + j - n_kept) * BKV; }
};

template <int DK, int DV>
__global__ void __launch_bounds__(THREADS, 1)
talk_flash_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k, const __grid_constant__ CUtensorMap tma_v,
                  const Params p) {
  constexpr int kQBytes = DK / 64 * kQHalf, kKBytes = DK / 64 * kKVHalf, kVBytes = DV / 64 * kKVHalf;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + p.bar_at);
  // blocks are numbered across items (g): index of a pair = g & 1, phase = g / 2; queries and accumulators by item
  uint64_t* qfull = bars;          // [2]
  uint64_t* qempty = bars + 2;     // [2] the scores of an item are complete
  uint64_t* bar_s = bars + 4;      // [2] S of block g is complete
  uint64_t* bar_p = bars + 6;      // [2] P of block g is written, S of block g is read
  uint64_t* bar_o = bars + 8;      // [2] the products of block g are in the accumulators
  uint64_t* kfull = bars + 10;     // [2]
  uint64_t* vfull = bars + 12;     // [2]
  uint64_t* kempty = bars + 14;    // [2]
  uint64_t* vempty = bars + 16;    // [2]
  uint64_t* bar_free = bars + 18;  // the accumulators of an item have been read
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 19);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* sums = reinterpret_cast<float*>(tmem_slot + 2);      // [2][4][128]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&qfull[i], 1);
      mbar_init(&qempty[i], 1);
      mbar_init(&bar_s[i], 1);
      mbar_init(&bar_p[i], SOFT / 2);
      mbar_init(&bar_o[i], 1);
      mbar_init(&kfull[i], 1);
      mbar_init(&vfull[i], 1);
      mbar_init(&kempty[i], 1);
      mbar_init(&vempty[i], 1);
    }
    mbar_init(bar_free, SOFT);
    *abort_flag = 0;
    if ((smem_u32(smem) & 1023u) != 0) {           // swizzled tiles need 1 KB alignment
      *abort_flag = 1;
      if (p.err) atomicCAS(p.err, kOk, kErrBadArgument);
    }
    fence_barrier_init();
  }
  if (warp == 17) {
    tmem_alloc<kTmemCols>(tmem_slot);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const bool dead = *abort_flag != 0;
  const int step = gridDim.x;

  if (warp == 16) {
    // ================================================================ TMA producer
    if (lane == 0 && !dead) {
      tma_prefetch_desc(&tma_q);
      tma_prefetch_desc(&tma_k);
      tma_prefetch_desc(&tma_v);
      const int rows = p.page < BKV ? p.page : BKV;          // rows per box
      bool ok = true;
      int g = 0, n = 0;
      for (int i = blockIdx.x; i < p.n_items && ok; i += step, ++n) {
        const Item w(p, i);
        const int* bt = p.block_tables + static_cast<size_t>(w.seg) * p.max_blocks;
        auto pool_row = [&](int pos) { return bt[min(pos / p.page, p.max_blocks - 1)] * p.page + pos % p.page; };
        ok = mbar_wait(&qempty[n & 1], (static_cast<uint32_t>(n >> 1) & 1) ^ 1, abort_flag, p.err);
        if (!ok) break;
        // the box holds `tokens` tokens of G heads: row = token * G + head; rows behind it are never stored
        mbar_expect_tx(&qfull[n & 1], static_cast<uint32_t>(p.tokens * p.G) * DK * 2);
        for (int c = 0; c < DK / 64; ++c) tma_load_3d(smem + (n & 1) * kQBytes + c * kQHalf, &tma_q, &qfull[n & 1], c * 64, w.kvh * p.G, w.row0);
        for (int j = 0; j < w.n_blocks; ++j, ++g) {
          const int s = g & 1, at = w.first_position(j);
          const uint32_t ph = (static_cast<uint32_t>(g >> 1) & 1) ^ 1;
          ok = mbar_wait(&kempty[s], ph, abort_flag, p.err);
          if (!ok) break;
          uint8_t* sk = smem + 2 * kQBytes + s * kKBytes;
          mbar_expect_tx(&kfull[s], kKBytes);
          for (int r = 0; r < BKV; r += rows) {
            const int row = pool_row(at + r);
            for (int c = 0; c < DK / 64; ++c) tma_load_3d(sk + c * kKVHalf + r * 128, &tma_k, &kfull[s], c * 64, w.kvh, row);
          }
          ok = mbar_wait(&vempty[s], ph, abort_flag, p.err);
          if (!ok) break;
          uint8_t* sv = smem + p.v_at + s * p.nv * kVBytes;
          mbar_expect_tx(&vfull[s], w.nv * kVBytes);
          for (int r = 0; r < BKV; r += rows) {
            const int row = pool_row(at + r);
            for (int v = 0; v < w.nv; ++v)
              for (int c = 0; c < DV / 64; ++c) tma_load_3d(sv + v * kVBytes + c * kKVHalf + r * 128, &tma_v, &vfull[s], c * 64, w.v0 + v, row);
          }
        }
      }
    }
  } else if (warp == 17) {
    // ================================================================ MMA issuer
    if (lane == 0 && !dead) {
      const uint32_t idesc_s = make_idesc_f16(BQ, BKV, true, false, false);
      const uint32_t idesc_o = make_idesc_f16(BQ, DV, true, false, true);
      const uint32_t sq = smem_u32(smem), sp = smem_u32(smem + p.p_at);
      // scores run two blocks ahead of the products, across items
      int si = blockIdx.x, sn = 0, sj = 0, sg = 0;
      int s_blocks = si < p.n_items ? Item(p, si).n_blocks : 0;
      auto issue_s = [&]() -> bool {
        if (si >= p.n_items) return true;
        const int s = sg & 1;
        if (sj == 0 && !mbar_wait(&qfull[sn & 1], static_cast<uint32_t>(sn >> 1) & 1, abort_flag, p.err)) return false;
        if (!mbar_wait(&kfull[s], static_cast<uint32_t>(sg >> 1) & 1, abort_flag, p.err)) return false;
        tc_fence_after();
        const uint32_t q = sq + (sn & 1) * kQBytes, sk = smem_u32(smem + 2 * kQBytes + s * kKBytes);
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint64_t da = make_smem_desc(q + (kk >> 2) * kQHalf + (kk & 3) * 32, 16, 1024, kSwizzle128B);
          const uint64_t db = make_smem_desc(sk + (kk >> 2) * kKVHalf + (kk & 3) * 32, 16, 1024, kSwizzle128B);
          umma_f16(tmem_base + T_S + s * BKV, da, db, idesc_s, kk > 0 ? 1u : 0u);
        }
        umma_commit(&kempty[s]);
        umma_commit(&bar_s[s]);
        ++sg;
        if (++sj == s_blocks) {
          umma_commit(&qempty[sn & 1]);
          sj = 0;
          ++sn;
          si += step;
          if (si < p.n_items) s_blocks = Item(p, si).n_blocks;
        }
        return true;
      };
      bool ok = issue_s() && issue_s();
      int g = 0, n = 0;
      for (int i = blockIdx.x; i < p.n_items && ok; i += step, ++n) {
        const Item w(p, i);
        if (n > 0) ok = mbar_wait(bar_free, static_cast<uint32_t>(n - 1) & 1, abort_flag, p.err);
        for (int j = 0; j < w.n_blocks && ok; ++j, ++g) {
          const int s = g & 1;
          const uint32_t ph = static_cast<uint32_t>(g >> 1) & 1;
          ok = mbar_wait(&bar_p[s], ph, abort_flag, p.err) && mbar_wait(&vfull[s], ph, abort_flag, p.err);
          if (!ok) break;
          tc_fence_after();
          for (int v = 0; v < w.nv; ++v) {
            const uint32_t sv = smem_u32(smem + p.v_at + (s * p.nv + v) * kVBytes);
#pragma unroll
            for (int kk = 0; kk < BKV / 16; ++kk) {
              const uint64_t da = make_smem_desc(sp + s * kPBytes + kk * 32, 16, 1024, kSwizzle128B);
              const uint64_t db = make_smem_desc(sv + kk * 2048, kKVHalf, 1024, kSwizzle128B);      // V tile [position][d]
              umma_f16(tmem_base + T_O + v * DV, da, db, idesc_o, (j > 0 || kk > 0) ? 1u : 0u);
            }
          }
          umma_commit(&vempty[s]);
          umma_commit(&bar_o[s]);
          ok = issue_s();      // S of block g was read before bar_p completed
        }
      }
    }
  } else {
    // ================================================================ softmax + epilogue (warps 0..15)
    const int set = warp >> 3, half = (warp >> 2) & 1;           // the set takes blocks set, set + 2, ..; columns half * 32 .. + 31 of a block
    const int r = (warp & 3) * 32 + lane;                        // row of the tile = TMEM lane
    const int t = r / p.G;
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    unsigned long long poly[7];
#pragma unroll
    for (int k = 0; k < 7; ++k) poly[k] = pair2(kTanh[k] * p.cap_log2, kTanh[k] * p.cap_log2);
    const unsigned long long cin = pair2(p.cap_in, p.cap_in);
    uint8_t* sp = smem + p.p_at + set * kPBytes + r * 128;
    bool ok = !dead;
    int g = 0, n = 0;
    for (int i = blockIdx.x; i < p.n_items && ok; i += step, ++n) {
      const Item w(p, i);
      const int head = w.kvh * p.G + r % p.G;
      const int limit = w.pos0 + t + 1;                          // this row sees positions first .. limit - 1, and those in front of p.keep
      const int first = p.chunk ? (w.pos0 + t) / p.chunk * p.chunk : limit - min(p.window, limit);
      const bool mine = t < w.ntok;
      float l = 0.f;
      if (p.sink && mine && warp < 4) l = exp2f(__bfloat162float(p.sink[head]) * 1.4426950408889634f);
      for (int j = (g ^ set) & 1; j < w.n_blocks; j += 2) {
        const uint32_t turn = static_cast<uint32_t>(g + j) >> 1;
        if (ok) ok = mbar_wait(&bar_s[set], turn & 1, abort_flag, p.err);
        if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
        tc_fence_after();
        uint32_t raw[32];
        tmem_ld_32x32b_x32(tmem_base + T_S + set * BKV + half * 32 + lane_addr, raw);
        tmem_wait_ld();
        float big = 0.f;
#pragma unroll
        for (int c = 0; c < 32; c += 2) big = fmaxf(fmaxf(big, fabsf(__uint_as_float(raw[c]))), fabsf(__uint_as_float(raw[c + 1])));
        if (__all_sync(0xffffffffu, big * p.cap_in <= 1.f)) {
#pragma unroll
          for (int c = 0; c < 32; c += 2) {
            const unsigned long long x = mul2(pair2(__uint_as_float(raw[c]), __uint_as_float(raw[c + 1])), cin), u = mul2(x, x);
            unsigned long long y = poly[6];
#pragma unroll
            for (int k = 5; k >= 0; --k) y = fma2(y, u, poly[k]);
            float a, b;
            split2(mul2(x, y), a, b);
            raw[c] = __float_as_uint(a);
            raw[c + 1] = __float_as_uint(b);
          }
        } else {
#pragma unroll
          for (int c = 0; c < 32; ++c) {
            const float x = 2.8853900817779268f * fminf(p.cap_in * __uint_as_float(raw[c]), 20.f);      // 2 / ln 2
            raw[c] = __float_as_uint(p.cap_log2 * (1.f - __fdividef(2.f, 1.f + exp2f(x))));
          }
        }
        const int at = w.first_position(j) + half * 32;
        const int lim = limit - at, low = first - at, kept = p.keep - at;      // columns low .. lim - 1 are seen, and those in front of `kept`
        if (!__all_sync(0xffffffffu, lim >= 32 && (low <= 0 || kept >= 32))) {
#pragma unroll
          for (int c = 0; c < 32; ++c)
            if (c >= lim || (c < low && c >= kept)) raw[c] = 0xff800000u;      // -inf
        }
        float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
        for (int c = 0; c < 32; c += 2) {
          const float a = exp2f(__uint_as_float(raw[c])), b = exp2f(__uint_as_float(raw[c + 1]));
          sum0 += a;
          sum1 += b;
          raw[c >> 1] = pack_bf16(a, b);
        }
        l += sum0 + sum1;
        if (turn > 0) {      // the products of the set's block before have read this P buffer
          if (ok) ok = mbar_wait(&bar_o[set], (turn - 1) & 1, abort_flag, p.err);
          if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
        }
#pragma unroll
        for (int k = 0; k < 4; ++k)
          *reinterpret_cast<uint4*>(sp + (((half * 4 + k) ^ (r & 7)) << 4)) = make_uint4(raw[4 * k], raw[4 * k + 1], raw[4 * k + 2], raw[4 * k + 3]);
        fence_proxy_async();
        tc_fence_before();
        mbar_arrive(&bar_p[set]);
      }
      g += w.n_blocks;
      float* sum = sums + (n & 1) * 4 * BQ;      // (two buffers: a warp may be one item ahead)
      sum[(set * 2 + half) * BQ + r] = l;
      // The set without the last block waits for its own last one first: products complete in order, so the other barrier is then at most
      // one phase behind and its parity says which.
      if (ok && ((g - 1) & 1) != set && w.n_blocks > 1) ok = mbar_wait(&bar_o[set], static_cast<uint32_t>((g - 2) >> 1) & 1, abort_flag, p.err);
      if (ok) ok = mbar_wait(&bar_o[(g - 1) & 1], static_cast<uint32_t>((g - 1) >> 1) & 1, abort_flag, p.err);
      ok = named_bar_and(1, SOFT, ok);      // (all leave together when a wait ran out)
      tc_fence_after();
      l = sum[r] + sum[BQ + r] + sum[2 * BQ + r] + sum[3 * BQ + r];
      const float inv_l = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* out = p.out + ((static_cast<size_t>(w.row0 + t) * p.H + head) * p.Hkv + w.v0) * p.out_d;
      if (ok) {
#pragma unroll 1
        for (int k = warp >> 2; k < w.nv * (DV / 32); k += 4) {      // the four warps of a lane quarter share the columns
          const int v = k / (DV / 32), c = (k % (DV / 32)) * 32;
          if (c >= p.out_d) continue;
          uint32_t o[32];
          tmem_ld_32x32b_x32(tmem_base + T_O + v * DV + c + lane_addr, o);
          tmem_wait_ld();
          if (mine) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              if (c + e * 8 < p.out_d) {
                uint4 pk;
                pk.x = pack_bf16(__uint_as_float(o[8 * e]) * inv_l, __uint_as_float(o[8 * e + 1]) * inv_l);
                pk.y = pack_bf16(__uint_as_float(o[8 * e + 2]) * inv_l, __uint_as_float(o[8 * e + 3]) * inv_l);
                pk.z = pack_bf16(__uint_as_float(o[8 * e + 4]) * inv_l, __uint_as_float(o[8 * e + 5]) * inv_l);
                pk.w = pack_bf16(__uint_as_float(o[8 * e + 6]) * inv_l, __uint_as_float(o[8 * e + 7]) * inv_l);
                reinterpret_cast<uint4*>(out + static_cast<size_t>(v) * p.out_d + c)[e] = pk;
              }
            }
          }
        }
      }
      tc_fence_before();
      mbar_arrive(bar_free);
    }
  }

  if (*abort_flag) __nanosleep(50000);
  tc_fence_before();
  __syncthreads();
  if (warp == 17) {
    tc_fence_after();
    tmem_dealloc<kTmemCols>(tmem_base);
  }
}

template <int DK, int DV>
static int launch(const void* q, const void* kc, const void* vc, int rows, int n, uint64_t pool_rows, Params p, cudaStream_t st) {
  CUtensorMap tq, tk, tv;
  int rc = encode_tma_3d_16bit(&tq, q, DK, p.H, rows, DK, static_cast<uint64_t>(p.H) * DK, 64, p.G, p.tokens);
  if (rc) return rc;
  const uint32_t box = p.page >= BKV ? BKV : p.page;
  rc = encode_tma_3d_16bit(&tk, kc, DK, p.Hkv, pool_rows, DK, static_cast<uint64_t>(p.Hkv) * DK, 64, 1, box);
  if (rc) return rc;
  rc = encode_tma_3d_16bit(&tv, vc, DV, p.Hkv, pool_rows, DV, static_cast<uint64_t>(p.Hkv) * DV, 64, 1, box);
  if (rc) return rc;
  // value groups whose accumulators fit (3 of 128 columns, 6 of 64), one less where two stages of their tiles do not
  constexpr int most = (kTmemCols - T_O) / DV - (DK == 128 ? 1 : 0);
  const int slices = (p.Hkv + most - 1) / most;
  p.nv = (p.Hkv + slices - 1) / slices;
  p.slices = (p.Hkv + p.nv - 1) / p.nv;
  const long long items = static_cast<long long>(n) * p.Hkv * p.slices;
  if (items > 1 << 30) return -20;
  p.n_items = static_cast<int>(items);
  p.v_at = DK / 64 * 2 * (kQHalf + kKVHalf);
  p.p_at = p.v_at + 2 * p.nv * (DV / 64) * kKVHalf;
  p.bar_at = p.p_at + 2 * kPBytes;
  const int total = p.bar_at + 256 + 8 * BQ * 4;
  if (total > 227 * 1024) return -20;
  auto kern = talk_flash_kernel<DK, DV>;
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr = true;
  }
  // two CTAs of an SM would take turns with all of its TMEM columns: ask for more than half of the shared memory
  kern<<<p.n_items < num_sms() ? p.n_items : num_sms(), THREADS, total < 116 * 1024 ? 116 * 1024 : total, st>>>(tq, tk, tv, p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace tf
}  // namespace rb

// q [rows][Hq][dk], pools [pool_rows][Hkv][dk / dv] (64 or 128 columns), out [rows][Hq][Hkv][out_d]; blocks, window, keep and chunk as in
// rb_paged_flash.  cap: in (0, 80]; sinks of up to 88.  Returns -20 for shapes outside that.
extern "C" int rb_talk_flash(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx, const int* blocks, const void* sink,
                             void* out, int rows, int n, int Hq, int Hkv, int dk, int dv, int out_d, long long pool_rows, int page, int max_blocks,
                             int window, int keep, int chunk, float scale, float cap, int* err, cudaStream_t st) {
  using namespace rb;
  using namespace rb::tf;
  if (rows <= 0 || n <= 0) return 0;
  if (Hkv < 1 || Hq % Hkv || window < 0 || keep < 0 || chunk < 0 || (keep && !window) || (chunk && window)) return -2;
  const int G = Hq / Hkv;
  if (G > BQ || Hkv > 65535 || (dk != 64 && dk != 128) || (dv != 64 && dv != 128) || out_d % 8 || out_d > dv || out_d < 1) return -20;
  if ((page != 16 && page != 32 && page % 64) || scale <= 0.f || cap <= 0.f || cap > 80.f) return -20;
  Params p{};
  p.blocks = blocks; p.ctx = ctx; p.block_tables = block_tables; p.sink = static_cast<const __nv_bfloat16*>(sink); p.out = static_cast<__nv_bfloat16*>(out);
  p.H = Hq; p.Hkv = Hkv; p.G = G; p.tokens = BQ / G; p.max_blocks = max_blocks; p.page = page; p.out_d = out_d;
  p.window = window ? window : INT_MAX; p.keep = keep; p.chunk = chunk;
  p.cap_in = scale / cap;
  p.cap_log2 = cap * 1.4426950408889634f;
  p.err = err;
  const uint64_t pr = static_cast<uint64_t>(pool_rows);
  if (dk == 128) return dv == 128 ? launch<128, 128>(q, kc, vc, rows, n, pr, p, st) : launch<128, 64>(q, kc, vc, rows, n, pr, p, st);
  return dv == 128 ? launch<64, 128>(q, kc, vc, rows, n, pr, p, st) : launch<64, 64>(q, kc, vc, rows, n, pr, p, st);
}
