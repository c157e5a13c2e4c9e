// Flash attention of prompt portions whose heads' weights are mixed afterwards, over paged keys and values: every head's weights meet the
// values of every group (see talk_decode_sm100.cu), out [rows][H][G][out_d].
//
// Tiles are those of paged_flash_sm100.cu (128 (token, head) rows of one key group, blocks of 64 positions straight from the pages), but a CTA
// keeps the accumulators of several groups' values (256 columns of TMEM), so scores and softmax are computed once for all of them.
// Scores are capped: the softmax has a fixed reference and nothing is rescaled; what a score costs is a polynomial and one
// exponential.  The CTAs are persistent and their blocks form one sequence across tiles.  Scores run four blocks ahead of the products; two
// sets of eight warps (two threads per row) take the blocks in turn, and P replaces S in TMEM, where the products read it.  Warps of
// their own read the accumulators of a finished tile while the softmax is at the next one; whole tiles leave through shared memory and TMA
// stores.  Keys (three stages) and values (two) have producers of their own: a block's arithmetic is shorter than the way of its tiles
// through the L2.  Issuing a block's products, with the waits around them, takes one thread longer than the tensor cores need for them, so scores
// and output products are issued by two.  Warps 0-15: softmax, warp 16: TMA of queries and keys, warp 17: scores, warps 18-21: outputs, warp
// 22: TMA of values, warp 23: products with the values.  Every wait is bounded; no load uses cluster multicast.
#include <limits.h>

#include "common.cuh"
#include "host_utils.h"

namespace rb {
namespace tf {

constexpr int BQ = 128;
constexpr int BKV = 64;
constexpr int SOFT = 512;                 // softmax threads: two sets of two per row
constexpr int kWarpK = 16, kWarpS = 17, kWarpOut = 18, kWarpV = 22, kWarpPv = 23;      // (four warps for the outputs)
constexpr int THREADS = 24 * 32;
constexpr int KST = 3, VST = 2;           // stages of keys and of values
constexpr int NS = 4;                     // buffers of scores
static_assert(KST < NS && VST < NS, "a producer is never two phases behind");
constexpr int RING = 8;                   // items whose sums are kept: the softmax is at most NS of them ahead of the outputs
constexpr int kTmemCols = 512;
constexpr int T_S = 0;                    // NS buffers of 64 columns; P takes the first 16 of every 32
constexpr int T_O = NS * 64;
constexpr int kQHalf = BQ * 128, kKVHalf = BKV * 128;      // bytes of 64 columns
constexpr int kStage = BQ * 128;          // 64 columns of outputs on their way out

struct Params {
  const int* blocks;         // [n][4]: segment, first row, rows, position of the first row; null: row i is segment i, at ctx[i] - 1
  const int* ctx;            // [S]
  const int* block_tables;   // [S][max_blocks]
  const __nv_bfloat16* sink; // [H] or null
  __nv_bfloat16* out;        // [rows][H][Hkv][out_d]
  int H, Hkv, G, tokens, max_blocks, page, out_d, nv;      // G: heads per group; nv: value groups per item
  int n_items, slices;       // items: query tile, key group, slice of value groups (the last one fastest)
  int window, keep, chunk;   // as in paged_flash
  int v_at, out_at, bar_at;  // bytes into shared memory
  int stores;                // whole tiles leave by TMA
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
                  const __grid_constant__ CUtensorMap tma_o, const Params p) {
  constexpr int kQBytes = DK / 64 * kQHalf, kKBytes = DK / 64 * kKVHalf, kVBytes = DV / 64 * kKVHalf;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + p.bar_at);
  // blocks are numbered across items (g): S and P of block g are buffer g % NS, its keys and values a stage each; queries and accumulators
  // go by item (n)
  uint64_t* qfull = bars;
  uint64_t* qempty = bars + 1;     // the scores of an item are complete
  uint64_t* bar_done = bars + 2;   // the products of an item are in the accumulators
  uint64_t* bar_free = bars + 3;   // the accumulators of an item have been read
  uint64_t* bar_s = bars + 4;      // [NS] S of a block is complete, and the stage of its keys free
  uint64_t* bar_pv = bar_s + NS;   // [NS] its products are: the buffer and the stage of its values are free
  uint64_t* bar_p = bar_pv + NS;   // [NS] P of a block is written
  uint64_t* bar_l = bar_p + NS;    // [RING] the sums of an item are written
  uint64_t* kfull = bar_l + RING;  // [KST]
  uint64_t* vfull = kfull + KST;   // [VST]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(vfull + VST);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* sums = reinterpret_cast<float*>(smem + p.bar_at + 512);      // [RING][4][128]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(qfull, 1);
    mbar_init(qempty, 1);
    mbar_init(bar_done, 1);
    mbar_init(bar_free, 128);
    for (int i = 0; i < NS; ++i) {
      mbar_init(&bar_s[i], 1);
      mbar_init(&bar_pv[i], 1);
      mbar_init(&bar_p[i], SOFT / 2);
    }
    for (int i = 0; i < RING; ++i) mbar_init(&bar_l[i], SOFT);
    for (int i = 0; i < KST; ++i) mbar_init(&kfull[i], 1);
    for (int i = 0; i < VST; ++i) mbar_init(&vfull[i], 1);
    *abort_flag = 0;
    if ((smem_u32(smem) & 1023u) != 0) {           // swizzled tiles need 1 KB alignment
      *abort_flag = 1;
      if (p.err) atomicCAS(p.err, kOk, kErrBadArgument);
    }
    fence_barrier_init();
  }
  if (warp == kWarpS) {
    tmem_alloc<kTmemCols>(tmem_slot);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const bool dead = *abort_flag != 0;
  const int step = gridDim.x;

  if (warp == kWarpK || warp == kWarpV) {
  // ================================================================ TMA producers: queries and keys; values
    if (lane == 0 && !dead) {
      const bool values = warp == kWarpV;
      tma_prefetch_desc(values ? &tma_v : &tma_k);
      if (!values) tma_prefetch_desc(&tma_q);
      const int rows = p.page < BKV ? p.page : BKV;          // rows per box
      uint64_t* full = values ? vfull : kfull;
      uint64_t* freed = values ? bar_pv : bar_s;
      const int stages = values ? VST : KST;
      bool ok = true;
      int s = 0, n = 0, g = 0;
      for (int i = blockIdx.x; i < p.n_items && ok; i += step, ++n) {
        const Item w(p, i);
        const int* bt = p.block_tables + static_cast<size_t>(w.seg) * p.max_blocks;
        if (!values) {
          ok = mbar_wait(qempty, (static_cast<uint32_t>(n) & 1) ^ 1, abort_flag, p.err);
          if (!ok) break;
          // the box holds `tokens` tokens of G heads: row = token * G + head; rows behind it are never stored
          mbar_expect_tx(qfull, static_cast<uint32_t>(p.tokens * p.G) * DK * 2);
          for (int c = 0; c < DK / 64; ++c) tma_load_3d(smem + c * kQHalf, &tma_q, qfull, c * 64, w.kvh * p.G, w.row0);
        }
        for (int j = 0; j < w.n_blocks; ++j, ++g) {
          const int at = w.first_position(j);
          if (g >= stages) ok = mbar_wait(&freed[(g - stages) % NS], static_cast<uint32_t>((g - stages) / NS) & 1, abort_flag, p.err);
          if (!ok) break;
          mbar_expect_tx(&full[s], values ? w.nv * kVBytes : kKBytes);
          for (int r = 0; r < BKV; r += rows) {
            const int pos = at + r, row = bt[min(pos / p.page, p.max_blocks - 1)] * p.page + pos % p.page;
            if (values) {
              uint8_t* sv = smem + p.v_at + s * p.nv * kVBytes + r * 128;
              for (int v = 0; v < w.nv; ++v)
                for (int c = 0; c < DV / 64; ++c) tma_load_3d(sv + v * kVBytes + c * kKVHalf, &tma_v, &full[s], c * 64, w.v0 + v, row);
            } else {
              uint8_t* sk = smem + kQBytes + s * kKBytes + r * 128;
              for (int c = 0; c < DK / 64; ++c) tma_load_3d(sk + c * kKVHalf, &tma_k, &full[s], c * 64, w.kvh, row);
            }
          }
          if (++s == stages) s = 0;
        }
      }
    }
  } else if (warp == kWarpS) {
    // ================================================================ scores, up to NS blocks ahead of the products
    if (lane == 0 && !dead) {
      const uint32_t idesc = make_idesc_f16(BQ, BKV, true, false, false);
      const uint32_t sq = smem_u32(smem);
      bool ok = true;
      int g = 0, n = 0, stage = 0;
      uint32_t ph = 0;
      for (int i = blockIdx.x; i < p.n_items && ok; i += step, ++n) {
        const int blocks = Item(p, i).n_blocks;
        ok = mbar_wait(qfull, static_cast<uint32_t>(n) & 1, abort_flag, p.err);
        for (int j = 0; j < blocks && ok; ++j, ++g) {
          const int s = g % NS;
          ok = mbar_wait(&kfull[stage], ph, abort_flag, p.err);
          if (ok && g >= NS) ok = mbar_wait(&bar_pv[s], static_cast<uint32_t>(g / NS - 1) & 1, abort_flag, p.err);
          if (!ok) break;
          tc_fence_after();
          const uint32_t sk = smem_u32(smem + kQBytes + stage * kKBytes);
#pragma unroll
          for (int kk = 0; kk < DK / 16; ++kk) {
            const uint64_t da = make_smem_desc(sq + (kk >> 2) * kQHalf + (kk & 3) * 32, 16, 1024, kSwizzle128B);
            const uint64_t db = make_smem_desc(sk + (kk >> 2) * kKVHalf + (kk & 3) * 32, 16, 1024, kSwizzle128B);
            umma_f16(tmem_base + T_S + s * BKV, da, db, idesc, kk > 0 ? 1u : 0u);
          }
          umma_commit(&bar_s[s]);
          if (++stage == KST) {
            stage = 0;
            ph ^= 1;
          }
        }
        if (ok) umma_commit(qempty);
      }
      if (ok && n > 0) mbar_wait(qempty, static_cast<uint32_t>(n - 1) & 1, abort_flag, p.err);      // (no commit outlives the CTA)
    }
  } else if (warp == kWarpPv) {
    // ================================================================ products with the values, all groups of an item at once
    if (lane == 0 && !dead) {
      bool ok = true;
      int g = 0, n = 0, stage = 0;
      uint32_t ph = 0;
      for (int i = blockIdx.x; i < p.n_items && ok; i += step, ++n) {
        const Item w(p, i);
        const uint32_t idesc = make_idesc_f16(BQ, w.nv * DV, true, false, true);
        if (n > 0) ok = mbar_wait(bar_free, static_cast<uint32_t>(n - 1) & 1, abort_flag, p.err);
        for (int j = 0; j < w.n_blocks && ok; ++j, ++g) {
          const int s = g % NS;
          ok = mbar_wait(&vfull[stage], ph, abort_flag, p.err) && mbar_wait(&bar_p[s], static_cast<uint32_t>(g / NS) & 1, abort_flag, p.err);
          if (!ok) break;
          tc_fence_after();
          const uint32_t sv = smem_u32(smem + p.v_at + stage * p.nv * kVBytes);
#pragma unroll
          for (int kk = 0; kk < BKV / 16; ++kk) {
            const uint64_t db = make_smem_desc(sv + kk * 2048, kKVHalf, 1024, kSwizzle128B);      // V tiles [position][d], 64 columns kKVHalf apart
            umma_f16_ts(tmem_base + T_O, tmem_base + T_S + s * BKV + (kk >> 1) * 32 + (kk & 1) * 8, db, idesc, (j > 0 || kk > 0) ? 1u : 0u);
          }
          umma_commit(&bar_pv[s]);
          if (++stage == VST) {
            stage = 0;
            ph ^= 1;
          }
        }
        if (ok) umma_commit(bar_done);
      }
      if (ok && n > 0) mbar_wait(bar_done, static_cast<uint32_t>(n - 1) & 1, abort_flag, p.err);
    }
  } else if (warp >= kWarpOut && warp < kWarpV) {
    // ================================================================ outputs (four warps)
    const int r = (warp & 3) * 32 + lane;                        // row of the tile = TMEM lane
    const int t = r / p.G;
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const bool issues = warp == kWarpOut && lane == 0;
    bool ok = !dead;
    int n = 0;
    for (int i = blockIdx.x; i < p.n_items && ok; i += step, ++n) {
      const Item w(p, i);
      ok = mbar_wait(&bar_l[n % RING], static_cast<uint32_t>(n / RING) & 1, abort_flag, p.err) &&
           mbar_wait(bar_done, static_cast<uint32_t>(n) & 1, abort_flag, p.err);
      if (issues) tma_store_wait_read<0>();                      // the item before has left shared memory
      ok = named_bar_and(1, 128, ok);                            // (all leave together when a wait ran out)
      if (!ok) break;
      tc_fence_after();
      const float* sum = sums + (n % RING) * 4 * BQ + r;
      const float l = sum[0] + sum[BQ] + sum[2 * BQ] + sum[3 * BQ];
      const float inv_l = l > 0.f ? 1.f / l : 0.f;
      const bool whole = p.stores && w.ntok == p.tokens, mine = t < w.ntok;
      __nv_bfloat16* out = p.out + ((static_cast<size_t>(w.row0 + t) * p.H + w.kvh * p.G + r % p.G) * p.Hkv + w.v0) * p.out_d;
      const int parts = w.nv * (DV / 32);                        // of 32 columns
#pragma unroll 1
      for (int part = 0; part < parts; ++part) {
        uint32_t o[32];
        tmem_ld_32x32b_x32(tmem_base + T_O + part * 32 + lane_addr, o);
        tmem_wait_ld();
        if (part + 1 == parts) {
          tc_fence_before();
          mbar_arrive(bar_free);
        }
        const int v = part / (DV / 32), c = (part % (DV / 32)) * 32;
        uint8_t* dst = smem + p.out_at + (part >> 1) * kStage + r * 128;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          uint4 pk;
          pk.x = pack_bf16(__uint_as_float(o[8 * e]) * inv_l, __uint_as_float(o[8 * e + 1]) * inv_l);
          pk.y = pack_bf16(__uint_as_float(o[8 * e + 2]) * inv_l, __uint_as_float(o[8 * e + 3]) * inv_l);
          pk.z = pack_bf16(__uint_as_float(o[8 * e + 4]) * inv_l, __uint_as_float(o[8 * e + 5]) * inv_l);
          pk.w = pack_bf16(__uint_as_float(o[8 * e + 6]) * inv_l, __uint_as_float(o[8 * e + 7]) * inv_l);
          if (whole) *reinterpret_cast<uint4*>(dst + ((((part & 1) * 4 + e) ^ (r & 7)) << 4)) = pk;
          else if (mine && c + e * 8 < p.out_d) *reinterpret_cast<uint4*>(out + static_cast<size_t>(v) * p.out_d + c + e * 8) = pk;
        }
      }
      if (whole) {
        fence_proxy_async();
        named_bar_sync(1, 128);
        if (issues) {
          for (int k = 0; k < parts / 2; ++k)
            tma_store_4d(&tma_o, smem + p.out_at + k * kStage, (k % (DV / 64)) * 64, w.v0 + k / (DV / 64), w.kvh * p.G, w.row0);
          tma_store_commit();
        }
      }
    }
    if (issues) tma_store_wait<0>();
  } else {
    // ================================================================ softmax (warps 0..15)
    const int set = warp >> 3, half = (warp >> 2) & 1;           // the set takes every other block; columns half * 32 .. + 31 of a block
    const int r = (warp & 3) * 32 + lane;                        // row of the tile = TMEM lane
    const int t = r / p.G;
    const uint32_t mine_at = tmem_base + T_S + half * 32 + (static_cast<uint32_t>((warp & 3) * 32) << 16);
    unsigned long long poly[7];
#pragma unroll
    for (int k = 0; k < 7; ++k) poly[k] = pair2(kTanh[k] * p.cap_log2, kTanh[k] * p.cap_log2);
    const unsigned long long cin = pair2(p.cap_in, p.cap_in);
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
        const int s = (g + j) % NS;
        if (ok) ok = mbar_wait(&bar_s[s], static_cast<uint32_t>((g + j) / NS) & 1, abort_flag, p.err);
        if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
        tc_fence_after();
        uint32_t raw[32];
        tmem_ld_32x32b_x32(mine_at + s * BKV, raw);
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
        tmem_st_32x32b_x16(mine_at + s * BKV, raw);
        tmem_wait_st();
        tc_fence_before();
        mbar_arrive(&bar_p[s]);
      }
      g += w.n_blocks;
      sums[((n % RING) * 4 + set * 2 + half) * BQ + r] = l;
      mbar_arrive(&bar_l[n % RING]);
    }
  }

  if (*abort_flag) __nanosleep(50000);
  tc_fence_before();
  __syncthreads();
  if (warp == kWarpS) {
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
  // value groups per item: as many as their accumulators and the stages of their tiles leave room for, shared out evenly
  int total = 0;
  for (int most = (kTmemCols - T_O) / DV;; --most) {
    if (most < 1) return -20;
    p.slices = (p.Hkv + most - 1) / most;
    p.nv = (p.Hkv + p.slices - 1) / p.slices;
    p.v_at = DK / 64 * (kQHalf + KST * kKVHalf);
    p.out_at = p.v_at + VST * p.nv * (DV / 64) * kKVHalf;
    p.bar_at = p.out_at + p.nv * (DV / 64) * kStage;
    total = p.bar_at + 512 + RING * 4 * BQ * 4;
    if (total <= 227 * 1024) break;
  }
  const long long items = static_cast<long long>(n) * p.Hkv * p.slices;
  if (items > 1 << 30) return -20;
  p.n_items = static_cast<int>(items);
  CUtensorMap to = tq;
  p.stores = p.out_d % 64 == 0 && reinterpret_cast<uintptr_t>(p.out) % 16 == 0;
  if (p.stores) {
    rc = encode_tma_4d_dense_bf16(&to, p.out, p.out_d, p.Hkv, p.H, rows, 64, 1, p.G, p.tokens);
    if (rc) return rc;
  }
  auto kern = talk_flash_kernel<DK, DV>;
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr = true;
  }
  // two CTAs of an SM would take turns with all of its TMEM columns: ask for more than half of the shared memory
  kern<<<p.n_items < num_sms() ? p.n_items : num_sms(), THREADS, total < 116 * 1024 ? 116 * 1024 : total, st>>>(tq, tk, tv, to, p);
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
