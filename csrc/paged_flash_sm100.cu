// Flash attention of prompt portions over PAGED keys and values on the 5th-generation tensor cores.
//
// A query tile is 128 rows of (token, head) pairs: up to 128 / G consecutive tokens of one segment times the G query heads of
// one key / value head, so every key and value tile is loaded once for the whole group and a portion of a few tokens
// still fills the tile.  Per block of 64 positions:
//   S = Q K^T      tcgen05.mma, fp32 accumulator in TMEM
//   softmax        one thread per row reads its row of S, keeps a running reference / sum, writes P = exp2(S - m) as bf16
//                  into shared memory (128-byte swizzle)
//   O += P V       V is read in place from its [position][d] tile (MN-major)
// Keys and values come straight from the pages (TMA, one box per page and 64 columns): new rows are written to the pages before
// this kernel runs, and nothing is gathered into a dense copy.  Keys and values that were projected for one call (of a latent cache's
// rows) lie side by side instead, every segment from a row of its own on.  Heads may be narrower than the 64-column boxes: what a box
// reads behind them is zero.  The running softmax starts from the head's sink logit
// (sum = 1 at reference = sink), or empty without one.  With a window a tile starts at the block of the first position that its first
// row sees, and every row masks what lies before its own.  A gate per output feature is applied in the epilogue.  S is double buffered, so the product of block j + 1 runs while the
// softmax of block j does.  Positions at a sequence's start may stay visible outside a window (their blocks come first), rows may see
// only their own chunk of positions, scores may be capped, and a head's weights may meet the values of every group (one group per
// blockIdx.z), for heads whose weights are mixed afterwards.  The accumulator is rescaled only when a row's maximum grows by more than 2^8 (decided per warp: TMEM
// accesses are warp-wide).  Warps 0-3: softmax and epilogue, warp 4: TMA, warp 5: MMA.  Two CTAs share an SM; keys of more than 128
// columns leave room for one stage of keys and values instead of two.  Every wait is bounded; no load uses cluster multicast.
#include <limits.h>

#include "common.cuh"
#include "host_utils.h"

namespace rb {
namespace pf {

constexpr int BQ = 128;
constexpr int BKV = 64;
constexpr int THREADS = 192;
constexpr int kTmemCols = 256;
constexpr int T_S = 0;           // two buffers of 64 columns
constexpr int T_O = 128;

template <int DK, int DV>
struct Tile {
  static_assert((DK == 64 || DK == 128 || DK == 192) && (DV == 64 || DV == 128), "key / value rows of 64, 128 or (keys) 192 columns");
  static constexpr int kStages = DK > 128 ? 1 : 2;
  static constexpr int kQHalf = BQ * 128, kKVHalf = BKV * 128;      // bytes of 64 columns
  static constexpr int kQBytes = DK / 64 * kQHalf;
  static constexpr int kKBytes = DK / 64 * kKVHalf, kVBytes = DV / 64 * kKVHalf;
  static constexpr int kK = kQBytes;
  static constexpr int kV = kK + kStages * kKBytes;
  static constexpr int kP = kV + kStages * kVBytes;
  static constexpr int kBar = kP + BQ * BKV * 2;
  static constexpr int kTotal = kBar + 256;
};

struct Params {
  const int* blocks;         // [n][4]: segment, first row, rows, position of the first row; null: row i is segment i, at ctx[i] - 1
  const int* ctx;            // [S]
  const int* block_tables;   // [S][max_blocks]
  const int* first_row;      // [S]: rows of a segment's positions lie side by side from here on (then there are no pages), or null
  const __nv_bfloat16* sink; // [H] or null
  const __nv_bfloat16* gate; // [rows][ld_gate], head h's features at h * out_d (head_gate: one for all of them at h), or null
  int head_gate;
  __nv_bfloat16* out;        // [rows][H][out_d]
  int H, G, tokens, max_blocks, page, out_d, ld_gate;
  int window;                // positions a row sees (INT_MAX: all)
  int keep;                  // first positions that stay visible outside the window
  int chunk;                 // > 0: a row sees its own chunk of this many positions
  float scale_log2;          // kCap: 1, scores come out of the cap in log2 units
  float cap_in, cap_log2;    // kCap: s <- cap_log2 tanh(cap_in q . k)
  int* err;
};

// tanh in fp32 up to about 1e-7
__device__ __forceinline__ float bounded(float x) {
  return 1.f - __fdividef(2.f, 1.f + exp2f(2.8853900817779268f * fminf(x, 20.f)));      // 2 / ln 2
}

// eight accumulators times sigmoid(gate)
__device__ __forceinline__ void gate8(uint32_t* o, const uint4& g) {
  const uint32_t w[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    o[2 * k] = __float_as_uint(__fdividef(__uint_as_float(o[2 * k]), 1.f + __expf(-__uint_as_float(w[k] << 16))));
    o[2 * k + 1] = __float_as_uint(__fdividef(__uint_as_float(o[2 * k + 1]), 1.f + __expf(-__uint_as_float(w[k] & 0xffff0000u))));
  }
}

template <int DK, int DV, bool kCap>
__global__ void __launch_bounds__(THREADS, 2)
paged_flash_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k,
                   const __grid_constant__ CUtensorMap tma_v, const Params p) {
  using L = Tile<DK, DV>;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kBar);
  uint64_t* bar_q = bars;
  uint64_t* bar_s = bars + 1;      // [2] S of block j is complete (index = block & 1)
  uint64_t* bar_p = bars + 3;      // [2] P of block j is written, S of block j is read
  uint64_t* bar_o = bars + 5;      // [2] the product of block j is in the accumulator
  uint64_t* kfull = bars + 7;      // [2]
  uint64_t* vfull = bars + 9;      // [2]
  uint64_t* kempty = bars + 11;    // [2]
  uint64_t* vempty = bars + 13;    // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = blockIdx.y, vh = gridDim.z > 1 ? blockIdx.z : blockIdx.y;      // group of the keys, and of the values
  int seg, row0, ntok, pos0;
  if (p.blocks) {
    const int4 b = reinterpret_cast<const int4*>(p.blocks)[blockIdx.x];
    seg = b.x; row0 = b.y; ntok = b.z; pos0 = b.w;
  } else {
    seg = row0 = blockIdx.x;
    ntok = 1;
    pos0 = p.ctx[seg] - 1;
  }
  const int seen = pos0 + ntok;                    // positions that the last token of the tile sees
  // block of the first position that the first token sees, kept ones aside; the blocks of kept positions in front of it come first
  const int block0 = (p.chunk ? pos0 / p.chunk * p.chunk : max(0, pos0 - p.window + 1)) / BKV;
  const int n_kept = min((p.keep + BKV - 1) / BKV, block0);
  const int n_blocks = n_kept + (seen + BKV - 1) / BKV - block0;
  auto block_at = [&](int j) { return j < n_kept ? j : block0 + j - n_kept; };
  const int base = p.first_row ? p.first_row[seg] : -1;
  const int* bt = p.block_tables + static_cast<size_t>(p.first_row ? 0 : seg) * p.max_blocks;
  constexpr int ST = L::kStages;

  if (threadIdx.x == 0) {
    mbar_init(bar_q, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bar_s[i], 1);
      mbar_init(&bar_p[i], 128);
      mbar_init(&bar_o[i], 1);
      mbar_init(&kfull[i], 1);
      mbar_init(&vfull[i], 1);
      mbar_init(&kempty[i], 1);
      mbar_init(&vempty[i], 1);
    }
    *abort_flag = 0;
    if ((smem_u32(smem) & 1023u) != 0) {           // swizzled tiles need 1 KB alignment
      *abort_flag = 1;
      if (p.err) atomicCAS(p.err, kOk, kErrBadArgument);
    }
    fence_barrier_init();
  }
  if (warp == 5) {
    tmem_alloc<kTmemCols>(tmem_slot);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const bool dead = *abort_flag != 0;

  if (warp == 4) {
    // ================================================================ TMA producer
    if (lane == 0 && !dead) {
      tma_prefetch_desc(&tma_q);
      tma_prefetch_desc(&tma_k);
      tma_prefetch_desc(&tma_v);
      // the box holds `tokens` tokens of G heads: row = token * G + head; rows behind it are never stored
      mbar_expect_tx(bar_q, static_cast<uint32_t>(p.tokens * p.G) * DK * 2);
      for (int c = 0; c < DK / 64; ++c) tma_load_3d(smem + c * L::kQHalf, &tma_q, bar_q, c * 64, kvh * p.G, row0);
      const int rows = p.page < BKV ? p.page : BKV;          // rows per box
      for (int j = 0; j < n_blocks; ++j) {
        const int s = j % ST;
        const uint32_t ph = (static_cast<uint32_t>(j / ST) & 1) ^ 1;
        auto pool_row = [&](int pos) { return base >= 0 ? base + pos : bt[min(pos / p.page, p.max_blocks - 1)] * p.page + pos % p.page; };
        if (!mbar_wait(&kempty[s], ph, abort_flag, p.err)) break;
        uint8_t* sk = smem + L::kK + s * L::kKBytes;
        mbar_expect_tx(&kfull[s], L::kKBytes);
        for (int r = 0; r < BKV; r += rows) {
          const int row = pool_row(block_at(j) * BKV + r);
          for (int c = 0; c < DK / 64; ++c) tma_load_3d(sk + c * L::kKVHalf + r * 128, &tma_k, &kfull[s], c * 64, kvh, row);
        }
        if (!mbar_wait(&vempty[s], ph, abort_flag, p.err)) break;
        uint8_t* sv = smem + L::kV + s * L::kVBytes;
        mbar_expect_tx(&vfull[s], L::kVBytes);
        for (int r = 0; r < BKV; r += rows) {
          const int row = pool_row(block_at(j) * BKV + r);
          for (int c = 0; c < DV / 64; ++c) tma_load_3d(sv + c * L::kKVHalf + r * 128, &tma_v, &vfull[s], c * 64, vh, row);
        }
      }
    }
  } else if (warp == 5) {
    // ================================================================ MMA issuer
    if (lane == 0 && !dead) {
      const uint32_t idesc_s = make_idesc_f16(BQ, BKV, true, false, false);
      const uint32_t idesc_o = make_idesc_f16(BQ, DV, true, false, true);
      const uint32_t sq = smem_u32(smem), sp = smem_u32(smem + L::kP);
      auto issue_s = [&](int j) -> bool {
        const int s = j & 1, st = j % ST;
        if (!mbar_wait(&kfull[st], static_cast<uint32_t>(j / ST) & 1, abort_flag, p.err)) return false;
        tc_fence_after();
        const uint32_t sk = smem_u32(smem + L::kK + st * L::kKBytes);
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint64_t da = make_smem_desc(sq + (kk >> 2) * L::kQHalf + (kk & 3) * 32, 16, 1024, kSwizzle128B);
          const uint64_t db = make_smem_desc(sk + (kk >> 2) * L::kKVHalf + (kk & 3) * 32, 16, 1024, kSwizzle128B);
          umma_f16(tmem_base + T_S + s * BKV, da, db, idesc_s, kk > 0 ? 1u : 0u);
        }
        umma_commit(&kempty[st]);
        umma_commit(&bar_s[s]);
        return true;
      };
      bool ok = mbar_wait(bar_q, 0, abort_flag, p.err);
      if (ok) ok = issue_s(0);
      if (ok && n_blocks > 1) ok = issue_s(1);
      for (int j = 0; j < n_blocks && ok; ++j) {
        const int s = j & 1, st = j % ST;
        if (!mbar_wait(&bar_p[s], static_cast<uint32_t>(j >> 1) & 1, abort_flag, p.err)) break;
        if (!mbar_wait(&vfull[st], static_cast<uint32_t>(j / ST) & 1, abort_flag, p.err)) break;
        tc_fence_after();
        const uint32_t sv = smem_u32(smem + L::kV + st * L::kVBytes);
#pragma unroll
        for (int kk = 0; kk < BKV / 16; ++kk) {
          const uint64_t da = make_smem_desc(sp + kk * 32, 16, 1024, kSwizzle128B);
          // V tile [position][d]: 64-column chunks kKVHalf apart, 16 positions = 2048 bytes
          const uint64_t db = make_smem_desc(sv + kk * 2048, L::kKVHalf, 1024, kSwizzle128B);
          umma_f16(tmem_base + T_O, da, db, idesc_o, (j > 0 || kk > 0) ? 1u : 0u);
        }
        umma_commit(&vempty[st]);
        umma_commit(&bar_o[s]);
        if (j + 2 < n_blocks && !issue_s(j + 2)) break;      // S of block j was read before bar_p completed
      }
    }
  } else {
    // ================================================================ softmax + epilogue (warps 0..3)
    const int r = warp * 32 + lane;                // row of the tile = TMEM lane
    const int t = r / p.G, head = kvh * p.G + r % p.G;
    const int limit = pos0 + t + 1;                // this row sees positions first .. limit - 1, and those in front of p.keep
    const int first = p.chunk ? (pos0 + t) / p.chunk * p.chunk : limit - min(p.window, limit);
    const bool mine = t < ntok;
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    float m_ref = -1e30f, l = 0.f;
    if (p.sink && mine) {
      m_ref = __bfloat162float(p.sink[head]) * 1.4426950408889634f;
      l = 1.f;
    }
    bool ok = !dead;
    uint8_t* sp = smem + L::kP + r * 128;
    for (int j = 0; j < n_blocks; ++j) {
      const int s = j & 1;
      if (ok) ok = mbar_wait(&bar_s[s], static_cast<uint32_t>(j >> 1) & 1, abort_flag, p.err);
      if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
      tc_fence_after();
      uint32_t raw[64];
      tmem_ld_32x32b_x32(tmem_base + T_S + s * BKV + lane_addr, raw);
      tmem_ld_32x32b_x32(tmem_base + T_S + s * BKV + lane_addr + 32, raw + 32);
      tmem_wait_ld();
      if constexpr (kCap) {
#pragma unroll
        for (int c = 0; c < 64; ++c) raw[c] = __float_as_uint(p.cap_log2 * bounded(p.cap_in * __uint_as_float(raw[c])));
      }
      const int at = block_at(j) * BKV;
      const int lim = limit - at, low = first - at, kept = p.keep - at;      // columns low .. lim - 1 are seen, and those in front of `kept`
      float mx = -1e30f;
      if (__all_sync(0xffffffffu, lim >= BKV && (low <= 0 || kept >= BKV))) {
#pragma unroll
        for (int c = 0; c < 64; ++c) mx = fmaxf(mx, __uint_as_float(raw[c]));
      } else {
#pragma unroll
        for (int c = 0; c < 64; ++c) {
          if (c >= lim || (c < low && c >= kept)) raw[c] = 0xff800000u;      // -inf
          mx = fmaxf(mx, __uint_as_float(raw[c]));
        }
      }
      mx *= p.scale_log2;                          // (the scale is positive)
      // the previous product must have finished before P is overwritten or O is rescaled
      if (j > 0) {
        if (ok) ok = mbar_wait(&bar_o[s ^ 1], static_cast<uint32_t>((j - 1) >> 1) & 1, abort_flag, p.err);
        if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
        tc_fence_after();
      }
      const bool grow = mx > m_ref + 8.f;
      if (__any_sync(0xffffffffu, grow)) {
        const float alpha = grow ? exp2f(m_ref - mx) : 1.f;
        if (grow) m_ref = mx;
        l *= alpha;
        if (j > 0) {
#pragma unroll 1
          for (int c = 0; c < DV / 32; ++c) {
            uint32_t o[32];
            tmem_ld_32x32b_x32(tmem_base + T_O + lane_addr + c * 32, o);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st_32x32b_x32(tmem_base + T_O + lane_addr + c * 32, o);
          }
          tmem_wait_st();
        }
      }
      float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
      for (int c8 = 0; c8 < 8; ++c8) {
        float e[8];
#pragma unroll
        for (int i = 0; i < 8; i += 2) {
          e[i] = exp2f(fmaf(__uint_as_float(raw[c8 * 8 + i]), p.scale_log2, -m_ref));
          e[i + 1] = exp2f(fmaf(__uint_as_float(raw[c8 * 8 + i + 1]), p.scale_log2, -m_ref));
          sum0 += e[i];
          sum1 += e[i + 1];
        }
        uint4 pk;
        pk.x = pack_bf16(e[0], e[1]);
        pk.y = pack_bf16(e[2], e[3]);
        pk.z = pack_bf16(e[4], e[5]);
        pk.w = pack_bf16(e[6], e[7]);
        *reinterpret_cast<uint4*>(sp + ((c8 ^ (r & 7)) << 4)) = pk;
      }
      l += sum0 + sum1;
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(&bar_p[s]);
    }
    // gates of 32 columns at a time are fetched ahead of their use
    const __nv_bfloat16* gate = p.gate && !p.head_gate && mine ? p.gate + static_cast<size_t>(row0 + t) * p.ld_gate + head * p.out_d : nullptr;
    uint4 g[4];
    auto fetch = [&](int c) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (gate && c + i * 8 < p.out_d) g[i] = *reinterpret_cast<const uint4*>(gate + c + i * 8);
    };
    fetch(0);
    if (ok) ok = mbar_wait(&bar_o[(n_blocks - 1) & 1], static_cast<uint32_t>((n_blocks - 1) >> 1) & 1, abort_flag, p.err);
    const bool all_ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    float inv_l = l > 0.f ? 1.f / l : 0.f;
    if (p.gate && p.head_gate && mine)
      inv_l = __fdividef(inv_l, 1.f + __expf(-__bfloat162float(p.gate[static_cast<size_t>(row0 + t) * p.ld_gate + head])));
    __nv_bfloat16* out = p.out + ((static_cast<size_t>(row0 + t) * p.H + head) * gridDim.z + blockIdx.z) * p.out_d;
    if (all_ok) {
#pragma unroll 1
      for (int c = 0; c < DV / 32; ++c) {
        if (c * 32 >= p.out_d) break;
        uint32_t o[32];
        tmem_ld_32x32b_x32(tmem_base + T_O + lane_addr + c * 32, o);
        tmem_wait_ld();
        if (gate) {
#pragma unroll
          for (int i = 0; i < 4; ++i) gate8(o + 8 * i, g[i]);
          fetch(c * 32 + 32);
        }
        if (mine) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (c * 32 + i * 8 < p.out_d) {
              uint4 pk;
              pk.x = pack_bf16(__uint_as_float(o[8 * i]) * inv_l, __uint_as_float(o[8 * i + 1]) * inv_l);
              pk.y = pack_bf16(__uint_as_float(o[8 * i + 2]) * inv_l, __uint_as_float(o[8 * i + 3]) * inv_l);
              pk.z = pack_bf16(__uint_as_float(o[8 * i + 4]) * inv_l, __uint_as_float(o[8 * i + 5]) * inv_l);
              pk.w = pack_bf16(__uint_as_float(o[8 * i + 6]) * inv_l, __uint_as_float(o[8 * i + 7]) * inv_l);
              reinterpret_cast<uint4*>(out + c * 32)[i] = pk;
            }
          }
        }
      }
    }
  }

  if (*abort_flag) __nanosleep(50000);
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc<kTmemCols>(tmem_base);
  }
}

struct Operands {      // widths dk, dv <= DK, DV; q_pitch: elements between two rows of q
  const void* q;
  const void* k;
  const void* v;
  int rows, n, Hkv, dk, dv;
  long long q_pitch;
  uint64_t pool_rows;
  bool wide;                // every head's weights meet the values of every group
};

template <int DK, int DV, bool kCap>
static int launch(const Operands& o, const Params& p, cudaStream_t st) {
  using L = Tile<DK, DV>;
  CUtensorMap tq, tk, tv;
  int rc = encode_tma_3d_16bit(&tq, o.q, o.dk, p.H, o.rows, o.dk, o.q_pitch, 64, p.G, p.tokens);
  if (rc) return rc;
  const uint32_t box = p.first_row || p.page >= BKV ? BKV : p.page;
  rc = encode_tma_3d_16bit(&tk, o.k, o.dk, o.Hkv, o.pool_rows, o.dk, static_cast<uint64_t>(o.Hkv) * o.dk, 64, 1, box);
  if (rc) return rc;
  rc = encode_tma_3d_16bit(&tv, o.v, o.dv, o.Hkv, o.pool_rows, o.dv, static_cast<uint64_t>(o.Hkv) * o.dv, 64, 1, box);
  if (rc) return rc;
  auto kern = paged_flash_kernel<DK, DV, kCap>;
  static bool attr_set = false;
  if (!attr_set) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::kTotal);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr_set = true;
  }
  kern<<<dim3(o.n, o.Hkv, o.wide ? o.Hkv : 1), THREADS, L::kTotal, st>>>(tq, tk, tv, p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

template <bool kCap>
static int dispatch(const Operands& o, const Params& p, cudaStream_t st) {
  const bool wide = o.dv > 64;
  if (o.dk > 128) {
    if constexpr (kCap) return -20;
    else return wide ? launch<192, 128, kCap>(o, p, st) : launch<192, 64, kCap>(o, p, st);
  }
  if (o.dk > 64) return wide ? launch<128, 128, kCap>(o, p, st) : launch<128, 64, kCap>(o, p, st);
  return wide ? launch<64, 128, kCap>(o, p, st) : launch<64, 64, kCap>(o, p, st);
}

}  // namespace pf
}  // namespace rb

// q [rows][Hq][dk], pools [pool_rows][Hkv][dk / dv] (dk, dv: 64 or 128, dk also 192), out [rows][Hq][out_d].  blocks [n][4]: query tiles of at
// most 128 / (Hq / Hkv) tokens, every row in exactly one (null: n = rows, one row per segment).  window: positions a row sees, its own
// included (0: all), besides the first `keep` of the sequence; chunk > 0: only its own chunk of that many positions; cap > 0: scores s become
// cap tanh(s / cap); wide: every head's weights meet the values of every group, out [rows][Hq][Hkv][out_d], no gate.  gate [rows][ld_gate] or
// null.  Returns -20 for shapes outside that.
extern "C" int rb_paged_flash(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx, const int* blocks,
                              const void* sink, const void* gate, int ld_gate, void* out, int rows, int n, int Hq, int Hkv, int dk, int dv, int out_d,
                              long long pool_rows, int page, int max_blocks, int window, int keep, int chunk, int wide, float scale, float cap, int* err,
                              cudaStream_t st) {
  using namespace rb;
  using namespace rb::pf;
  if (rows <= 0 || n <= 0) return 0;
  if (Hkv < 1 || Hq % Hkv || keep < 0 || chunk < 0 || cap < 0.f || (wide && gate) || (keep && !window) || (chunk && window)) return -2;
  const int G = Hq / Hkv;
  if (G > BQ || Hkv > 65535 || dk % 64 || dk < 64 || dk > 192 || (dv != 64 && dv != 128) || out_d % 8 || out_d > dv || out_d < 1) return -20;
  if ((page != 16 && page != 32 && page % 64) || scale <= 0.f) return -20;
  if (window < 0 || (gate && (ld_gate % 8 || ld_gate < Hq * out_d || reinterpret_cast<uintptr_t>(gate) % 16))) return -2;
  Params p{};
  p.blocks = blocks; p.ctx = ctx; p.block_tables = block_tables; p.sink = (const __nv_bfloat16*)sink; p.out = (__nv_bfloat16*)out;
  p.gate = (const __nv_bfloat16*)gate; p.ld_gate = ld_gate; p.window = window ? window : INT_MAX;
  p.H = Hq; p.G = G; p.tokens = BQ / G; p.max_blocks = max_blocks; p.page = page; p.out_d = out_d;
  p.keep = keep; p.chunk = chunk;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.err = err;
  const Operands o{q, kc, vc, rows, n, Hkv, dk, dv, static_cast<long long>(Hq) * dk, static_cast<uint64_t>(pool_rows), wide != 0};
  if (cap <= 0.f) return dispatch<false>(o, p, st);
  p.scale_log2 = 1.f;
  p.cap_in = scale / cap;
  p.cap_log2 = cap * 1.4426950408889634f;
  return dispatch<true>(o, p, st);
}

// The same without pages: segment s has its keys and values [rows][H][dk / dv] (dk up to 192, dv up to 128, multiples of 8) from row first[s] on, every
// head its own.  q [rows][H][dk] with q_pitch elements between rows; out [rows][H][dv]; blocks: query tiles of at most 128 tokens; gate
// [rows][ld_gate]: one per head (head_gate) or per output feature, or null.  Returns -20 for shapes outside that.
extern "C" int rb_dense_flash(const void* q, long long q_pitch, const void* k, const void* v, const int* first, const int* blocks, const void* gate,
                              int ld_gate, int head_gate, void* out, int rows, int n, int H, int dk, int dv, long long k_rows, float scale, int* err,
                              cudaStream_t st) {
  using namespace rb;
  using namespace rb::pf;
  if (rows <= 0 || n <= 0) return 0;
  if (H < 1 || H > 65535 || dk % 8 || dk < 8 || dk > 192 || dv % 8 || dv < 8 || dv > 128 || q_pitch % 8 || q_pitch < static_cast<long long>(H) * dk || scale <= 0.f)
    return -20;
  const uintptr_t bases = reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v);
  if (bases % 16 || !first || !blocks) return -2;
  if (gate && !head_gate && (ld_gate % 8 || ld_gate < H * dv || reinterpret_cast<uintptr_t>(gate) % 16)) return -2;
  Params p{};
  p.blocks = blocks; p.first_row = first; p.out = (__nv_bfloat16*)out;
  p.gate = (const __nv_bfloat16*)gate; p.ld_gate = ld_gate; p.head_gate = head_gate; p.window = INT_MAX;
  p.H = H; p.G = 1; p.tokens = BQ; p.max_blocks = 1; p.page = BKV; p.out_d = dv;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.err = err;
  return dispatch<false>({q, k, v, rows, n, H, dk, dv, q_pitch, static_cast<uint64_t>(k_rows), false}, p, st);
}
