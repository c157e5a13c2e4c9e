// Attention over paged latent rows on the 5th-generation tensor cores.
//
// In latent attention every head's keys and values are linear maps of ONE cached row per token.  With those maps folded
// into the queries (and applied to the attended rows afterwards) a tile of latent rows is key and value of all heads at
// once, so a CTA streams each row once and serves a group of up to N (token, head) query columns with it:
//
//   S^T[128 positions][N]   = C_tile[128][R]   * Q^T            (Q: N absorbed queries, K-major)
//   O^T[Rv][N]             += C_tile^T[Rv][128] * P              (the same tile, read MN-major in place)
//
// Rows may end in features that only join the scores (a rotated key part: Rv < R): their slots are free again as soon as S has read
// them.
// The columns of a group belong to one sequence: the heads of one decoded token, or of several consecutive tokens of a
// prompt portion, each with its own causal limit.  Rows are gathered page by page with TMA into the 128-byte swizzled
// layout; a ring of 32 KB slots (128 positions x 128 latent features) keeps loads in flight while a tile is processed: a
// slot is free again when the O product has read it.  Two threads share a position of S^T (and a latent feature of
// O^T), each with half of the columns; maxima are shared by the CTA, the accumulator is rescaled lazily (threshold 2^8, decided for the whole CTA).
// CTA = (column group, split of the positions); partial results of several splits are merged by a second kernel, which
// also applies the output gate.  Every wait is bounded; no load uses cluster multicast.
#include "common.cuh"
#include "host_utils.h"

namespace rb {
namespace la {

constexpr int TILE = 128;                 // positions per tile
constexpr int SLOT = 32768;               // ring slot: two 64-feature chunks of a tile
constexpr int MAX_SLOTS = 5;
constexpr int SOFTMAX = 256;               // eight warps: positions by warp % 4, columns by halves
constexpr int THREADS = SOFTMAX + 64;      // and a TMA and an MMA warp
constexpr int SCRATCH = 2560;               // barriers (256 B), then 8 N words

struct Params {
  const int* items;          // [n][4]: segment, first column, columns, base; null: one row per segment (decode)
  const int* block_tables;   // [S][max_blocks]
  const int* ctx;            // [S] (decode)
  const __nv_bfloat16* gate; // [rows][ld_gate] or null
  __nv_bfloat16* out;        // [columns][Rv]
  float* part_o;             // [splits][columns][Rv]
  float* part_ml;            // [splits][columns][2]
  int H, Rv;
  int NC, NP, NV;            // 64-feature chunks of a row; slots per tile, the first NV of which hold values
  int slots, max_blocks, page, splits, columns, groups_per_row, ld_gate, ahead;
  float scale_log2;
  int* err;
};

__device__ __forceinline__ float redux_max(float v) {
  float r;
  asm("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(r) : "f"(v));
  return r;
}

// barrier `id` of `threads` threads that also ORs a predicate over them
__device__ __forceinline__ bool named_bar_or(int id, int threads, bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbar.red.or.pred q, %2, %3, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
      : "=r"(r)
      : "r"(static_cast<uint32_t>(v)), "r"(id), "r"(threads)
      : "memory");
  return r != 0;
}

// W consecutive accumulator columns of this warp's 32 lanes
template <int W>
__device__ __forceinline__ void tmem_get(uint32_t addr, uint32_t* r) {
  if constexpr (W == 8) tmem_ld_32x32b_x8(addr, r);
  else tmem_ld_32x32b_x16(addr, r);
}
template <int W>
__device__ __forceinline__ void tmem_put(uint32_t addr, const uint32_t* r) {
  if constexpr (W == 8) tmem_st_32x32b_x8(addr, r);
  else tmem_st_32x32b_x16(addr, r);
}

template <int N>
struct Layout {
  static constexpr int kP = 2 * N * 128;                     // one P buffer: two 64-position halves of N rows
  static int total(int slots, int NC) { return slots * SLOT + NC * N * 128 + 2 * kP + SCRATCH; }
};

template <int N>
__global__ void __launch_bounds__(THREADS)
latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_c, const Params p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* sq = smem + p.slots * SLOT;                        // [NC][N rows][128 B]
  uint8_t* sp = sq + p.NC * N * 128;                          // two P buffers
  uint64_t* bars = reinterpret_cast<uint64_t*>(sp + 2 * Layout<N>::kP);
  uint64_t* bar_q = bars;
  uint64_t* bar_s = bars + 1;                                 // [2], like bar_p and bar_o: index = tile & 1
  uint64_t* bar_p = bars + 3;
  uint64_t* bar_o = bars + 5;
  uint64_t* full = bars + 7;                                  // [MAX_SLOTS]
  uint64_t* empty = full + MAX_SLOTS;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(empty + MAX_SLOTS);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* red = reinterpret_cast<float*>(bars + 32);           // [4][N] maxima, later sums
  float* s_m = red + 4 * N;                                   // [N] running reference maximum
  float* s_alpha = s_m + N;                                   // [N]
  float* s_gate = s_alpha + N;                                // [N]
  int* s_lim = reinterpret_cast<int*>(s_gate + N);            // [N] positions a column sees

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int kTmemCols = N == 16 ? 128 : (N == 32 ? 256 : 512);      // (2 + NV) * N columns, NV <= 4
  constexpr int T_S = 0, T_O = 2 * N;

  int seg, col0, ncols, base;
  if (p.items) {
    const int4 it = reinterpret_cast<const int4*>(p.items)[blockIdx.x];
    seg = it.x; col0 = it.y; ncols = it.z; base = it.w;
  } else {
    seg = blockIdx.x / p.groups_per_row;
    const int part = blockIdx.x - seg * p.groups_per_row;
    col0 = seg * p.H + part * N;
    ncols = min(N, p.H - part * N);
    base = p.ctx[seg] - seg;
  }
  const int first_lim = base + col0 / p.H;                    // fewest / most positions seen by a column of the group
  const int last_lim = base + (col0 + ncols - 1) / p.H;
  const int all_tiles = (last_lim + TILE - 1) / TILE;
  const int per = (all_tiles + p.splits - 1) / p.splits;
  const int split = blockIdx.y;
  const int tile0 = split * per;
  const int n_tiles = max(0, min(all_tiles, tile0 + per) - tile0);
  const int* bt = p.block_tables + static_cast<size_t>(seg) * p.max_blocks;

  if (threadIdx.x == 0) {
    mbar_init(bar_q, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bar_s[i], 1);
      mbar_init(&bar_p[i], SOFTMAX);
      mbar_init(&bar_o[i], 1);
    }
    for (int s = 0; s < p.slots; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    *abort_flag = 0;
    if ((smem_u32(smem) & 1023u) != 0) {
      *abort_flag = 1;
      if (p.err) atomicCAS(p.err, kOk, kErrBadArgument);
    }
    fence_barrier_init();
  }
  for (int n = threadIdx.x; n < N; n += THREADS) {
    const int c = col0 + n, row = c / p.H;
    const bool live = n < ncols;
    s_lim[n] = live ? base + row : 0;
    s_m[n] = -1e30f;
    s_alpha[n] = 1.f;
    float g = 1.f;
    if (live && p.gate) g = 1.f / (1.f + __expf(-__bfloat162float(p.gate[static_cast<size_t>(row) * p.ld_gate + (c - row * p.H)])));
    s_gate[n] = g;
  }
  if (warp == 9) {
    tmem_alloc<kTmemCols>(tmem_slot);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const bool dead = (*abort_flag != 0);

  if (warp == 8) {
    // ================================================================ TMA producer (page gather)
    // lane i gathers page i of every tile: the page number is looked up once per tile and the copies of a slot are issued
    // by all lanes together
    if (!dead && n_tiles > 0) {
      if (lane == 0) {
        mbar_expect_tx(bar_q, p.NC * N * 128);
        for (int c = 0; c < p.NC; ++c) tma_load_2d(sq + c * N * 128, &tma_q, bar_q, c * 64, col0);
      }
      const int pages = TILE / p.page, page_bytes = p.page * 128;
      // pages behind the context: any row, masked
      auto page_row = [&](int j) { return lane < pages ? bt[min((tile0 + j) * pages + lane, p.max_blocks - 1)] * p.page : 0; };
      int row = page_row(0);
      int s = 0;
      uint32_t ph = 1;
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int next = j + 1 < n_tiles ? page_row(j + 1) : 0;
        for (int pr = 0; pr < p.NP; ++pr) {
          ok = mbar_wait(&empty[s], ph, abort_flag, p.err);
          ok = __all_sync(0xffffffffu, ok);
          if (!ok) break;
          const int nch = min(2, p.NC - 2 * pr);
          if (lane == 0) mbar_expect_tx(&full[s], nch * (SLOT / 2));
          __syncwarp();
          uint8_t* dst = smem + s * SLOT + lane * page_bytes;
          if (lane < pages) {
            tma_load_2d(dst, &tma_c, &full[s], pr * 128, row);
            if (nch == 2) tma_load_2d(dst + SLOT / 2, &tma_c, &full[s], pr * 128 + 64, row);
          }
          if (++s == p.slots) { s = 0; ph ^= 1; }
        }
        row = next;
      }
    }
  } else if (warp == 9) {
    // ================================================================ MMA issuer
    if (lane == 0 && !dead && n_tiles > 0) {
      constexpr uint32_t id_s = make_idesc_f16(TILE, N, true, false, false);
      constexpr uint32_t id_o = make_idesc_f16(TILE, N, true, true, false);
      // One thread issues everything, so it must spend few instructions per product: descriptors are formed once and
      // advanced by adding to their address field (units of 16 bytes).
      const uint64_t ring_k = make_smem_desc(smem_u32(smem), 16, 1024, kSwizzle128B);            // tile rows as K-major A
      const uint64_t ring_mn = make_smem_desc(smem_u32(smem), SLOT / 2, 1024, kSwizzle128B);     // the same tile as C^T, MN-major A
      const uint64_t q0 = make_smem_desc(smem_u32(sq), 16, 1024, kSwizzle128B), p0 = make_smem_desc(smem_u32(sp), 16, 1024, kSwizzle128B);
      int ss = 0, so = 0;              // ring slots of the next S and O products
      uint32_t phase = 0;
      auto issue_s = [&](int j) -> bool {
        const uint32_t d = tmem_base + T_S + (j & 1) * N;
        uint64_t db = q0;
        for (int pr = 0; pr < p.NP; ++pr) {
          if (!mbar_wait(&full[ss], phase, abort_flag, p.err)) return false;
          tc_fence_after();
          const uint64_t da = ring_k + static_cast<uint32_t>(ss) * (SLOT >> 4);
          umma_f16(d, da, db, id_s, pr > 0 ? 1u : 0u);
#pragma unroll
          for (int kk = 1; kk < 4; ++kk) umma_f16(d, da + kk * 2, db + kk * 2, id_s, 1u);
          if (2 * pr + 1 < p.NC) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) umma_f16(d, da + (SLOT >> 5) + kk * 2, db + (N * 128 >> 4) + kk * 2, id_s, 1u);
          }
          db += 2 * (N * 128 >> 4);
          if (pr >= p.NV) umma_commit(&empty[ss]);
          if (++ss == p.slots) { ss = 0; phase ^= 1; }
        }
        umma_commit(&bar_s[j & 1]);
        return true;
      };
      bool ok = mbar_wait(bar_q, 0, abort_flag, p.err);
      if (ok) {
        tc_fence_after();
        ok = issue_s(0);
      }
      for (int j = 0; j < n_tiles && ok; ++j) {
        // the ring holds two tiles: the scores of the next tile are computed beside the softmax of this one
        if (p.ahead && j + 1 < n_tiles && !issue_s(j + 1)) break;
        if (!mbar_wait(&bar_p[j & 1], static_cast<uint32_t>(j >> 1) & 1, abort_flag, p.err)) break;
        tc_fence_after();
        const uint64_t db = p0 + static_cast<uint32_t>(j & 1) * (Layout<N>::kP >> 4);
        const uint32_t first = j > 0 ? 1u : 0u;
        for (int pr = 0; pr < p.NV; ++pr) {
          // A: M = 128 latent features (two chunks SLOT / 2 apart), K = 16 positions (2048 bytes).  In the last slot of an odd
          // chunk count the upper 64 rows of the product come from stale data and are never read
          const uint64_t da = ring_mn + static_cast<uint32_t>(so) * (SLOT >> 4);
          const uint32_t d = tmem_base + T_O + pr * N;
          umma_f16(d, da, db, id_o, first);
#pragma unroll
          for (int kk = 1; kk < TILE / 16; ++kk) umma_f16(d, da + kk * 128, db + (kk >> 2) * (N * 128 >> 4) + (kk & 3) * 2, id_o, 1u);
          umma_commit(&empty[so]);
          if (++so == p.slots) so = 0;
        }
        for (int pr = p.NV; pr < p.NP; ++pr)
          if (++so == p.slots) so = 0;
        umma_commit(&bar_o[j & 1]);
        if (!p.ahead && j + 1 < n_tiles && !issue_s(j + 1)) break;
      }
    }
  } else {
    // ================================================================ softmax + epilogue (warps 0..7)
    constexpr int NH = N / 2, CW = NH < 16 ? NH : 16;
    const int quad = warp & 3;
    const int r = quad * 32 + lane;          // position of the tile, latent feature of a pair
    const int n0 = (warp >> 2) * NH;         // this warp's columns
    const uint32_t lane_addr = (static_cast<uint32_t>(quad * 32) << 16) + n0;
    float l_part[NH];
#pragma unroll
    for (int n = 0; n < NH; ++n) l_part[n] = 0.f;
    bool ok = !dead;
    // A wait that runs out only clears `ok`; the loop keeps its shape so that all threads meet at the barriers.
    for (int j = 0; j < n_tiles; ++j) {
      if (ok) ok = mbar_wait(&bar_s[j & 1], static_cast<uint32_t>(j >> 1) & 1, abort_flag, p.err);
      __syncwarp();
      tc_fence_after();
      float s[NH];
#pragma unroll
      for (int c = 0; c < NH; c += CW) tmem_get<CW>(tmem_base + T_S + (j & 1) * N + c + lane_addr, reinterpret_cast<uint32_t*>(s) + c);
      tmem_wait_ld();
      const int tok = (tile0 + j) * TILE + r;
      const bool masked = (tile0 + j + 1) * TILE > first_lim || ncols < N;      // uniform: some column ends inside this tile
      if (masked) {
#pragma unroll
        for (int n = 0; n < NH; ++n)
          if (tok >= s_lim[n0 + n]) s[n] = -INFINITY;
      }
      // distances to the reference maxima; the maxima themselves are reduced only when a score outgrows its reference
      float top = -1e30f;
#pragma unroll
      for (int n = 0; n < NH; n += 4) {
        const float4 m = *reinterpret_cast<const float4*>(s_m + n0 + n);
        top = fmaxf(top, fmaxf(fmaxf(s[n] * p.scale_log2 - m.x, s[n + 1] * p.scale_log2 - m.y),
                               fmaxf(s[n + 2] * p.scale_log2 - m.z, s[n + 3] * p.scale_log2 - m.w)));
      }
      const bool outgrown = named_bar_or(1, SOFTMAX, top > 8.f);
      if (j >= 2 && ok) ok = mbar_wait(&bar_o[j & 1], static_cast<uint32_t>((j - 2) >> 1) & 1, abort_flag, p.err);
      if (outgrown) {
        __syncwarp();
        float mine = 0.f;
#pragma unroll
        for (int n = 0; n < NH; ++n) {
          const float wm = redux_max(s[n] * p.scale_log2);
          if (lane == n) mine = wm;
        }
        if (lane < NH) red[quad * N + n0 + lane] = mine;
        named_bar_sync(1, SOFTMAX);
        if (threadIdx.x < N) {
          const int c = threadIdx.x;
          const float tm = fmaxf(fmaxf(red[c], red[N + c]), fmaxf(red[2 * N + c], red[3 * N + c]));
          const float m = s_m[c];
          s_alpha[c] = tm > m + 8.f ? exp2f(m - tm) : 1.f;
          if (tm > m + 8.f) s_m[c] = tm;
        }
        named_bar_sync(1, SOFTMAX);
#pragma unroll
        for (int n = 0; n < NH; ++n) l_part[n] *= s_alpha[n0 + n];
        if (j > 0) {       // O^T may be rescaled only when the product of tile j - 1 has landed
          if (ok) ok = mbar_wait(&bar_o[(j - 1) & 1], static_cast<uint32_t>((j - 1) >> 1) & 1, abort_flag, p.err);
          __syncwarp();
          tc_fence_after();
#pragma unroll 1
          for (int pr = 0; pr < p.NV; ++pr) {
#pragma unroll
            for (int c = 0; c < NH; c += CW) {
              uint32_t o[CW];
              tmem_get<CW>(tmem_base + T_O + pr * N + c + lane_addr, o);
              tmem_wait_ld();
#pragma unroll
              for (int i = 0; i < CW; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * s_alpha[n0 + c + i]);
              tmem_put<CW>(tmem_base + T_O + pr * N + c + lane_addr, o);
            }
          }
          tmem_wait_st();
        }
      }
      // P[n][position]: K-major, two 64-position halves
      const int half = r >> 6, col = r & 63;
      uint8_t* prow = sp + (j & 1) * Layout<N>::kP + half * N * 128 + n0 * 128 + ((col & 7) << 1);      // n0 is a multiple of 8
#pragma unroll
      for (int n = 0; n < NH; n += 4) {
        const float4 m = *reinterpret_cast<const float4*>(s_m + n0 + n);
        const float mm[4] = {m.x, m.y, m.z, m.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float pv = exp2f(s[n + i] * p.scale_log2 - mm[i]);      // masked: exp2(-inf) = 0
          l_part[n + i] += pv;
          *reinterpret_cast<__nv_bfloat16*>(prow + (n + i) * 128 + (((col >> 3) ^ ((n + i) & 7)) << 4)) = __float2bfloat16(pv);
        }
      }
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(&bar_p[j & 1]);
    }
    if (ok && n_tiles > 1) ok = mbar_wait(&bar_o[(n_tiles - 2) & 1], static_cast<uint32_t>((n_tiles - 2) >> 1) & 1, abort_flag, p.err);
    if (ok && n_tiles > 0) ok = mbar_wait(&bar_o[(n_tiles - 1) & 1], static_cast<uint32_t>((n_tiles - 1) >> 1) & 1, abort_flag, p.err);
    __syncwarp();
    tc_fence_after();
#pragma unroll
    for (int n = 0; n < NH; ++n) {
      const float ws = warp_sum(l_part[n]);
      if (lane == 0) red[quad * N + n0 + n] = ws;
    }
    named_bar_sync(1, SOFTMAX);
#pragma unroll
    for (int n = 0; n < NH; ++n) l_part[n] = red[n0 + n] + red[N + n0 + n] + red[2 * N + n0 + n] + red[3 * N + n0 + n];
    const bool have = n_tiles > 0;           // uniform
    if (p.splits > 1 && static_cast<int>(threadIdx.x) < ncols) {
      const int c = threadIdx.x;
      float* ml = p.part_ml + (static_cast<size_t>(split) * p.columns + col0 + c) * 2;
      ml[0] = s_m[c];
      ml[1] = have && ok ? red[c] + red[N + c] + red[2 * N + c] + red[3 * N + c] : 0.f;
    }
    if (have) {
#pragma unroll 1
      for (int pr = 0; pr < p.NV; ++pr) {
        const int d = pr * 128 + r;
#pragma unroll
        for (int c = 0; c < NH; c += CW) {
          uint32_t o[CW];
          tmem_get<CW>(tmem_base + T_O + pr * N + c + lane_addr, o);
          tmem_wait_ld();
          if (d < p.Rv) {
#pragma unroll
            for (int i = 0; i < CW; ++i) {
              const int n = n0 + c + i;
              if (n < ncols) {
                const float v = __uint_as_float(o[i]);
                if (p.splits == 1)
                  p.out[static_cast<size_t>(col0 + n) * p.Rv + d] = __float2bfloat16(ok && l_part[c + i] > 0.f ? v / l_part[c + i] * s_gate[n] : 0.f);
                else
                  p.part_o[(static_cast<size_t>(split) * p.columns + col0 + n) * p.Rv + d] = v;
              }
            }
          }
        }
      }
    } else if (p.splits == 1) {
      for (int i = threadIdx.x; i < ncols * p.Rv; i += SOFTMAX) p.out[static_cast<size_t>(col0) * p.Rv + i] = __float2bfloat16(0.f);
    }
  }

  if (*abort_flag) __nanosleep(50000);
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc<kTmemCols>(tmem_base);
  }
}

// one CTA per (row, head) column: merges the splits and applies the gate
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                             const __nv_bfloat16* __restrict__ gate, __nv_bfloat16* __restrict__ out,
                                                             int splits, int columns, int H, int R, int ld_gate) {
  const int col = blockIdx.x, lane = threadIdx.x & 31;
  // lane s holds the weight of split s (at most 32 splits; splits without positions weigh nothing)
  float m = -1e30f, l = 0.f;
  if (lane < splits) {
    const float2 ml = *reinterpret_cast<const float2*>(part_ml + (static_cast<size_t>(lane) * columns + col) * 2);
    l = ml.y;
    if (l > 0.f) m = ml.x;
  }
  const float top = warp_max(m);
  const float w = l > 0.f ? exp2f(m - top) : 0.f;
  l = warp_sum(w * l);
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
  for (int s = 0; s < splits; ++s) {
    const float ws = __shfl_sync(0xffffffffu, w, s);
    const float* o = part_o + (static_cast<size_t>(s) * columns + col) * R;
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (ws > 0.f && threadIdx.x + k * 128 < R) acc[k] += ws * o[threadIdx.x + k * 128];
  }
  float f = l > 0.f ? 1.f / l : 0.f;
  if (gate) {
    const int row = col / H;
    f *= 1.f / (1.f + __expf(-__bfloat162float(gate[static_cast<size_t>(row) * ld_gate + (col - row * H)])));
  }
#pragma unroll
  for (int k = 0; k < 4; ++k)
    if (threadIdx.x + k * 128 < R) out[static_cast<size_t>(col) * R + threadIdx.x + k * 128] = __float2bfloat16(acc[k] * f);
}

template <int N>
static int launch(const CUtensorMap& tq, const CUtensorMap& tc, const Params& p, int items, int smem, cudaStream_t st) {
  auto kern = latent_attn_tc_kernel<N>;
  static int attr = 0;
  if (smem > attr) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr = smem;
  }
  kern<<<dim3(items, p.splits), THREADS, smem, st>>>(tq, tc, p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace la
}  // namespace rb

// q [rows][H][R] bf16 (absorbed queries), pool [pool_rows][R] bf16 in pages of `page` rows (16, 32, 64 or 128), out [rows][H][Rv]: the
// first Rv features are values, all R join the scores; both multiples of 64, Rv up to 512, R up to 640.  width: columns per group (16, 32 or 64).  items [n_items][4] or null (one row per segment: ctx is read
// on the device).  part_o / part_ml: scratch for splits > 1.  Returns -20 for shapes outside this range.
extern "C" int rb_latent_attn_tc(const void* q, const void* pool, const int* block_tables, const int* items, const int* ctx, const void* gate,
                                 void* out, float* part_o, float* part_ml, int rows, int H, int R, int Rv, long long pool_rows, int max_blocks, int page,
                                 int n_items, int width, int splits, int ld_gate, float scale, int* err, cudaStream_t st) {
  using namespace rb;
  using namespace rb::la;
  if (rows <= 0) return 0;
  if (!(scale > 0.f)) return -20;            // masking relies on the sign
  if (R % 64 || R > 640 || Rv % 64 || Rv > 512 || Rv > R || Rv < 64 || (page != 16 && page != 32 && page != 64 && page != 128)) return -20;
  if ((width != 16 && width != 32 && width != 64) || splits < 1 || splits > 32 || (splits > 1 && (!part_o || !part_ml))) return -2;
  if ((reinterpret_cast<uintptr_t>(q) % 16) || (reinterpret_cast<uintptr_t>(pool) % 16)) return -2;
  Params p{};
  p.items = items; p.block_tables = block_tables; p.ctx = ctx;
  p.gate = static_cast<const __nv_bfloat16*>(gate); p.out = static_cast<__nv_bfloat16*>(out); p.part_o = part_o; p.part_ml = part_ml;
  p.H = H; p.Rv = Rv; p.NC = R / 64; p.NP = (p.NC + 1) / 2; p.NV = (Rv / 64 + 1) / 2; p.max_blocks = max_blocks; p.page = page; p.splits = splits;
  p.columns = rows * H; p.groups_per_row = (H + width - 1) / width; p.ld_gate = ld_gate;
  p.scale_log2 = scale * 1.4426950408889634f; p.err = err;
  const int fixed = p.NC * width * 128 + 2 * (2 * width * 128) + SCRATCH;
  p.slots = p.NP == 1 ? 3 : MAX_SLOTS;       // one pair: a small CTA, so that two share an SM
  while (p.slots > 0 && p.slots * SLOT + fixed > 227 * 1024) --p.slots;
  if (p.slots < p.NP) return -20;
  p.ahead = p.slots >= 2 * p.NP;
  CUtensorMap tq, tc;
  int rc = encode_tma_2d_bf16(&tq, q, R, static_cast<uint64_t>(rows) * H, R, 64, width);
  if (rc) return rc;
  rc = encode_tma_2d_bf16(&tc, pool, R, pool_rows, R, 64, page);
  if (rc) return rc;
  const int n = items ? n_items : rows * p.groups_per_row;
  const int smem = p.slots * SLOT + fixed;
  rc = width == 16 ? launch<16>(tq, tc, p, n, smem, st) : width == 32 ? launch<32>(tq, tc, p, n, smem, st) : launch<64>(tq, tc, p, n, smem, st);
  if (rc) return rc;
  if (splits > 1)
    latent_combine_kernel<<<p.columns, 128, 0, st>>>(part_o, part_ml, p.gate, p.out, splits, p.columns, H, Rv, ld_gate);
  rb_note_launch(splits > 1 ? 2 : 1);
  return static_cast<int>(cudaGetLastError());
}
