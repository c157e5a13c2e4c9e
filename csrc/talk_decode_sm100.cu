// Paged decode attention whose heads' weights are mixed before they meet the values, on the 5th-generation tensor cores.
//
//   out_h = sum_j (sum_g T[h][g] p_g(j)) v_j  =  sum_g T[h][g] (P_g V)         (V of head h's own group)
//
// The mixing is linear, so every head's weights may meet the values of every group first, and T joins when the splits are merged:
// no second pass over the scores is needed for their denominators.  One CTA serves ALL heads of a sequence (and split), so keys and
// values are read once, and the products with the other groups' values cost tensor-core columns that a decode step has to spare.
//
//   S^T_c[128 tokens][16]        = K_c[128][DK] Q_c^T                 group c's heads, padded to the MMA's 16 columns
//   O^T_c[DV][all heads]        += V_c^T[DV][128 tokens] P^T          P: all heads, packed
//
// Scores are capped (s <- cap tanh(s / cap)), which bounds them: the softmax needs no running maximum, its reference is 0, nothing is ever
// rescaled, and partial results of splits just add up.  Warps 0-3: softmax (one thread per token row) and epilogue, warp 4: TMA (page
// by page into one ring of K and V tiles, in the order of their use), warp 5: MMA.  Every wait is bounded; no load uses cluster multicast.
#include <limits.h>

#include "common.cuh"
#include "host_utils.h"

namespace rb {
namespace td {

constexpr int TILE = 128;                       // tokens per tile
constexpr int THREADS = 192;
constexpr int HALF = TILE * 128;                // 16 KB: 64 columns of a tile
constexpr int kMaxBuf = 12;
constexpr int kMaxCols = 128;                   // packed head columns
constexpr int kTmemCols = 512;

struct Params {
  const __nv_bfloat16* q;   // [B][H][DK]
  const int* block_tables;  // [B][max_blocks]
  const int* ctx_lens;      // [B]
  float* part_o;            // [B][splits][G][cols][128]
  float* part_l;            // [B][splits][cols]
  int H, G, rep, cols, nv, nbuf, max_blocks, page, num_splits, split_tokens;      // cols: packed heads rounded up to 16; nv: value groups per CTA
  int window, keep, chunk;  // as in decode_attn_tc
  int q_at, p_at, bar_at;   // bytes into shared memory
  float cap_in, cap_log2;
  int* err;
};

// REPP: heads of a group, rounded up (4, 8 or 16); group c's heads are the packed columns c * REPP ..
template <int DK, int DV, int REPP>
__global__ void __launch_bounds__(THREADS, 1)
talk_decode_kernel(const __grid_constant__ CUtensorMap tma_k, const __grid_constant__ CUtensorMap tma_v, const Params p) {
  constexpr int BUF = (DK > DV ? DK : DV) * 256;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + p.bar_at);
  uint64_t* bar_s = bars;             // [2] scores of a tile are complete
  uint64_t* bar_p = bars + 2;         // [2] its weights are written, its scores are read
  uint64_t* bar_o = bars + 4;         // [2] its products are in the accumulators
  uint64_t* full = bars + 6;          // [nbuf]
  uint64_t* empty = full + kMaxBuf;   // [nbuf]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(empty + kMaxBuf);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* red = reinterpret_cast<float*>(tmem_slot + 2);      // [4][kMaxCols]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.x, v0 = blockIdx.y * p.nv, split = blockIdx.z;
  const int nv = min(p.nv, p.G - v0), G = p.G;
  const int ctx = p.ctx_lens[b];
  const int from = p.chunk ? (ctx - 1) / p.chunk * p.chunk : max(0, ctx - p.window);      // first position of the chunk or window
  const int first = from / p.page, kept = min((p.keep + p.page - 1) / p.page, first);      // pages: 0 .. kept - 1, then first ..
  const int total = kept * p.page + ctx - first * p.page;
  const int t_begin = split * p.split_tokens, t_end = min(total, t_begin + p.split_tokens);
  const int n_tiles = t_end > t_begin ? (t_end - t_begin + TILE - 1) / TILE : 0;
  const int* bt = p.block_tables + static_cast<size_t>(b) * p.max_blocks;
  auto page_at = [&](int i) { return i < kept ? i : first + i - kept; };

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bar_s[i], 1);
      mbar_init(&bar_p[i], 128);
      mbar_init(&bar_o[i], 1);
    }
    for (int s = 0; s < p.nbuf; ++s) {
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
  // stage Q (16 rows per group, those behind the group's heads zero) and clear P, both in the swizzled K-major layout
  for (int i = threadIdx.x; i < G * 2 * 16 * 8; i += THREADS) {
    const int c = i >> 8, half = (i >> 7) & 1, row = (i >> 3) & 15, k = i & 7;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row < p.rep && half * 64 < DK) v = *reinterpret_cast<const uint4*>(p.q + (static_cast<size_t>(b) * p.H + c * p.rep + row) * DK + half * 64 + k * 8);
    *reinterpret_cast<uint4*>(smem + p.q_at + c * 4096 + half * 2048 + row * 128 + ((k ^ (row & 7)) << 4)) = v;
  }
  for (int i = threadIdx.x; i < p.cols * 32; i += THREADS) *reinterpret_cast<uint4*>(smem + p.p_at + i * 16) = make_uint4(0, 0, 0, 0);
  fence_proxy_async();
  if (warp == 5) {
    tmem_alloc<kTmemCols>(tmem_slot);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t s_cols = static_cast<uint32_t>(G) * 16;      // columns of a score buffer
  const uint32_t t_o = 2 * s_cols;
  const bool dead = (*abort_flag != 0);

  if (warp == 4) {
    // ================================================================ TMA producer (page gather)
    if (lane == 0 && !dead) {
      tma_prefetch_desc(&tma_k);
      tma_prefetch_desc(&tma_v);
      int u = 0;
      auto load = [&](const CUtensorMap* map, bool two, int group, int j) -> bool {
        const int s = u % p.nbuf;
        if (!mbar_wait(&empty[s], (static_cast<uint32_t>(u / p.nbuf) & 1) ^ 1, abort_flag, p.err)) return false;
        ++u;
        uint8_t* dst = smem + s * BUF;
        mbar_expect_tx(&full[s], two ? 2 * HALF : HALF);
        const int page0 = (t_begin + j * TILE) / p.page;
        for (int pg = 0; pg < TILE / p.page; ++pg) {
          const int row = bt[min(page_at(page0 + pg), p.max_blocks - 1)] * p.page;
          tma_load_3d(dst + pg * p.page * 128, map, &full[s], 0, group, row);
          if (two) tma_load_3d(dst + HALF + pg * p.page * 128, map, &full[s], 64, group, row);
        }
        return true;
      };
      auto keys = [&](int j) {
        bool ok = true;
        for (int c = 0; c < G && ok; ++c) ok = load(&tma_k, DK == 128, c, j);
        return ok;
      };
      bool ok = n_tiles > 0 && keys(0);
      if (ok && n_tiles > 1) ok = keys(1);
      for (int j = 0; j < n_tiles && ok; ++j) {
        for (int c = 0; c < nv && ok; ++c) ok = load(&tma_v, DV == 128, v0 + c, j);
        if (ok && j + 2 < n_tiles) ok = keys(j + 2);
      }
    }
  } else if (warp == 5) {
    // ================================================================ MMA issuer
    if (lane == 0 && !dead && n_tiles > 0) {
      const uint32_t id_s = make_idesc_f16(128, 16, true, false, false);            // K tile x Q^T, both K-major
      const uint32_t id_o = make_idesc_f16(128, p.cols, true, true, false);         // V^T (MN-major) x P (K-major)
      const uint32_t sq = smem_u32(smem + p.q_at), sp = smem_u32(smem + p.p_at);
      const uint32_t p_half = static_cast<uint32_t>(p.cols) * 128;                  // 64 tokens of all columns
      int u = 0;
      auto wait_tile = [&](uint32_t& at) -> bool {
        const int s = u % p.nbuf;
        if (!mbar_wait(&full[s], static_cast<uint32_t>(u / p.nbuf) & 1, abort_flag, p.err)) return false;
        tc_fence_after();
        at = smem_u32(smem + s * BUF);
        return true;
      };
      auto done_tile = [&]() { umma_commit(&empty[u % p.nbuf]); ++u; };
      auto issue_s = [&](int j) -> bool {
        for (int c = 0; c < G; ++c) {
          uint32_t sk;
          if (!wait_tile(sk)) return false;
#pragma unroll
          for (int kk = 0; kk < DK / 16; ++kk) {
            const uint64_t da = make_smem_desc(sk + (kk >> 2) * HALF + (kk & 3) * 32, 16, 1024, kSwizzle128B);
            const uint64_t db = make_smem_desc(sq + c * 4096 + (kk >> 2) * 2048 + (kk & 3) * 32, 16, 1024, kSwizzle128B);
            umma_f16(tmem_base + (j & 1) * s_cols + c * 16, da, db, id_s, kk > 0 ? 1u : 0u);
          }
          done_tile();
        }
        umma_commit(&bar_s[j & 1]);
        return true;
      };
      bool ok = issue_s(0);
      if (ok && n_tiles > 1) ok = issue_s(1);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (!mbar_wait(&bar_p[j & 1], static_cast<uint32_t>(j >> 1) & 1, abort_flag, p.err)) break;
        tc_fence_after();
        for (int c = 0; c < nv && ok; ++c) {
          uint32_t sv;
          ok = wait_tile(sv);
          if (!ok) break;
#pragma unroll
          for (int kk = 0; kk < TILE / 16; ++kk) {
            const uint64_t da = make_smem_desc(sv + kk * 2048, HALF, 1024, kSwizzle128B);      // M = features, two 64-wide chunks
            const uint64_t db = make_smem_desc(sp + (j & 1) * 2 * p_half + (kk >> 2) * p_half + (kk & 3) * 32, 16, 1024, kSwizzle128B);
            umma_f16(tmem_base + t_o + c * p.cols, da, db, id_o, (j > 0 || kk > 0) ? 1u : 0u);
          }
          done_tile();
        }
        if (!ok) break;
        umma_commit(&bar_o[j & 1]);
        if (j + 2 < n_tiles) ok = issue_s(j + 2);      // the scores of tile j were read before bar_p completed
      }
    }
  } else {
    // ================================================================ softmax + epilogue (warps 0..3)
    constexpr int GB = 32 / REPP;                 // groups per batch of 32 packed columns
    constexpr int LD = REPP > 8 ? 16 : 8;         // columns fetched per group
    const int r = warp * 32 + lane;               // token row of S^T, feature row of O^T
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    float l[kMaxCols / 32];                       // lane k: sum of packed column 32 * batch + k over this warp's tokens
#pragma unroll
    for (int i = 0; i < kMaxCols / 32; ++i) l[i] = 0.f;
    bool ok = !dead;
    for (int j = 0; j < n_tiles; ++j) {
      if (ok) ok = mbar_wait(&bar_s[j & 1], static_cast<uint32_t>(j >> 1) & 1, abort_flag, p.err);
      if (ok && j >= 2) ok = mbar_wait(&bar_o[j & 1], static_cast<uint32_t>((j - 2) >> 1) & 1, abort_flag, p.err);      // P of tile j - 2 was read
      if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
      tc_fence_after();
      const int i = t_begin + j * TILE + r, tok = page_at(i / p.page) * p.page + i % p.page;
      const bool valid = i < t_end && (tok >= from || tok < p.keep);
      uint8_t* prow = smem + p.p_at + (j & 1) * p.cols * 256 + (r >> 6) * p.cols * 128 + ((r & 7) << 1);
      const int chunk16 = (r & 63) >> 3;
#pragma unroll
      for (int batch = 0; batch < kMaxCols / 32; ++batch) {
        if (batch * GB < G) {
          float e[32];
#pragma unroll
          for (int gb = 0; gb < GB; ++gb) {
            uint32_t raw[LD];
            const int c = min(batch * GB + gb, G - 1);
            if constexpr (LD == 16) tmem_ld_32x32b_x16(tmem_base + (j & 1) * s_cols + c * 16 + lane_addr, raw);
            else tmem_ld_32x32b_x8(tmem_base + (j & 1) * s_cols + c * 16 + lane_addr, raw);
            tmem_wait_ld();
#pragma unroll
            for (int h = 0; h < REPP; ++h) {
              // tanh in fp32 up to about 1e-7 (2 / ln 2)
              const float x = 2.8853900817779268f * fminf(p.cap_in * __uint_as_float(raw[h]), 20.f);
              const float s = p.cap_log2 * (1.f - __fdividef(2.f, 1.f + exp2f(x)));
              e[gb * REPP + h] = valid && h < p.rep && batch * GB + gb < G ? exp2f(s) : 0.f;
            }
          }
#pragma unroll
          for (int k = 0; k < 32; ++k) {
            const int col = batch * 32 + k;
            if (col < p.cols) *reinterpret_cast<__nv_bfloat16*>(prow + col * 128 + ((chunk16 ^ (col & 7)) << 4)) = __float2bfloat16(e[k]);
          }
          // sums over the warp's tokens: halves change places, lane k ends up with column k
#pragma unroll
          for (int half = 16; half > 0; half >>= 1) {
            const bool up = lane & half;
#pragma unroll
            for (int k = 0; k < half; ++k) {
              const float mine = up ? e[k + half] : e[k], give = up ? e[k] : e[k + half];
              e[k] = mine + __shfl_xor_sync(0xffffffffu, give, half);
            }
          }
          l[batch] += e[0];
        }
      }
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(&bar_p[j & 1]);
    }
    if (ok && n_tiles > 1) ok = mbar_wait(&bar_o[(n_tiles - 2) & 1], static_cast<uint32_t>((n_tiles - 2) >> 1) & 1, abort_flag, p.err);
    if (ok && n_tiles > 0) ok = mbar_wait(&bar_o[(n_tiles - 1) & 1], static_cast<uint32_t>((n_tiles - 1) >> 1) & 1, abort_flag, p.err);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    const size_t part = static_cast<size_t>(b) * p.num_splits + split;
    for (int c = 0; c < nv; ++c) {
      float* out = p.part_o + ((part * G + v0 + c) * p.cols) * 128 + r;
      for (int col = 0; col < p.cols; col += 16) {
        uint32_t o[16];
        if (n_tiles > 0 && ok) {
          tmem_ld_32x32b_x16(tmem_base + t_o + c * p.cols + col + lane_addr, o);
          tmem_wait_ld();
        } else {
#pragma unroll
          for (int k = 0; k < 16; ++k) o[k] = 0;
        }
        if (r < DV) {
#pragma unroll
          for (int k = 0; k < 16; ++k) out[(col + k) * 128] = __uint_as_float(o[k]);
        }
      }
    }
#pragma unroll
    for (int batch = 0; batch < kMaxCols / 32; ++batch) red[warp * kMaxCols + batch * 32 + lane] = l[batch];
    named_bar_sync(1, 128);
    if (blockIdx.y == 0 && r < p.cols) p.part_l[part * p.cols + r] = red[r] + red[kMaxCols + r] + red[2 * kMaxCols + r] + red[3 * kMaxCols + r];
  }

  if (*abort_flag) __nanosleep(50000);
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc<kTmemCols>(tmem_base);
  }
}

// Merges the splits, divides by the sums (the sink's exponential included) and mixes the heads.  CTA = (sequence, group): the group's heads
// read what every head's weights made of the group's values.
struct MergeParams {
  const float* part_o;
  const float* part_l;
  const __nv_bfloat16* sink;      // [H] or null
  const __nv_bfloat16* mix;       // [H][H]
  __nv_bfloat16* out;             // [B][H][out_d]
  int H, G, rep, repp, cols, splits, out_d;
};
constexpr int MG_WARPS = 8;      // every warp takes every eighth head g; a lane has four features
template <int REPP>
__global__ void __launch_bounds__(MG_WARPS * 32) talk_merge_kernel(const MergeParams p) {
  __shared__ float inv[kMaxCols];
  extern __shared__ __align__(16) float sm[];      // [H][REPP]: what head i of this group takes of head g; then [MG_WARPS][REPP][128] sums
  float* sums = sm + p.H * REPP;
  const int b = blockIdx.x, c = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, d = (tid & 31) * 4;
  for (int g = tid; g < p.H; g += MG_WARPS * 32) {
    const int col = g / p.rep * REPP + g % p.rep;
    float l = p.sink ? exp2f(__bfloat162float(p.sink[g]) * 1.4426950408889634f) : 0.f;
#pragma unroll 4
    for (int s = 0; s < p.splits; ++s) l += p.part_l[(static_cast<size_t>(b) * p.splits + s) * p.cols + col];
    inv[g] = l > 0.f ? 1.f / l : 0.f;
  }
  for (int i = tid; i < p.H * REPP; i += MG_WARPS * 32) {
    const int g = i / REPP, h = i - g * REPP;
    sm[i] = h < p.rep ? __bfloat162float(p.mix[static_cast<size_t>(c * p.rep + h) * p.H + g]) : 0.f;
  }
  __syncthreads();
  float4 acc[REPP];
#pragma unroll
  for (int i = 0; i < REPP; ++i) acc[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  const float* base = p.part_o + (static_cast<size_t>(b) * p.splits * p.G + c) * p.cols * 128 + d;
  const size_t step = static_cast<size_t>(p.G) * p.cols * 128;
  if (d < p.out_d) {      // (features behind the values' columns were never written)
    for (int g = warp; g < p.H; g += MG_WARPS) {
      const float* src = base + static_cast<size_t>(g / p.rep * REPP + g % p.rep) * 128;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (int s = 0; s < p.splits; ++s) {
        const float4 x = *reinterpret_cast<const float4*>(src + s * step);
        a.x += x.x; a.y += x.y; a.z += x.z; a.w += x.w;
      }
      const float f = inv[g];
#pragma unroll
      for (int i = 0; i < REPP; ++i) {
        const float m = sm[g * REPP + i] * f;
        acc[i].x += m * a.x; acc[i].y += m * a.y; acc[i].z += m * a.z; acc[i].w += m * a.w;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < REPP; ++i) *reinterpret_cast<float4*>(sums + (warp * REPP + i) * 128 + d) = acc[i];
  __syncthreads();
  for (int i = tid; i < p.rep * 128; i += MG_WARPS * 32) {
    const int h = i >> 7, k = i & 127;
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < MG_WARPS; ++w) o += sums[(w * REPP + h) * 128 + k];
    if (k < p.out_d) p.out[(static_cast<size_t>(b) * p.H + c * p.rep + h) * p.out_d + k] = __float2bfloat16(o);
  }
}

struct Plan {
  int repp, cols, nv, nbuf, q_at, p_at, bar_at, total;
};
// 0 when the kernel takes these heads
static int plan(int H, int G, int dk, int dv, Plan& o) {
  if (G < 1 || H % G || (dk != 64 && dk != 128) || (dv != 64 && dv != 128)) return -20;
  const int rep = H / G;
  if (rep > 16 || H > 1024) return -20;
  o.repp = rep <= 4 ? 4 : rep <= 8 ? 8 : 16;
  o.cols = (G * o.repp + 15) / 16 * 16;
  if (o.cols > kMaxCols || 32 * G > kTmemCols) return -20;
  o.nv = (kTmemCols - 32 * G) / o.cols;
  if (o.nv > G) o.nv = G;
  if (o.nv < 1) return -20;
  const int buf = (dk > dv ? dk : dv) * 256, q = G * 4096, w = o.cols * 512;
  const int tail = 512 + 4 * kMaxCols * 4;
  int rest = q + w + tail;
  if (rest < HALF) rest = HALF;      // the discarded half of 64-column values lies in shared memory
  o.nbuf = (226 * 1024 - rest) / buf;
  if (o.nbuf > kMaxBuf) o.nbuf = kMaxBuf;
  if (o.nbuf < 2) return -20;
  o.q_at = o.nbuf * buf;
  o.p_at = o.q_at + q;
  o.bar_at = o.p_at + w;
  o.total = o.q_at + rest;
  return 0;
}

template <int DK, int DV, int REPP>
static int launch(const void* kc, const void* vc, uint64_t slots, const Params& p, const Plan& o, int B, cudaStream_t st) {
  CUtensorMap tk, tv;
  int rc = encode_tma_3d_16bit(&tk, kc, DK, p.G, slots, DK, static_cast<uint64_t>(p.G) * DK, 64, 1, p.page);
  if (rc) return rc;
  rc = encode_tma_3d_16bit(&tv, vc, DV, p.G, slots, DV, static_cast<uint64_t>(p.G) * DV, 64, 1, p.page);
  if (rc) return rc;
  auto kern = talk_decode_kernel<DK, DV, REPP>;
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr = true;
  }
  kern<<<dim3(B, (p.G + p.nv - 1) / p.nv, p.num_splits), THREADS, o.total, st>>>(tk, tv, p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}
template <int REPP>
static int dispatch(int dk, int dv, const void* kc, const void* vc, uint64_t slots, const Params& p, const Plan& o, const MergeParams& m, int B, cudaStream_t st) {
  int rc;
  if (dk == 128) rc = dv == 128 ? launch<128, 128, REPP>(kc, vc, slots, p, o, B, st) : launch<128, 64, REPP>(kc, vc, slots, p, o, B, st);
  else rc = dv == 128 ? launch<64, 128, REPP>(kc, vc, slots, p, o, B, st) : launch<64, 64, REPP>(kc, vc, slots, p, o, B, st);
  if (rc) return rc;
  const int smem = (m.H + MG_WARPS * 128) * REPP * 4;
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(talk_merge_kernel<REPP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (kMaxCols + MG_WARPS * 128) * REPP * 4);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr = true;
  }
  talk_merge_kernel<REPP><<<dim3(B, m.G), MG_WARPS * 32, smem, st>>>(m);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace td
}  // namespace rb

// Packed head columns and value groups per CTA for these heads; 0: the kernel does not take them.
extern "C" int rb_talk_decode_plan(int H, int G, int dk, int dv, int* value_groups) {
  rb::td::Plan o;
  if (rb::td::plan(H, G, dk, dv, o)) return 0;
  *value_groups = o.nv;
  return o.cols;
}

// q [B][H][dk] over pools [rows][G][dk / dv] (64 or 128 columns), pages of 16 to 128 tokens; out [B][H][out_d] = mixed heads.  cap: in (0, 80];
// sinks of up to 88.  window / keep / chunk and max_ctx as in rb_paged_decode_tc.  Scratch: part_o [B][splits][G][cols][128] and part_l
// [B][splits][cols] fp32.  Returns -20 for shapes outside that.
extern "C" int rb_talk_decode(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx_lens, const void* sink, const void* mix,
                              void* out, float* part_o, float* part_l, int B, int H, int G, int dk, int dv, int out_d, long long pool_rows, int page,
                              int max_blocks, int max_ctx, int window, int keep, int chunk, float scale, float cap, int splits, int* err, cudaStream_t st) {
  using namespace rb;
  using namespace rb::td;
  if (B == 0) return 0;
  Plan o;
  if (plan(H, G, dk, dv, o) || out_d > dv || out_d < 1 || cap <= 0.f || cap > 80.f || scale <= 0.f) return -20;
  if ((page != 16 && page != 32 && page != 64 && page != 128) || splits < 1 || splits > 65535) return -20;
  if (window < 0 || keep < 0 || chunk < 0 || (chunk && window) || (keep && !window)) return -2;
  const long long most = chunk ? static_cast<long long>(chunk) + page : window + static_cast<long long>(keep) + 2 * page;
  if ((chunk || window) && most < max_ctx) max_ctx = static_cast<int>(most);
  Params p{};
  p.q = static_cast<const __nv_bfloat16*>(q); p.block_tables = block_tables; p.ctx_lens = ctx_lens; p.part_o = part_o; p.part_l = part_l;
  p.H = H; p.G = G; p.rep = H / G; p.cols = o.cols; p.nv = o.nv; p.nbuf = o.nbuf; p.max_blocks = max_blocks; p.page = page; p.num_splits = splits;
  p.split_tokens = ((max_ctx + splits - 1) / splits + TILE - 1) / TILE * TILE;
  p.window = window ? window : INT_MAX; p.keep = keep; p.chunk = chunk;
  p.q_at = o.q_at; p.p_at = o.p_at; p.bar_at = o.bar_at;
  p.cap_in = scale / cap;
  p.cap_log2 = cap * 1.4426950408889634f;
  p.err = err;
  const MergeParams m{part_o, part_l, static_cast<const __nv_bfloat16*>(sink), static_cast<const __nv_bfloat16*>(mix), static_cast<__nv_bfloat16*>(out),
                      H, G, H / G, o.repp, o.cols, splits, out_d};
  const uint64_t slots = static_cast<uint64_t>(pool_rows);
  if (o.repp == 4) return dispatch<4>(dk, dv, kc, vc, slots, p, o, m, B, st);
  if (o.repp == 8) return dispatch<8>(dk, dv, kc, vc, slots, p, o, m, B, st);
  return dispatch<16>(dk, dv, kc, vc, slots, p, o, m, B, st);
}
