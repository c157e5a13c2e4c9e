// HGRN2 over prompt segments, 16 tokens at a time, with the matrix products on the tensor cores.
//
// Per head (gate g in [0, 1] per channel, k = 1 - g, state S [dk][dv]) a chunk of 16 tokens that starts from S is
//
//   q~_t = q_t * prod_{u <= t} g_u          k^_s = k_s * prod_{u > s} g_u          G = prod_u g_u
//   a_ts = sum_d q_t k_s prod_{s < u <= t} g_u   (s <= t)
//   o_t  = S^T q~_t + sum_s a_ts v_s        S <- diag(G) S + sum_s k^_s v_s^T
//
// All decays are running PRODUCTS of gates, never exponentials of sums or quotients: every factor is at most one, so
// nothing overflows however far a gate closes, and what underflows is zero in the exact result too.
//
// A warp keeps S^T for 16 value columns in registers as fp32 accumulator fragments of mma.m16n8k16 (the 16-token chunk is
// exactly its k), so the state never leaves the registers inside a segment, and an accumulator pair is the A fragment
// of the read-out product as it stands.  The state path is exact to fp32: v is bf16 and k^ is split into three bf16
// parts (24 bits) whose products accumulate in fp32.  The read-out, which is rounded to bf16 anyway, uses two parts of
// q~, S and a (17 bits).  CTA = (segment, head), all value columns: gates and a_ts are computed once, half of the warps
// build the products along time while the other half builds a_ts, and the per-head norm is applied before the output is
// written.
// The same kernel serves linear attention whose rows decay by gates of their own (kGla): k and q are projections, the gates
// g = sigmoid(z) ^ r come from an fp32 projection, and the normed output is multiplied by silu of a gate per feature.
#include "common.cuh"
#include "host_utils.h"

namespace rb {
namespace hc {

constexpr int CH = 16;
// Long segments are cut into SPANS that run side by side: kStates computes what a span adds to a zero state and the product
// of its gates, span_scan_kernel chains the spans of a segment, kFromScratch computes the outputs from the chained states.
// kWhole: every segment is one span and carries its state itself.
enum Mode { kWhole = 0, kStates = 1, kFromScratch = 2 };

struct Params {
  const __nv_bfloat16* qfv;      // [T][ld]: q (H*dim) | f (H*dim) | v (H*vdim)
  const __nv_bfloat16* f_bias;
  const __nv_bfloat16* lower;
  const __nv_bfloat16* norm_w;
  float* state;                  // [slots][H][dim][vp]
  const int* slot;
  const int* ctx;
  const int* cu;
  __nv_bfloat16* out;            // [T][ldo]
  const int* spans;              // [n][2]: first and last + 1 row (not kWhole)
  float* span_state;             // [n][H][dim][vp]: kStates: sum of the span; kFromScratch: state at its start
  float* span_gate;              // [n][H][dim]
  int H, dim, vdim, vp, ld, ldo;
  float eps;
  // kGla: qfv is q (H*dim) | k (H*dim) | v (H*vdim) and, from column gate_col on, output gates (H*vdim); f_bias joins z
  const float* z;                // [T][ldz]
  int ldz, gate_col;
  float q_scale, inv_root;
};

__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ float lo16(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float hi16(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
// (a, b) = bf16 pair `h` + remainder left in a, b
__device__ __forceinline__ uint32_t split_off(float& a, float& b) {
  const uint32_t h = pack_bf16(a, b);
  a -= lo16(h);
  b -= hi16(h);
  return h;
}
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
union Pair {
  unsigned long long u;
  float2 f;
};

template <int NP>
__device__ __forceinline__ void load_pairs(Pair* d, const float* p) {
  if constexpr (NP == 2) {
    const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
    d[0].u = v.x;
    d[1].u = v.y;
  } else {
    d[0].u = *reinterpret_cast<const unsigned long long*>(p);
  }
}
// 16 bytes global -> shared, zeros when `in` is false
__device__ __forceinline__ void copy16(void* dst, const void* src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copies_landed() { asm volatile("cp.async.wait_all;" ::: "memory"); }

template <int DK, int NW, bool kGla>
struct Smem {
  static constexpr int GP = DK + 4;                  // fp32 row pitch
  static constexpr int DP = DK + 8;                  // bf16 row pitch of the products (conflict-free ldmatrix)
  static constexpr int VP = NW * 16 + 8;             // bf16 row pitch of v and of the output tile
  float g[CH][GP], k[CH][GP], q[CH][GP];
  float G[DK], fb[DK], fl[DK];
  float red[NW][CH];
  __nv_bfloat16 qh[CH][DP], ql[CH][DP];              // q~
  __nv_bfloat16 kh[CH][DP], km[CH][DP], kl[CH][DP];  // k^
  __nv_bfloat16 ah[CH][24], al[CH][24];              // a_ts
  __nv_bfloat16 v[CH][VP], o[CH][VP];
  __nv_bfloat16 rq[CH][DK], rf[CH][DK], rv[CH][NW * 16];   // raw projections on their way in
  float rz[kGla ? CH : 1][DK];
  __nv_bfloat16 rg[kGla ? CH : 1][NW * 16];
};

template <int DK, int NW, int kMode, bool kGla>
__global__ void __launch_bounds__(NW * 32, NW == 8 ? 2 : 3) hgrn2_chunk_kernel(const Params p) {
  constexpr int NT = NW * 32, UQ = (2 * DK + NT - 1) / NT, TILES = DK / 8;
  extern __shared__ __align__(16) uint8_t raw_smem[];
  using S_ = Smem<DK, NW, kGla>;
  S_& sm = *reinterpret_cast<S_*>(raw_smem);
  const int seg = blockIdx.x, hd = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int lo = kMode == kWhole ? p.cu[seg] : p.spans[2 * seg], hi = kMode == kWhole ? p.cu[seg + 1] : p.spans[2 * seg + 1];
  const int qd = p.H * p.dim;
  const bool fresh = kMode == kStates || (kMode == kWhole && p.ctx[seg] == hi - lo);
  float* S = kMode == kWhole ? p.state + (static_cast<long long>(p.slot[seg]) * p.H + hd) * p.dim * p.vp
                             : p.span_state + (static_cast<long long>(seg) * p.H + hd) * p.dim * p.vp;

  // state fragments: tile j holds channels 8 j + (lane % 4) * 2 + {0, 1} of value columns warp * 16 + lane / 4 + {0, 8}
  const int fd = (lane & 3) * 2, fv = warp * 16 + (lane >> 2);
  float s[TILES][4];
#pragma unroll
  for (int j = 0; j < TILES; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = j * 8 + fd + (e & 1), v = fv + (e >> 1) * 8;
      s[j][e] = (!fresh && d < p.dim && v < p.vp) ? S[static_cast<long long>(d) * p.vp + v] : 0.f;
    }
  for (int i = tid; i < CH * 24; i += NT) {
    (&sm.ah[0][0])[i] = __float2bfloat16(0.f);
    (&sm.al[0][0])[i] = __float2bfloat16(0.f);
  }

  // raw projections of the next chunk, eight channels of one token per unit: a thread copies (asynchronously) exactly what
  // it will read itself, so the copies need no barrier
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < UQ; ++i) {
      const int u = tid + i * NT, t = u / (DK / 8), d = (u % (DK / 8)) * 8;
      if (u < 2 * DK) {
        const bool in = t0 + t < hi && d < p.dim;
        const __nv_bfloat16* a = in ? p.qfv + static_cast<long long>(t0 + t) * p.ld + hd * p.dim + d : p.qfv;
        if (kMode != kStates) copy16(&sm.rq[t][d], a, in);
        copy16(&sm.rf[t][d], in ? a + qd : a, in);
        if constexpr (kGla) {
          const float* z = in ? p.z + static_cast<long long>(t0 + t) * p.ldz + hd * p.dim + d : p.z;
          copy16(&sm.rz[t][d], z, in);
          copy16(&sm.rz[t][d + 4], in ? z + 4 : z, in);
        }
      }
    }
    const int t = tid / (NW * 2), c = (tid % (NW * 2)) * 8;
    const bool in = t0 + t < hi && c < p.vdim;
    copy16(&sm.rv[t][c], in ? p.qfv + static_cast<long long>(t0 + t) * p.ld + 2 * qd + hd * p.vdim + c : p.qfv, in);
    if constexpr (kGla && kMode != kStates)
      copy16(&sm.rg[t][c], in ? p.qfv + static_cast<long long>(t0 + t) * p.ld + p.gate_col + hd * p.vdim + c : p.qfv, in);
  };
  for (int d = tid; d < DK; d += NT) {      // padding channels: gate 1, nothing is written
    sm.fb[d] = d < p.dim ? __bfloat162float(p.f_bias[hd * p.dim + d]) : 0.f;
    if constexpr (!kGla) sm.fl[d] = d < p.dim ? __bfloat162float(p.lower[hd * p.dim + d]) : 1.f;
  }
  __syncthreads();
  float gate0 = 1.f, gate1 = 1.f;             // kStates: product of the span's gates (threads DK / 2 .. DK - 1)
  const int dpre = (tid % (DK / 8)) * 8;      // the channels this thread prepares, the same for all of its units
  fetch(lo);
  for (int t0 = lo; t0 < hi; t0 += CH) {
    const int n = min(CH, hi - t0);
    // ---------------------------------------------------------------- gates and activations of the chunk
    copies_landed();
#pragma unroll
    for (int i = 0; i < UQ; ++i) {
      const int u = tid + i * NT, t = u / (DK / 8);
      if (u < 2 * DK) {
        const uint4 uq = kMode != kStates ? *reinterpret_cast<const uint4*>(&sm.rq[t][dpre]) : make_uint4(0, 0, 0, 0);
        const uint4 uf = *reinterpret_cast<const uint4*>(&sm.rf[t][dpre]);
        const uint32_t wq[4] = {uq.x, uq.y, uq.z, uq.w}, wf[4] = {uf.x, uf.y, uf.z, uf.w};
        float g[8], k[8], q[8];
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          const float x = (c & 1) ? hi16(wq[c >> 1]) : lo16(wq[c >> 1]);
          if constexpr (kGla) {      // tokens and channels behind the last one: gate 1, k = 0
            const float z = sm.rz[t][dpre + c] + sm.fb[dpre + c], e = __expf(-fabsf(z));
            // log(1 + e) of small e keeps its leading digits
            const float l = fminf(z, 0.f) - (e < 1e-3f ? e * (1.f - 0.5f * e) : __logf(1.f + e));
            const bool in = t < n && dpre + c < p.dim;
            g[c] = in ? __expf(l * p.inv_root) : 1.f;
            k[c] = in ? ((c & 1) ? hi16(wf[c >> 1]) : lo16(wf[c >> 1])) : 0.f;
            q[c] = x * p.q_scale;
            continue;
          }
          const float f = ((c & 1) ? hi16(wf[c >> 1]) : lo16(wf[c >> 1])) + sm.fb[dpre + c];
          // one exponential of -|f| gives both halves of the gate without overflow or cancellation
          // (and likewise for silu; the two denominators lie in [1, 2] and share one reciprocal)
          const float e = __expf(-fabsf(f)), ex = __expf(-fabsf(x)), both = __fdividef(1.f, (1.f + e) * (1.f + ex));
          const float r = both * (1.f + ex), er = e * r, rx = both * (1.f + e);
          const float low = sm.fl[dpre + c], span = 1.f - low;
          k[c] = t < n ? span * (f >= 0.f ? er : r) : 0.f;
          g[c] = f >= 0.f || t >= n ? 1.f - k[c] : low + span * er;      // from the side on which the small part is known
          q[c] = x * (x >= 0.f ? rx : ex * rx);
        }
#pragma unroll
        for (int c = 0; c < 8; c += 4) {
          *reinterpret_cast<float4*>(&sm.g[t][dpre + c]) = make_float4(g[c], g[c + 1], g[c + 2], g[c + 3]);
          *reinterpret_cast<float4*>(&sm.k[t][dpre + c]) = make_float4(k[c], k[c + 1], k[c + 2], k[c + 3]);
          if (kMode != kStates) *reinterpret_cast<float4*>(&sm.q[t][dpre + c]) = make_float4(q[c], q[c + 1], q[c + 2], q[c + 3]);
        }
      }
    }
    *reinterpret_cast<uint4*>(&sm.v[tid / (NW * 2)][(tid % (NW * 2)) * 8]) = *reinterpret_cast<const uint4*>(&sm.rv[tid / (NW * 2)][(tid % (NW * 2)) * 8]);
    uint4 out_gate = make_uint4(0, 0, 0, 0);      // of the eight output columns that this thread stores
    if constexpr (kGla && kMode != kStates) out_gate = *reinterpret_cast<const uint4*>(&sm.rg[tid / (NW * 2)][(tid % (NW * 2)) * 8]);
    __syncthreads();
    if (t0 + CH < hi) fetch(t0 + CH);
    // ---------------------------------------------------------------- products along time: one thread per channel pair
    if (tid < DK) {
      const int d = (tid % (DK / 2)) * 2;
      float a = 1.f, b = 1.f;
      if (tid < DK / 2) {
        if (kMode != kStates) {
#pragma unroll
        for (int tb = 0; tb < CH; tb += 4) {      // four tokens are read before any is written
          float2 g[4], q[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            g[j] = *reinterpret_cast<const float2*>(&sm.g[tb + j][d]);
            q[j] = *reinterpret_cast<const float2*>(&sm.q[tb + j][d]);
          }
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            a *= g[j].x;
            b *= g[j].y;
            float x = q[j].x * a, y = q[j].y * b;
            *reinterpret_cast<uint32_t*>(&sm.qh[tb + j][d]) = split_off(x, y);
            *reinterpret_cast<uint32_t*>(&sm.ql[tb + j][d]) = pack_bf16(x, y);
          }
        }
        }
      } else {
#pragma unroll
        for (int tb = CH - 4; tb >= 0; tb -= 4) {
          float2 g[4], k[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            g[j] = *reinterpret_cast<const float2*>(&sm.g[tb + j][d]);
            k[j] = *reinterpret_cast<const float2*>(&sm.k[tb + j][d]);
          }
#pragma unroll
          for (int j = 3; j >= 0; --j) {
            float x = k[j].x * a, y = k[j].y * b;
            a *= g[j].x;
            b *= g[j].y;
            *reinterpret_cast<uint32_t*>(&sm.kh[tb + j][d]) = split_off(x, y);
            *reinterpret_cast<uint32_t*>(&sm.km[tb + j][d]) = split_off(x, y);
            *reinterpret_cast<uint32_t*>(&sm.kl[tb + j][d]) = pack_bf16(x, y);
          }
        }
        *reinterpret_cast<float2*>(&sm.G[d]) = make_float2(a, b);
        if (kMode == kStates) {
          gate0 *= a;
          gate1 *= b;
        }
      }
    }
    // ---------------------------------------------------------------- a_ts: a warp has four source tokens and the rows of
    // all later ones; every lane owns DK / 32 channels, so a row of gates is read once for the four sources
    if (kMode != kStates && (NW == 4 || warp >= 4)) {
      const int s0 = (warp & 3) * 4, c = lane * (DK / 32);
      constexpr int NP = DK / 64;      // channel pairs per lane
      Pair P[4][NP];                   // k_s times the gates since s
#pragma unroll
      for (int i = 0; i < 4; ++i) load_pairs<NP>(P[i], &sm.k[s0 + i][c]);
      for (int tb = s0; tb < n; tb += 4) {
        float r[16];                   // [source][token]
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          Pair g[NP], q[NP];
          load_pairs<NP>(g, &sm.g[tb + j][c]);
          load_pairs<NP>(q, &sm.q[tb + j][c]);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            Pair acc;
            acc.u = 0ull;
#pragma unroll
            for (int e = 0; e < NP; ++e) {
              if (tb > s0 || j > i) P[i][e].u = mul2(P[i][e].u, g[e].u);      // in the first group: gates up to the source do not count
              acc.u = fma2(P[i][e].u, q[e].u, acc.u);
            }
            r[i * 4 + j] = acc.f.x + acc.f.y;
          }
        }
        // sums of sixteen values over the lanes: halves change places, lane pair l / 2 ends up with value index
        int index = 0;
#pragma unroll
        for (int half = 8, mask = 16; half > 0; half >>= 1, mask >>= 1) {
          const bool up = lane & mask;
          index += up ? half : 0;
#pragma unroll
          for (int i = 0; i < half; ++i) {
            const float keep = up ? r[i + half] : r[i], give = up ? r[i] : r[i + half];
            r[i] = keep + __shfl_xor_sync(0xffffffffu, give, mask);
          }
        }
        r[0] += __shfl_xor_sync(0xffffffffu, r[0], 1);
        const int src = s0 + (index >> 2), t = tb + (index & 3);
        if ((lane & 1) == 0 && t >= src) {
          const __nv_bfloat16 h = __float2bfloat16(r[0]);
          sm.ah[t][src] = h;
          sm.al[t][src] = __float2bfloat16(r[0] - __bfloat162float(h));
        }
      }
    }
    __syncthreads();
    // ---------------------------------------------------------------- read-out and state update on the tensor cores
    float o[2][4], ox[2][4];      // leading parts and corrections: two shorter chains of dependent products
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[i][e] = ox[i][e] = 0.f;
    const int mi = lane >> 3, mr = lane & 7;             // matrix and row this lane addresses for ldmatrix
    uint32_t va[4];                                      // V^T: rows = value columns, k = tokens
    ldsm4_t(va, &sm.v[(mi >> 1) * 8 + mr][warp * 16 + (mi & 1) * 8]);
    if constexpr (kMode != kStates) {
      uint32_t bh[4], bl[4];
      ldsm4(bh, &sm.ah[(mi >> 1) * 8 + mr][(mi & 1) * 8]);
      ldsm4(bl, &sm.al[(mi >> 1) * 8 + mr][(mi & 1) * 8]);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mma_bf16(o[i], va, bh[2 * i], bh[2 * i + 1]);
        mma_bf16(ox[i], va, bl[2 * i], bl[2 * i + 1]);
      }
    }
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      if constexpr (kMode != kStates) {
      uint32_t ah[4], al[4], bh[4], bl[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float x = s[2 * kk + (i >> 1)][(i & 1) * 2], y = s[2 * kk + (i >> 1)][(i & 1) * 2 + 1];
        ah[i] = split_off(x, y);
        al[i] = pack_bf16(x, y);
      }
      ldsm4(bh, &sm.qh[(mi >> 1) * 8 + mr][kk * 16 + (mi & 1) * 8]);
      ldsm4(bl, &sm.ql[(mi >> 1) * 8 + mr][kk * 16 + (mi & 1) * 8]);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mma_bf16(o[i], ah, bh[2 * i], bh[2 * i + 1]);
        mma_bf16(ox[i], ah, bl[2 * i], bl[2 * i + 1]);
        mma_bf16(ox[i], al, bh[2 * i], bh[2 * i + 1]);
      }
      }
      // both state tiles of this step have been read: decay them and add the chunk's writes
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float2 G = *reinterpret_cast<const float2*>(&sm.G[(2 * kk + i) * 8 + fd]);
        s[2 * kk + i][0] *= G.x;
        s[2 * kk + i][1] *= G.y;
        s[2 * kk + i][2] *= G.x;
        s[2 * kk + i][3] *= G.y;
      }
      uint32_t b[4];
      const int row = (mi & 1) * 8 + mr, col = kk * 16 + (mi >> 1) * 8;
      ldsm4_t(b, &sm.kh[row][col]);
      mma_bf16(s[2 * kk], va, b[0], b[1]);
      mma_bf16(s[2 * kk + 1], va, b[2], b[3]);
      ldsm4_t(b, &sm.km[row][col]);
      mma_bf16(s[2 * kk], va, b[0], b[1]);
      mma_bf16(s[2 * kk + 1], va, b[2], b[3]);
      ldsm4_t(b, &sm.kl[row][col]);
      mma_bf16(s[2 * kk], va, b[0], b[1]);
      mma_bf16(s[2 * kk + 1], va, b[2], b[3]);
    }
    if constexpr (kMode == kStates) {
      __syncthreads();      // the next chunk rewrites what the products above have read
    } else {
    // ---------------------------------------------------------------- norm over the head's value columns
    // o[i][e]: token i * 8 + fd + (e & 1), value column fv + (e >> 1) * 8
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[i][e] += ox[i][e];
    float ss[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      ss[i] = o[i >> 1][i & 1] * o[i >> 1][i & 1] + o[i >> 1][2 + (i & 1)] * o[i >> 1][2 + (i & 1)];
#pragma unroll
      for (int w = 4; w < 32; w <<= 1) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], w);
    }
    if (lane < 4) {
#pragma unroll
      for (int i = 0; i < 4; ++i) sm.red[warp][(i >> 1) * 8 + fd + (i & 1)] = ss[i];
    }
    __syncthreads();
    {
      const float w0 = fv < p.vdim ? __bfloat162float(p.norm_w[fv]) : 0.f, w1 = fv + 8 < p.vdim ? __bfloat162float(p.norm_w[fv + 8]) : 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = (i >> 1) * 8 + fd + (i & 1);
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < NW; ++w) sum += sm.red[w][t];
        const float r = 1.f / sqrtf(sum / p.vdim + p.eps);
        sm.o[t][fv] = __float2bfloat16(o[i >> 1][i & 1] * r * w0);
        sm.o[t][fv + 8] = __float2bfloat16(o[i >> 1][2 + (i & 1)] * r * w1);
      }
    }
    __syncthreads();
    {
      const int t = tid / (NW * 2), c = (tid % (NW * 2)) * 8;
      if (t < n && c < p.vdim) {
        uint4 o = *reinterpret_cast<const uint4*>(&sm.o[t][c]);
        if constexpr (kGla) {
          uint32_t* w = reinterpret_cast<uint32_t*>(&o);
          const uint32_t gw[4] = {out_gate.x, out_gate.y, out_gate.z, out_gate.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float a = lo16(gw[i]), b = hi16(gw[i]);
            w[i] = pack_bf16(lo16(w[i]) * __fdividef(a, 1.f + __expf(-a)), hi16(w[i]) * __fdividef(b, 1.f + __expf(-b)));
          }
        }
        *reinterpret_cast<uint4*>(p.out + static_cast<long long>(t0 + t) * p.ldo + hd * p.vdim + c) = o;
      }
    }
    }
  }
  if (kMode == kFromScratch) return;
  asm volatile("" : "+l"(S));      // addresses are computed again here instead of living in registers all along
  if (kMode == kStates && tid >= DK / 2 && tid < DK) {
    const int d = (tid - DK / 2) * 2;
    float* g = p.span_gate + (static_cast<long long>(seg) * p.H + hd) * p.dim + d;
    if (d < p.dim) g[0] = gate0;
    if (d + 1 < p.dim) g[1] = gate1;
  }
#pragma unroll
  for (int j = 0; j < TILES; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = j * 8 + fd + (e & 1), v = fv + (e >> 1) * 8;
      if (d < p.dim && v < p.vp) S[static_cast<long long>(d) * p.vp + v] = s[j][e];
    }
}

// chains the spans of a segment: what kStates left in span_state[i] becomes the state at the start of span i
__global__ void __launch_bounds__(256) span_scan_kernel(const Params p, const int* __restrict__ first) {
  const int seg = blockIdx.x, hd = blockIdx.y;
  const int q4 = p.vp / 4, i = blockIdx.z * 256 + threadIdx.x;
  if (i >= p.dim * q4) return;
  const int d = i / q4;
  const int a = first[seg], b = first[seg + 1];
  const bool fresh = p.ctx[seg] == p.spans[2 * b - 1] - p.spans[2 * a];
  const long long head = static_cast<long long>(p.dim) * p.vp, off = static_cast<long long>(i) * 4;
  float4* S = reinterpret_cast<float4*>(p.state + (static_cast<long long>(p.slot[seg]) * p.H + hd) * head + off);
  float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *S;
  for (int k = a; k < b; ++k) {
    float4* D = reinterpret_cast<float4*>(p.span_state + (static_cast<long long>(k) * p.H + hd) * head + off);
    const float4 x = *D;
    const float g = p.span_gate[(static_cast<long long>(k) * p.H + hd) * p.dim + d];
    *D = s;
    s.x = g * s.x + x.x;
    s.y = g * s.y + x.y;
    s.z = g * s.z + x.z;
    s.w = g * s.w + x.w;
  }
  *S = s;
}

template <int DK, int NW, int kMode, bool kGla>
static int launch_mode(const Params& p, int n, cudaStream_t st) {
  auto k = hgrn2_chunk_kernel<DK, NW, kMode, kGla>;
  const int smem = static_cast<int>(sizeof(Smem<DK, NW, kGla>));
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr = true;
  }
  k<<<dim3(n, p.H), NW * 32, smem, st>>>(p);
  rb_note_launch(1);
  return static_cast<int>(cudaGetLastError());
}
template <int DK, int NW, bool kGla>
static int launch(const Params& p, int segs, int spans, const int* first, cudaStream_t st) {
  if (!spans) return launch_mode<DK, NW, kWhole, kGla>(p, segs, st);
  int rc = launch_mode<DK, NW, kStates, kGla>(p, spans, st);
  if (rc) return rc;
  span_scan_kernel<<<dim3(segs, p.H, (p.dim * (p.vp / 4) + 255) / 256), 256, 0, st>>>(p, first);
  rb_note_launch(1);
  return launch_mode<DK, NW, kFromScratch, kGla>(p, spans, st);
}

template <bool kGla>
static int dispatch(const Params& p, int segs, int n_spans, const int* first, cudaStream_t st) {
  if (p.dim <= 64) return p.vdim <= 64 ? launch<64, 4, kGla>(p, segs, n_spans, first, st) : launch<64, 8, kGla>(p, segs, n_spans, first, st);
  return p.vdim <= 64 ? launch<128, 4, kGla>(p, segs, n_spans, first, st) : launch<128, 8, kGla>(p, segs, n_spans, first, st);
}

}  // namespace hc
}  // namespace rb

// bf16 segments (cu [segs + 1]) of heads with dim and vdim multiples of 8 up to 128; ldo = H * vdim.  n_spans > 0: spans
// [n_spans][2] rows, those of segment s being first[s] .. first[s + 1], with scratch for their states and gates; 0: every
// segment runs as a whole.  Returns -20 outside that range.
extern "C" int rb_hgrn2_chunk(const void* qfv, const void* f_bias, const void* lower, const void* norm_w, float* state, const int* slot, const int* ctx,
                              const int* cu, const int* spans, const int* first, float* span_state, float* span_gate, void* out, int rows, int segs,
                              int n_spans, int H, int dim, int vdim, int vp, int ld, int ldo, float eps, cudaStream_t st) {
  using namespace rb;
  using namespace rb::hc;
  if (rows <= 0 || segs <= 0) return 0;
  if (dim % 8 || vdim % 8 || dim > 128 || vdim > 128 || ld % 8 || ldo != H * vdim || vp < vdim || vp % 4 || H > 65535) return -20;
  if ((reinterpret_cast<uintptr_t>(qfv) % 16) || (reinterpret_cast<uintptr_t>(out) % 16)) return -20;
  if (n_spans && (!spans || !first || !span_state || !span_gate)) return -2;
  Params p{static_cast<const __nv_bfloat16*>(qfv), static_cast<const __nv_bfloat16*>(f_bias), static_cast<const __nv_bfloat16*>(lower),
           static_cast<const __nv_bfloat16*>(norm_w), state, slot, ctx, cu, static_cast<__nv_bfloat16*>(out), spans, span_state, span_gate,
           H, dim, vdim, vp, ld, ldo, eps};
  return dispatch<false>(p, segs, n_spans, first, st);
}

// The same for linear attention with decaying rows: in [T][ld] is q | k | v and, from gate_col on, output gates; z [T][ldz] fp32.
extern "C" int rb_gla_chunk(const void* in, const float* z, int ldz, const void* z_bias, const void* norm_w, float* state, const int* slot, const int* ctx,
                            const int* cu, const int* spans, const int* first, float* span_state, float* span_gate, void* out, int rows, int segs,
                            int n_spans, int H, int dim, int vdim, int vp, int ld, int ldo, int gate_col, float eps, float q_scale, float inv_root,
                            cudaStream_t st) {
  using namespace rb;
  using namespace rb::hc;
  if (rows <= 0 || segs <= 0) return 0;
  if (dim % 8 || vdim % 8 || dim > 128 || vdim > 128 || ld % 8 || ldo != H * vdim || vp < vdim || vp % 4 || H > 65535 || ldz % 4 || gate_col % 8) return -20;
  if ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(z)) % 16) return -20;
  if (n_spans && (!spans || !first || !span_state || !span_gate)) return -2;
  Params p{static_cast<const __nv_bfloat16*>(in), static_cast<const __nv_bfloat16*>(z_bias), nullptr, static_cast<const __nv_bfloat16*>(norm_w), state, slot,
           ctx, cu, static_cast<__nv_bfloat16*>(out), spans, span_state, span_gate, H, dim, vdim, vp, ld, ldo, eps, z, ldz, gate_col, q_scale, inv_root};
  return dispatch<true>(p, segs, n_spans, first, st);
}
