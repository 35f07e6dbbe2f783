// Talking-heads attention, bf16 tensor-core path for ragged prompts and portions (mathematics: talking_attention.cu).
//
// The head mix couples all heads of a (query, key) pair, so one CTA owns 16 (or 8) query rows of one sequence with ALL
// heads and walks the visible keys in tiles of 32:
//
//   QK   a warp holds one or two heads: S = Q K^T on mma.sync m16n8k16, fp32 scores to shared memory
//   mix  a warp owns query rows: soft cap, distance bias, the H x H mix, mask, exp2 -> bf16 weights, which overwrite
//        the scores of the same row.  The mix runs on tensor cores without losing fp32 accuracy: a score is the sum of
//        three bf16 values, the matrix is exact in bf16, so all products are exact (more than eight heads); else, and
//        for matrices that bf16 does not hold, on the FMA pipe with the matrix as constant-bank operands
//   PV   the warp again holds its heads: O += P V, fp32 accumulators in registers; row sums from the same fragments
//
// A tile takes two barrier intervals: its mix, then its PV together with the next tile's QK (two score buffers).
// K of the tile after next and V of the next one arrive (cp.async) during the mix.  Scores are fp32 from the
// accumulator to the exponential.  The running maximum is lazy: a row keeps the reference maximum of an earlier tile
// until a score exceeds it by 2^kSlack, so the ordinary tile needs no reduction over lanes; the maximum only has to
// keep the exponentials in range.
#include <string.h>

#include "talking_attention.cuh"

namespace b200 {
namespace {

constexpr int BK = 32;
constexpr int kSRow = 36;            // floats per score row: 32 keys + padding (odd multiple of 16 bytes)
// floats per head of a tile of `rows` queries: heads two apart start eight banks apart
__host__ __device__ constexpr int plane_floats(int rows) { return rows * kSRow + 4; }
constexpr int kBiasRow = 52;              // biases of one head for the BQ + BK - 1 distances of a tile, padded
constexpr int kQueryInSmem = 1, kTwoScores = 2;
constexpr float kSlack = 30.f;       // log2 of how far a score may exceed the row's reference

constexpr float kNoRef = -3.0e38f;   // reference of a row that has seen no key
constexpr float kLog2e = 1.4426950408889634f;

// the two warps that share a query row of the mix
__device__ __forceinline__ void pair_barrier(int row) { asm volatile("bar.sync %0, 64;" ::"r"(row + 1) : "memory"); }

template <int HP>
struct MixParam {
  float t[HP * HP];                  // talk * log2(e), [out][in], zero-padded
  float r1[HP], r2[HP];
  uint32_t tb[HP * HP / 2];          // talk in bf16 pairs of neighbouring in-heads (tensor-core mix)
};

__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// cap tanh(x scale / cap) - bias; k = 2 log2(e) scale / cap
__device__ __forceinline__ float capped(float x, float k, float cap, float two_cap, float bias) {
  return (cap - bias) - two_cap * rcp_approx(1.f + fast_exp2(x * k));
}

// HP: heads padded; NW: warps; MAXC: value columns per CTA in units of 16; MODE: 0 any constants, 1 soft cap and bias table
// present, 2 also H == HP, 3 as 1 with the mix on tensor cores (a talk matrix of bf16 values); q_smem: the query rows are staged in shared memory (else their fragments are read from global memory)
// PAIR: tiles of eight queries, and the sixteen rows of a warp's MMA tile are those of two neighbouring heads that
// share a key head: half the accumulators per head, so that many or wide heads fit
template <int HP, int NW, int MAXC, int MINB, int MODE, bool PAIR>
__global__ void __launch_bounds__(NW * 32, MINB)
talking_prefill_kernel(const TalkArgs a, const __grid_constant__ MixParam<HP> mp, const int layout) {
  constexpr int BQ = PAIR ? kTalkTileRows / 2 : kTalkTileRows, kPlane = plane_floats(BQ);
  static_assert(!PAIR || (MODE == 3 && HP == 2 * NW), "a pair of heads per warp");
  constexpr bool kHalfRow = PAIR && NW == 16;          // two warps share a query row of the mix
  constexpr int HPW = PAIR ? 1 : HP / NW, kThreads = NW * 32, kTpr = kThreads / BK;    // kTpr: threads that load one key row
  const bool q_smem = layout & kQueryInSmem, two_scores = layout & kTwoScores;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ __align__(16) float s_ref[BQ * HP];     // reference maximum (log2 domain) per (row, head)
  __shared__ float s_cor[2][BQ * HP];  // by tile parity: factor for accumulators and sums, 1 unless the flag is set
  constexpr int kTalkRow = HP / 2 + 4;           // words per row of the matrix, padded against bank conflicts
  __shared__ uint32_t s_talk[MODE == 3 ? HP * kTalkRow : 1];
  __shared__ float s_top[kHalfRow ? 2 * BQ * HP : 1];
  __shared__ int s_up[kHalfRow ? BQ : 1];
  __shared__ int s_flag[2], s_seq, s_tile;       // flag (by tile parity): some reference moved
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int H = MODE == 2 ? HP : a.H, G = a.Hkv, Gs = H / G, dk = a.dk;
  const int dvc = a.dv / gridDim.y, dv0 = blockIdx.y * dvc, nc = dvc / 16;

  // ---- which (sequence, tile): from the step's tile list (heaviest first), or numbered sequence by sequence ----
  if (a.plan) {
    if (static_cast<int>(blockIdx.x) >= a.plan[0]) return;
    if (tid == 0) {
      const uint32_t entry = static_cast<uint32_t>(a.plan[kPlanHeader + blockIdx.x]);
      s_seq = entry >> 16;
      s_tile = entry & 0xffffu;
    }
  } else if (warp == 0) {
    int left = blockIdx.x, seq = -1, tile = 0;
    for (int base = 0; base < a.n && seq < 0; base += 32) {
      const int s = base + lane;
      const int t = s < a.n ? (a.cu_q[s + 1] - a.cu_q[s] + kTalkTileRows - 1) / kTalkTileRows : 0;
      int incl = t;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += y;
      }
      const unsigned hit = __ballot_sync(0xffffffffu, left < incl);
      if (hit) {
        const int src = __ffs(hit) - 1;
        seq = base + src;
        // last tile of the sequence first: it sees the most keys
        tile = __shfl_sync(0xffffffffu, incl, src) - 1 - left;
      } else {
        left -= __shfl_sync(0xffffffffu, incl, 31);
      }
    }
    if (lane == 0) {
      s_seq = seq;
      s_tile = tile;
    }
  }
  __syncthreads();
  const int seq = s_seq;
  if (seq < 0) return;
  const int q0 = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q0;
  const int k_len = a.cu_k[seq + 1] - a.cu_k[seq];
  const int m0 = s_tile * kTalkTileRows + (PAIR ? blockIdx.z * BQ : 0), rows = min(BQ, q_len - m0);
  if (rows <= 0) return;
  const int pos0 = k_len - q_len + m0;                 // position of row 0
  const int klo = a.window > 0 ? max(0, pos0 - a.window + 1) : 0;
  const int khi = pos0 + rows;                         // one past the last visible key
  const int ntiles = (khi - klo + BK - 1) / BK;

  const int strQ = dk + 8, strK = G * dk + 8, strV = G * dvc + 8;      // elements; odd multiples of 16 bytes
  const uint32_t sQ = smem_u32(smem);
  const uint32_t sS = sQ + (q_smem ? H * BQ * strQ * 2 : 0);
  const uint32_t s_bytes = H * kPlane * 4;         // one of two score buffers
  const uint32_t sK = sS + (two_scores ? 2 : 1) * s_bytes;
  const uint32_t sV = sK + BK * strK * 2;
  const uint32_t sB = sV + BK * strV * 2;              // two bias tiles [H][kBiasRow] (MODE > 0)
  const float* bias0 = reinterpret_cast<const float*>(smem + (sB - sQ));
  float* S0 = reinterpret_cast<float*>(smem + (sS - sQ));

  // ---- loads ----
  auto pool_row = [&](int j) -> int64_t {
    const int blk = a.bs_log2 >= 0 ? j >> a.bs_log2 : j / a.bs;
    const int id = blk < a.bt_stride ? __ldg(a.bt + static_cast<int64_t>(seq) * a.bt_stride + blk) : -1;
    if (id < 0 || id >= a.num_blocks) {
      report(a.status, B200_ERR_BOUNDS);
      return -1;
    }
    return static_cast<int64_t>(id) * a.bs + (j - blk * a.bs);
  };
  // row of the pool this thread's key row of tile t has, -1: none
  const int my_row = tid / kTpr, my_chunk = tid % kTpr;
  auto tile_row = [&](int t) -> int64_t {
    const int j = klo + t * BK + my_row;
    return j < khi ? pool_row(j) : -1;
  };
  // 32 rows x G heads x width columns (from column d0 of d) of the pool; kTpr threads per row
  auto load_rows = [&](int64_t row, const void* cache, int d, int d0, int width, uint32_t dst, int stride) {
    const int cpw = width / 8, total = G * cpw;
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(cache) + (row < 0 ? 0 : row) * G * d + d0;
    const int bytes = row >= 0 ? 16 : 0;
    dst += my_row * stride * 2;
    if (width == d) {
#pragma unroll 4
      for (int c = my_chunk; c < total; c += kTpr) cp_async16(dst + c * 16, src + c * 8, bytes);
    } else {
      for (int c = my_chunk; c < total; c += kTpr) {
        const int hd = c / cpw, cc = c - hd * cpw;
        cp_async16(dst + c * 16, src + hd * d + cc * 8, bytes);
      }
    }
  };
  // biases of tile t: entry i of a head is the distance of row 0 to the tile's last key, plus i
  auto load_bias = [&](int t) {
    if constexpr (MODE > 0) {
      const int dmin = pos0 - (klo + t * BK + BK - 1);
      const uint32_t dst = sB + (t & 1) * (H * kBiasRow * 4);
      for (int i = tid; i < H * 48; i += kThreads) {
        const int h = i / 48, k = i - h * 48, dist = min(max(dmin + k, 0), a.bias_len - 1);
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(dst + (h * kBiasRow + k) * 4),
                     "l"(a.bias_table + h * a.bias_len + dist) : "memory");
      }
    }
  };
  const __nv_bfloat16* qrow = static_cast<const __nv_bfloat16*>(a.q) + static_cast<int64_t>(q0 + m0) * a.q_stride;
  if (q_smem) {
    const int cpr = dk / 8, per_row = H * cpr;
    for (int i = tid; i < BQ * per_row; i += kThreads) {
      const int r = i / per_row, c = i - r * per_row, h = c / cpr, cc = c - h * cpr;
      const __nv_bfloat16* src = qrow + static_cast<int64_t>(r < rows ? r : 0) * a.q_stride + h * dk + cc * 8;
      cp_async16(sQ + ((h * BQ + r) * strQ + cc * 8) * 2, src, r < rows ? 16 : 0);
    }
  }
  int64_t next_row = tile_row(0);
  load_rows(next_row, a.kc, dk, 0, dk, sK, strK);
  cp_async_commit();
  load_rows(next_row, a.vc, a.dv, dv0, dvc, sV, strV);
  load_bias(0);
  load_bias(1);
  cp_async_commit();
  for (int i = tid; i < HP * BQ; i += kThreads) {
    s_ref[i] = i % HP < H ? kNoRef : INFINITY;
    s_cor[0][i] = s_cor[1][i] = 1.f;
  }
  if (tid < 2) s_flag[tid] = 0;
  if (kHalfRow && tid < BQ) s_up[tid] = 0;
  if constexpr (MODE == 3)
    for (int i = tid; i < HP * HP / 2; i += kThreads) s_talk[i / (HP / 2) * kTalkRow + i % (HP / 2)] = mp.tb[i];

  float o[HPW][2 * MAXC][4], l[HPW][2];
#pragma unroll
  for (int hh = 0; hh < HPW; ++hh) {
    l[hh][0] = l[hh][1] = 0.f;
#pragma unroll
    for (int c = 0; c < 2 * MAXC; ++c) o[hh][c][0] = o[hh][c][1] = o[hh][c][2] = o[hh][c][3] = 0.f;
  }
  // shared-memory addresses of this warp's fragments; kv: the key head of each of its heads
  const int ar = (lane & 7) + ((lane >> 3) & 1) * 8, ac = lane >> 4;
  const int br = (lane & 7) + (lane >> 4) * 8, bc = (lane >> 3) & 1;
  int kv[HPW];
#pragma unroll
  for (int hh = 0; hh < HPW; ++hh) kv[hh] = min(PAIR ? 2 * warp : warp * HPW + hh, H - 1) / Gs;
  // row of a lane's fragment: ar of one head, or with PAIR row (lane & 7) of head 2 warp + bc
  const uint32_t adQ = sQ + ((PAIR ? (2 * warp + bc) * BQ + (lane & 7) : warp * HPW * BQ + ar) * strQ + ac * 8) * 2, stepQ = BQ * strQ * 2;     // per head
  const uint32_t adK = sK + (br * strK + bc * 8) * 2, adV = sV + (ar * strV + ac * 8) * 2;
  const uint32_t adP = sS + (PAIR ? (2 * warp + bc) * kPlane + (lane & 7) * kSRow : warp * HPW * kPlane + ar * kSRow) * 4 + ac * 16;
  const float kx = a.cap > 0.f ? 2.f * kLog2e * a.scale / a.cap : 0.f;
  const float cap = a.cap, two_cap = 2.f * a.cap;
  cp_async_wait<1>();
  __syncthreads();

  const float cap_l2 = cap * kLog2e, two_cap_l2 = two_cap * kLog2e;
  // The mix of one tile on tensor cores: warp = query row, [32 keys x in-heads] x [in-heads x out-heads].  The capped
  // scores are split into three bf16 parts whose sum is the fp32 value and the matrix is exact in bf16, so that every
  // product is exact and the sums are fp32.
  auto mix_mma = [&](float* S, int t) {
    constexpr int KS = HP / 16, NT = HP / 8, NM = kHalfRow ? 1 : 2;      // NM: row tiles of 16 keys per warp
    const int mt0 = kHalfRow ? warp / BQ : 0;
#pragma unroll 1
    for (int r = kHalfRow ? warp % BQ : warp; r < rows; r += NW) {
      float c[NM][NT][4];
#pragma unroll
      for (int mt = 0; mt < NM; ++mt) {
#pragma unroll
        for (int n = 0; n < NT; ++n) c[mt][n][0] = c[mt][n][1] = c[mt][n][2] = c[mt][n][3] = 0.f;
        const int key = (mt0 + mt) * 16 + g, dist = pos0 + r - (klo + t * BK + key);        // keys g and g + 8 of the row tile
        const bool seen0 = dist >= 0 && dist < a.window, seen1 = dist >= 8 && dist - 8 < a.window;
        const float* Sr = S + r * kSRow + key;
        const float* Br = bias0 + (t & 1) * (H * kBiasRow) + r + BK - 1 - key;
#pragma unroll
        for (int kk = 0; kk < KS; ++kk) {
          uint32_t part[3][4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {          // fragment register e: keys g + 8 (e & 1), in-heads 2 tq + 8 (e >> 1)
            float x[2];
#pragma unroll
            for (int j = 0; j < 2; ++j) {
              const int h = min(kk * 16 + (e >> 1) * 8 + tq * 2 + j, H - 1);        // padding meets zeros of the matrix
              const float bias = Br[h * kBiasRow - (e & 1) * 8];
              x[j] = fmaf(-kLog2e, bias, cap_l2) - two_cap_l2 * rcp_approx(1.f + fast_exp2(Sr[h * kPlane + (e & 1) * 8] * kx));
            }
#pragma unroll
            for (int q = 0; q < 3; ++q) {
              part[q][e] = pack_bf16x2(x[0], x[1]);
              if (q < 2) {
                x[0] -= __uint_as_float(part[q][e] << 16);
                x[1] -= __uint_as_float(part[q][e] & 0xffff0000u);
              }
            }
          }
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            const uint32_t* tp = s_talk + (n * 8 + g) * kTalkRow + kk * 8 + tq;
            const uint32_t bf[2] = {tp[0], tp[4]};
#pragma unroll
            for (int q = 0; q < 3; ++q) mma_bf16_16816(c[mt][n], part[q], bf);
          }
        }
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          c[mt][n][0] = seen0 ? c[mt][n][0] : -INFINITY;
          c[mt][n][1] = seen0 ? c[mt][n][1] : -INFINITY;
          c[mt][n][2] = seen1 ? c[mt][n][2] : -INFINITY;
          c[mt][n][3] = seen1 ? c[mt][n][3] : -INFINITY;
        }
      }
      float2* refp = reinterpret_cast<float2*>(s_ref + r * HP + tq * 2);
      float top = -INFINITY;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const float2 ref = refp[n * 4];
#pragma unroll
        for (int mt = 0; mt < NM; ++mt)
          top = fmaxf(top, fmaxf(fmaxf(c[mt][n][0], c[mt][n][2]) - ref.x, fmaxf(c[mt][n][1], c[mt][n][3]) - ref.y));
      }
      bool up = __any_sync(0xffffffffu, top > kSlack);
      if constexpr (kHalfRow) {          // both halves of a row use one reference; after this both have read their scores
        if (up && lane == 0) s_up[r] = 1;
        pair_barrier(r);
        up = s_up[r] != 0;
      }
      if (up) {                          // some head of this row needs a new reference
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            float mx = fmaxf(c[0][n][j], c[0][n][j + 2]);
            if constexpr (NM == 2) mx = fmaxf(mx, fmaxf(c[NM - 1][n][j], c[NM - 1][n][j + 2]));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
            const int at = r * HP + n * 8 + tq * 2 + j;
            if constexpr (kHalfRow) {
              if (g == 0) s_top[mt0 * BQ * HP + at] = mx;
            } else if (g == 0 && mx > s_ref[at] + kSlack) {
              s_cor[t & 1][at] = fast_exp2(s_ref[at] - mx);
              s_ref[at] = mx;
              s_flag[t & 1] = 1;
            }
          }
        if constexpr (kHalfRow) {
          pair_barrier(r);
          if (mt0 == 0 && lane < HP) {
            const int at = r * HP + lane;
            const float mx = fmaxf(s_top[at], s_top[BQ * HP + at]);
            if (mx > s_ref[at] + kSlack) {
              s_cor[t & 1][at] = fast_exp2(s_ref[at] - mx);
              s_ref[at] = mx;
              s_flag[t & 1] = 1;
            }
          }
          pair_barrier(r);
        }
      }
      __syncwarp();                              // references are set, every lane has read its scores of the row
      __nv_bfloat16* Pr = reinterpret_cast<__nv_bfloat16*>(S + r * kSRow) + g;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const float2 ref = refp[n * 4];
        __nv_bfloat16* Ph = Pr + (n * 8 + tq * 2) * (kPlane * 2);
#pragma unroll
        for (int mt = 0; mt < NM; ++mt)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (HP == H || n * 8 + tq * 2 + (e & 1) < H)
              Ph[(e & 1) * (kPlane * 2) + (mt0 + mt) * 16 + (e >> 1) * 8] =
                  __float2bfloat16_rn(fast_exp2(c[mt][n][e] - (e & 1 ? ref.y : ref.x)));
      }
    }
  };
  // scores of the K tile in shared memory -> S
  auto qk = [&](float* S) {
#pragma unroll
      for (int h0 = 0; h0 < HPW; h0 += 2) {            // two heads at a time share the key fragments of their group
        constexpr int HS = HPW < 2 ? 1 : 2;
        float s[HS][4][4];
#pragma unroll
        for (int hh = 0; hh < HS; ++hh)
#pragma unroll
          for (int n = 0; n < 4; ++n) s[hh][n][0] = s[hh][n][1] = s[hh][n][2] = s[hh][n][3] = 0.f;
        const int hbase = PAIR ? 2 * warp : warp * HPW + h0;
        if (hbase < H) {
#pragma unroll 4
          for (int ks = 0; ks < dk / 16; ++ks) {
            uint32_t b0[4], b1[4];
#pragma unroll
            for (int hh = 0; hh < HS; ++hh) {
              const int h = hbase + hh;
              if (h < H) {
                if (hh == 0 || kv[h0 + hh] != kv[h0]) {
                  const uint32_t at = adK + kv[h0 + hh] * dk * 2 + ks * 32;
                  ldmatrix_x4(b0, at);
                  ldmatrix_x4(b1, at + 32 * strK);
                }
                uint32_t af[4];
                if (q_smem) {
                  ldmatrix_x4(af, adQ + (h0 + hh) * stepQ + ks * 32);
                } else {             // rows past the portion repeat its last row: their scores are never used
                  const __nv_bfloat16* q0p = qrow + static_cast<int64_t>(min(g, rows - 1)) * a.q_stride + h * dk + ks * 16 + tq * 2;
                  const __nv_bfloat16* q1p = qrow + static_cast<int64_t>(min(PAIR ? g : g + 8, rows - 1)) * a.q_stride + (PAIR ? h + 1 : h) * dk + ks * 16 + tq * 2;
                  af[0] = __ldg(reinterpret_cast<const uint32_t*>(q0p));
                  af[1] = __ldg(reinterpret_cast<const uint32_t*>(q1p));
                  af[2] = __ldg(reinterpret_cast<const uint32_t*>(q0p + 8));
                  af[3] = __ldg(reinterpret_cast<const uint32_t*>(q1p + 8));
                }
                const uint32_t f0[2] = {b0[0], b0[1]}, f1[2] = {b0[2], b0[3]}, f2[2] = {b1[0], b1[1]},
                               f3[2] = {b1[2], b1[3]};
                mma_bf16_16816(s[hh][0], af, f0);
                mma_bf16_16816(s[hh][1], af, f1);
                mma_bf16_16816(s[hh][2], af, f2);
                mma_bf16_16816(s[hh][3], af, f3);
              }
            }
          }
#pragma unroll
          for (int hh = 0; hh < HS; ++hh) {
            const int h = hbase + hh;
            if (h < H) {
              float* row = S + h * kPlane + g * kSRow + tq * 2;
#pragma unroll
              for (int n = 0; n < 4; ++n) {
                *reinterpret_cast<float2*>(row + n * 8) = make_float2(s[hh][n][0], s[hh][n][1]);
                *reinterpret_cast<float2*>(row + (PAIR ? kPlane : 8 * kSRow) + n * 8) = make_float2(s[hh][n][2], s[hh][n][3]);
              }
            }
          }
        }
      }
  };
  qk(S0);
  cp_async_wait<0>();
  __syncthreads();
  if (ntiles > 1) {
    next_row = tile_row(1);
    load_rows(next_row, a.kc, dk, 0, dk, sK, strK);
  }
  cp_async_commit();

  bool dirty = false;
  for (int t = 0; t < ntiles; ++t) {
    const int buf = two_scores ? t & 1 : 0;
    float* S = S0 + buf * (H * kPlane);
    // ---- mix ----
    if constexpr (MODE == 3) mix_mma(S, t);
    else
#pragma unroll 1
    for (int r = warp; r < rows; r += NW) {
      const int dist = pos0 + r - (klo + t * BK + lane);
      const bool seen = dist >= 0 && (a.window <= 0 || dist < a.window);
      const int dc = seen ? dist : 0;      // MODE 0
      float* Sr = S + r * kSRow + lane;
      const float* Br = bias0 + (t & 1) * (H * kBiasRow) + r + BK - 1 - lane;
      float s[HP];
#pragma unroll
      for (int h = 0; h < HP; ++h) s[h] = h < H ? Sr[h * kPlane] : 0.f;
#pragma unroll
      for (int h = 0; h < HP; ++h) {
        if constexpr (MODE > 0) {
          const float bias = h < H ? Br[h * kBiasRow] : 0.f;
          s[h] = capped(s[h], kx, cap, two_cap, bias);    // a padding head is finite and meets zeros of the mix
        } else {
          const float bias = a.bias_len > 0 ? __ldg(a.bias_table + min(h, H - 1) * a.bias_len + dc)
                                            : mp.r1[h] * logf(1.f + mp.r2[h] * static_cast<float>(dc));
          s[h] = cap > 0.f ? capped(s[h], kx, cap, two_cap, bias) : s[h] * a.scale - bias;
        }
      }
      __nv_bfloat16* Pr = reinterpret_cast<__nv_bfloat16*>(S + r * kSRow) + lane;
      const float base = seen ? 0.f : -INFINITY;
      __syncwarp();                            // every lane has read its scores of the row
      // eight mixed heads at a time: few registers stay live beside the accumulators
#pragma unroll
      for (int hb = 0; hb < HP; hb += 8) {
        float m[8], top = -INFINITY;
#pragma unroll
        for (int i = 0; i < 8; ++i) m[i] = base;
#pragma unroll
        for (int k = 0; k < HP; ++k)
#pragma unroll
          for (int i = 0; i < 8; ++i) m[i] = fmaf(mp.t[(hb + i) * HP + k], s[k], m[i]);
        float4* ref4 = reinterpret_cast<float4*>(s_ref + r * HP + hb);
        float4 ra = ref4[0], rb = ref4[1];
        // a row without a reference yet holds the largest negative float; padding heads hold +inf and stay out
        top = fmaxf(fmaxf(fmaxf(m[0] - ra.x, m[1] - ra.y), fmaxf(m[2] - ra.z, m[3] - ra.w)),
                    fmaxf(fmaxf(m[4] - rb.x, m[5] - rb.y), fmaxf(m[6] - rb.z, m[7] - rb.w)));
        if (__any_sync(0xffffffffu, top > kSlack)) {     // some head of this row needs a new reference
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const float mx = warp_max(m[i]);
            if (lane == 0) {
              const float ref = s_ref[r * HP + hb + i];
              if (mx > ref + kSlack) {
                s_ref[r * HP + hb + i] = mx;
                s_cor[t & 1][r * HP + hb + i] = fast_exp2(ref - mx);
                s_flag[t & 1] = 1;
              }
            }
          }
          __syncwarp();
          ra = ref4[0], rb = ref4[1];
        }
        const float ref[8] = {ra.x, ra.y, ra.z, ra.w, rb.x, rb.y, rb.z, rb.w};
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (hb + i < H) Pr[(hb + i) * kPlane * 2] = __float2bfloat16_rn(fast_exp2(m[i] - ref[i]));
      }
    }
    cp_async_wait<0>();
    __syncthreads();

    // ---- PV of this tile, QK of the next ----
    {
      const uint32_t pt = adP + buf * s_bytes;
      const bool rescale = s_flag[t & 1] != 0;
      // the other parity's flag and factors were last read one tile ago: ready them for the next one
      if (tid == 0) s_flag[(t + 1) & 1] = 0;
      if (kHalfRow && tid < BQ) s_up[tid] = 0;
      if (dirty)
        for (int i = tid; i < HP * BQ; i += kThreads) s_cor[(t + 1) & 1][i] = 1.f;
      dirty = rescale;
      uint32_t pf[HPW][2][4];
#pragma unroll
      for (int hh = 0; hh < HPW; ++hh) {
        const int h = PAIR ? 2 * warp : warp * HPW + hh;
        if (h < H) {
          if (rescale) {
            const float c0 = s_cor[t & 1][g * HP + h], c1 = s_cor[t & 1][PAIR ? g * HP + h + 1 : (g + 8) * HP + h];
            l[hh][0] *= c0;
            l[hh][1] *= c1;
#pragma unroll
            for (int c = 0; c < 2 * MAXC; ++c) {
              o[hh][c][0] *= c0;
              o[hh][c][1] *= c0;
              o[hh][c][2] *= c1;
              o[hh][c][3] *= c1;
            }
          }
#pragma unroll
          for (int kk = 0; kk < 2; ++kk) {
            ldmatrix_x4(pf[hh][kk], pt + hh * (kPlane * 4) + kk * 32);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 p = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&pf[hh][kk][e]));
              l[hh][e & 1] += p.x + p.y;
            }
          }
        }
      }
#pragma unroll
      for (int kk = 0; kk < 2; ++kk) {
#pragma unroll
        for (int c = 0; c < MAXC; ++c) {
          if (c < nc) {
            uint32_t bf[4];
#pragma unroll
            for (int hh = 0; hh < HPW; ++hh) {
              const int h = PAIR ? 2 * warp : warp * HPW + hh;
              if (h < H) {
                if (hh == 0 || kv[hh] != kv[hh - 1])
                  ldmatrix_x4_trans(bf, adV + kv[hh] * dvc * 2 + kk * 32 * strV + c * 32);
                const uint32_t b0[2] = {bf[0], bf[1]}, b1[2] = {bf[2], bf[3]};
                mma_bf16_16816(o[hh][2 * c], pf[hh][kk], b0);
                mma_bf16_16816(o[hh][2 * c + 1], pf[hh][kk], b1);
              }
            }
          }
        }
      }
    }
    if (!two_scores) __syncthreads();        // the weights are read, their buffer takes the next scores
    if (t + 1 < ntiles) qk(S0 + (two_scores ? (t + 1) & 1 : 0) * (H * kPlane));
    __syncthreads();
    if (t + 1 < ntiles) load_rows(next_row, a.vc, a.dv, dv0, dvc, sV, strV);
    if (t + 2 < ntiles) {
      next_row = tile_row(t + 2);
      load_rows(next_row, a.kc, dk, 0, dk, sK, strK);
      load_bias(t + 2);
    }
    cp_async_commit();
  }

  // ---- normalise, gate, store ----
#pragma unroll
  for (int hh = 0; hh < HPW; ++hh) {
    const int h0 = PAIR ? 2 * warp : warp * HPW + hh;
    if (h0 >= H) continue;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = PAIR ? h0 + e : h0;
      float sum = l[hh][e];
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      const int r = PAIR ? g : g + e * 8;
      if (r >= rows) continue;
      const float inv = sum > 0.f ? 1.f / sum : 0.f;
      const int64_t row = q0 + m0 + r;
      __nv_bfloat16* op = static_cast<__nv_bfloat16*>(a.out) + (row * H + h) * a.dv + dv0 + tq * 2;
      const __nv_bfloat16* gp =
          a.gate ? static_cast<const __nv_bfloat16*>(a.gate) + row * a.gate_stride + h * a.dv + dv0 + tq * 2 : nullptr;
#pragma unroll
      for (int c = 0; c < 2 * MAXC; ++c) {
        if (c < 2 * nc) {
          float x = o[hh][c][e * 2] * inv, y = o[hh][c][e * 2 + 1] * inv;
          if (gp) {
            const float2 gv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gp + c * 8));
            x = x / (1.f + __expf(-gv.x));
            y = y / (1.f + __expf(-gv.y));
          }
          *reinterpret_cast<uint32_t*>(op + c * 8) = pack_bf16x2(x, y);
        }
      }
    }
  }
}

// upper half of a float: its bf16 value if it is exact
inline uint32_t bf16_bits(float x) {
  uint32_t u;
  memcpy(&u, &x, 4);
  return u >> 16;
}
inline bool exact_in_bf16(const float* x, int n) {
  for (int i = 0; i < n; ++i) {
    uint32_t u;
    memcpy(&u, x + i, 4);
    if (u & 0xffffu) return false;
  }
  return true;
}

template <int HP, int NW, int MAXC, int MINB, int MODE, bool PAIR = false>
int launch_prefill(const TalkArgs& a, int chunks, size_t smem, int layout, cudaStream_t s) {
  MixParam<HP> mp;
  memset(&mp, 0, sizeof(mp));
  for (int h = 0; h < a.H; ++h)
    for (int k = 0; k < a.H; ++k) mp.t[h * HP + k] = a.talk_host[h * a.H + k] * kLog2e;
  for (int h = 0; h < a.H; ++h) {
    mp.r1[h] = a.r1_host[h];
    mp.r2[h] = a.r2_host[h];
  }
  for (int i = 0; i < HP * HP / 2; ++i) {
    const int h = i / (HP / 2), k = i % (HP / 2) * 2;
    if (h < a.H)
      mp.tb[i] = (k < a.H ? bf16_bits(a.talk_host[h * a.H + k]) : 0u) |
                 (k + 1 < a.H ? bf16_bits(a.talk_host[h * a.H + k + 1]) << 16 : 0u);
  }
  auto kern = talking_prefill_kernel<HP, NW, MAXC, MINB, MODE, PAIR>;
  static size_t configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64 || configured[dev] < smem) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
      return B200_ERR_LAUNCH;
    if (dev >= 0 && dev < 64) configured[dev] = smem;
  }
  const int64_t tiles = a.plan ? a.plan_capacity : a.rows / kTalkTileRows + a.n;          // sum over sequences of ceil(q_len / 16) is at most this
  kern<<<dim3(static_cast<unsigned>(tiles), chunks, PAIR ? 2 : 1), NW * 32, smem, s>>>(a, mp, layout);
  return launch_result();
}

template <int HP, int NW, int MAXC, int MINB>
int launch_prefill(const TalkArgs& a, int chunks, size_t smem, int layout, cudaStream_t s) {
  if (a.cap > 0.f && a.window > 0 && a.bias_len >= a.window) {
    if constexpr (HP >= 16) {
      if (exact_in_bf16(a.talk_host, a.H * a.H))
        return launch_prefill<HP, NW, MAXC, MINB, 3>(a, chunks, smem, layout, s);
    } else if (a.H == HP) {
      return launch_prefill<HP, NW, MAXC, MINB, 2>(a, chunks, smem, layout, s);
    }
    return launch_prefill<HP, NW, MAXC, MINB, 1>(a, chunks, smem, layout, s);
  }
  return launch_prefill<HP, NW, MAXC, MINB, 0>(a, chunks, smem, layout, s);
}

}  // namespace

int talking_prefill_mma_launch(const TalkArgs& a, cudaStream_t s) {
  if (!a.talk_host || !a.r1_host || !a.r2_host || !a.cu_q || a.H > 32 || a.dk % 16 || a.dv % 16 || a.dk > 256)
    return B200_ERR_UNSUPPORTED;
  if (a.q_stride % 8 || (a.gate && a.gate_stride % 2) || !aligned16(a.q) || !aligned16(a.kc) || !aligned16(a.vc) ||
      !aligned16(a.out) || (reinterpret_cast<uintptr_t>(a.gate) & 3))
    return B200_ERR_UNSUPPORTED;
  // value columns per CTA: what the accumulators of a warp's heads hold, and what shared memory leaves room for
  const int max_c = a.H <= 8 ? 16 : a.H <= 16 ? 8 : 4;     // units of 16 columns
  auto smem_of = [&](int rows, int dvc, int layout) {
    const size_t kv = size_t(BK) * (a.Hkv * a.dk + 8) * 2 + size_t(BK) * (a.Hkv * dvc + 8) * 2 +
                      2 * size_t(a.H) * kBiasRow * 4;      // keys, values, biases
    return kv + (layout & kTwoScores ? 2 : 1) * size_t(a.H) * plane_floats(rows) * 4 +
           (layout & kQueryInSmem ? size_t(a.H) * rows * (a.dk + 8) * 2 : 0);
  };
  const bool tensor_mix = a.cap > 0.f && a.window > 0 && a.bias_len >= a.window && exact_in_bf16(a.talk_host, a.H * a.H);
  if (tensor_mix && a.H > 16 && (a.H / a.Hkv) % 2 == 0 && a.dv <= 128) {     // many heads: pairs of heads on eight queries
    for (int l : {kQueryInSmem | kTwoScores, +kTwoScores, +kQueryInSmem, 0}) {
      const size_t smem = smem_of(kTalkTileRows / 2, a.dv, l);
      if (smem <= 212 * 1024) return launch_prefill<32, 16, 8, 1, 3, true>(a, 1, smem, l, s);
    }
  }
  for (int chunks = 1; chunks <= a.dv / 16; ++chunks) {
    if (a.dv % (16 * chunks)) continue;
    const int dvc = a.dv / chunks;
    if (dvc / 16 > max_c) continue;
    size_t smem = 0;
    int layout = -1;
    for (int l : {kQueryInSmem | kTwoScores, +kTwoScores, +kQueryInSmem, 0}) {
      smem = smem_of(kTalkTileRows, dvc, l);
      if (smem <= 216 * 1024) {
        layout = l;
        break;
      }
    }
    if (layout < 0) continue;
    const bool two = smem <= 108 * 1024 && dvc / 16 <= 8;             // two CTAs per SM: half the registers each
    if (a.H <= 8) return two ? launch_prefill<8, 8, 8, 2>(a, chunks, smem, layout, s)
                             : launch_prefill<8, 8, 16, 1>(a, chunks, smem, layout, s);
    if (a.H <= 16) return dvc <= 64 ? launch_prefill<16, 16, 4, 1>(a, chunks, smem, layout, s)
                                    : launch_prefill<16, 16, 8, 1>(a, chunks, smem, layout, s);
    return launch_prefill<32, 16, 4, 1>(a, chunks, smem, layout, s);
  }
  return B200_ERR_UNSUPPORTED;
}

}  // namespace b200
