// Gated delta rule of prompts and portions on tensor cores: sequences are cut into chunks of 64 tokens, and within a chunk
// the 64 dependent rank-one updates become one triangular solve.  With b_i the running sum of ln g inside the chunk,
// gamma_i = exp(b_i), S the state at the chunk's start and K, Q, V the chunk's rows (K, Q behind silu, not yet of unit
// length; rk_i, rq_i their reciprocal norms, rq_i with the factor dk^-1/2):
//
//   A_ij = beta_i rk_i rk_j exp(b_i - b_j) (k_i . k_j)   j < i          T = (I + A)^-1 diag(beta)
//   P_ij = rq_i rk_j exp(b_i - b_j) (q_i . k_j)          j <= i
//   U = T (V - diag(gamma rk) K S),   O = diag(gamma rq) Q S + P U,   S' = gamma_C S + K^T diag(rk gamma_C / gamma) U
//
// delta_prepare_kernel  T and P of every (chunk, value head), all in parallel
// delta_scan_kernel     one CTA per (sequence, value head) walks the chunks.  A warp owns 16 value columns of the state for
//                       the whole sequence: S^T [16, dk] stays in registers as accumulators, and because the accumulators
//                       of one product have the layout of the next product's A operand, S^T, U^T and O^T never leave the
//                       registers between the five products.  Norm and output gate follow in the same launch.
//
// Precision: everything behind the activations is fp32.  K, Q and V are bf16 as they come, so they are exact operands, and
// their norms are factors outside the products.  Every fp32 operand (S, U, T, P) is split into three bf16 parts that
// carry 24 bits together: products with one fp32 operand take three tensor-core products, those with two take the six
// that matter; sums are fp32.  Differences of b are taken in double precision.
#include <type_traits>

#include "delta_common.cuh"

namespace b200 {
namespace {

constexpr int C = 64;                          // tokens per chunk
constexpr int kPrepThreads = 128;
constexpr int kPlane = C * C;                  // elements of one part of T or P
constexpr size_t kBlobBytes = 6 * kPlane * 2 + 4 * C * 4;   // T parts, P parts, then four fp32 vectors per token

struct ChunkArgs {
  DeltaArgs d;
  uint8_t* blobs;                              // [chunks, H] x kBlobBytes
};

// x0, x1 -> three packed bf16 pairs whose sum is x to 24 bits
__device__ __forceinline__ void split3(float x0, float x1, uint32_t& h, uint32_t& m, uint32_t& l) {
  h = pack_bf16x2(x0, x1);
  x0 -= __uint_as_float(h << 16);
  x1 -= __uint_as_float(h & 0xffff0000u);
  m = pack_bf16x2(x0, x1);
  x0 -= __uint_as_float(m << 16);
  x1 -= __uint_as_float(m & 0xffff0000u);
  l = pack_bf16x2(x0, x1);
}

// A operand of k-step tiles t0, t1 (accumulator layout) in three parts
__device__ __forceinline__ void split_a(const float (&t0)[4], const float (&t1)[4], uint32_t (&h)[4], uint32_t (&m)[4],
                                        uint32_t (&l)[4]) {
  split3(t0[0], t0[1], h[0], m[0], l[0]);
  split3(t0[2], t0[3], h[1], m[1], l[1]);
  split3(t1[0], t1[1], h[2], m[2], l[2]);
  split3(t1[2], t1[3], h[3], m[3], l[3]);
}

template <int DK>
struct PrepSmem {
  static constexpr int ROW = DK + 8;           // padded row, elements
  static constexpr int LDA = C + 4;
  __nv_bfloat16 k[C * ROW], q[C * ROW];
  float a[C * LDA];
  double b[C];
  float rk[C], rq[C], beta[C];
};

template <int DK>
__global__ void __launch_bounds__(kPrepThreads) delta_prepare_kernel(const ChunkArgs args) {
  using Sm = PrepSmem<DK>;
  extern __shared__ __align__(16) uint8_t raw[];
  Sm& sm = *reinterpret_cast<Sm*>(raw);
  const DeltaArgs& a = args.d;
  const int head = blockIdx.y, kh = head / (a.H / a.G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int seq, index;
  if (!find_segment(a.cu_q, a.n, C, blockIdx.x, &seq, &index)) return;
  SeqInfo info;
  if (!sequence_info(a, seq, &info)) return;
  const int nt = min(C, info.len - index * C);
  const int64_t tok0 = info.tok0 + index * C;
  // ---- K and Q rows, zero beyond the chunk's tokens and beyond dk
  {
    constexpr int CPR = DK / 8;
    const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + tok0 * a.act_stride + kh * a.dk;
    const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + tok0 * a.act_stride + kh * a.dk;
    for (int i = tid; i < C * CPR; i += kPrepThreads) {
      const int r = i / CPR, c = i % CPR;
      const bool ok = r < nt && c * 8 < a.dk;
      const int64_t off = ok ? r * a.act_stride + c * 8 : 0;
      cp_async16(smem_u32(sm.k + r * Sm::ROW + c * 8), kp + off, ok ? 16 : 0);
      cp_async16(smem_u32(sm.q + r * Sm::ROW + c * 8), qp + off, ok ? 16 : 0);
    }
    cp_async_commit();
  }
  // ---- running sum of ln g (warp 0, two tokens per lane), write strengths
  if (warp == 0) {
    double g[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      float lg = 0.f, beta = 0.f;
      if (t < nt) {
        const int64_t row = (tok0 + t) * a.proj_stride + head;
        lg = log_decay(__bfloat162float(static_cast<const __nv_bfloat16*>(a.a)[row]) + a.dt_bias[head], a.a_log[head]);
        beta = sigmoid_f(__bfloat162float(static_cast<const __nv_bfloat16*>(a.b)[row]));
      }
      g[e] = lg;
      sm.beta[t] = beta;
    }
    double incl = g[0] + g[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double y = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += y;
    }
    sm.b[2 * lane] = incl - g[1];
    sm.b[2 * lane + 1] = incl;
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- reciprocal norms: two threads per row
  {
    const int r = tid >> 1;
    float kk = 0.f, qq = 0.f;
    for (int c = (tid & 1) * 8; c < DK; c += 16) {
      const uint4 kv = *reinterpret_cast<const uint4*>(sm.k + r * Sm::ROW + c);
      const uint4 qv = *reinterpret_cast<const uint4*>(sm.q + r * Sm::ROW + c);
      const __nv_bfloat162* k2 = reinterpret_cast<const __nv_bfloat162*>(&kv);
      const __nv_bfloat162* q2 = reinterpret_cast<const __nv_bfloat162*>(&qv);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 x = __bfloat1622float2(k2[e]), y = __bfloat1622float2(q2[e]);
        kk += x.x * x.x + x.y * x.y;
        qq += y.x * y.x + y.y * y.y;
      }
    }
    kk += __shfl_xor_sync(0xffffffffu, kk, 1);
    qq += __shfl_xor_sync(0xffffffffu, qq, 1);
    if ((tid & 1) == 0) {
      sm.rk[r] = rsqrtf(kk + 1e-6f);
      sm.rq[r] = rsqrtf(qq + 1e-6f) * rsqrtf(static_cast<float>(a.dk));
    }
  }
  __syncthreads();
  uint8_t* blob = args.blobs + (static_cast<size_t>(blockIdx.x) * a.H + head) * kBlobBytes;
  uint32_t* planes = reinterpret_cast<uint32_t*>(blob);
  // ---- K K^T and Q K^T of this warp's 16 rows, columns up to the diagonal
  {
    uint32_t kf[DK / 16][4], qf[DK / 16][4];
    const int r = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, chalf = lane >> 4;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      ldmatrix_x4(kf[ks], smem_u32(sm.k + r * Sm::ROW + ks * 16 + chalf * 8));
      ldmatrix_x4(qf[ks], smem_u32(sm.q + r * Sm::ROW + ks * 16 + chalf * 8));
    }
    const int g = lane >> 2, tq = lane & 3, r_in = (lane & 7) + (lane >> 4) * 8, bh = (lane >> 3) & 1;
    for (int p = 0; p <= warp; ++p) {            // 16 columns at a time
      float kk[2][4], qk[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) kk[n][e] = qk[n][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        uint32_t bf[4];
        ldmatrix_x4(bf, smem_u32(sm.k + (p * 16 + r_in) * Sm::ROW + ks * 16 + bh * 8));
        const uint32_t b0[2] = {bf[0], bf[1]}, b1[2] = {bf[2], bf[3]};
        mma_bf16_16816(kk[0], kf[ks], b0);
        mma_bf16_16816(kk[1], kf[ks], b1);
        mma_bf16_16816(qk[0], qf[ks], b0);
        mma_bf16_16816(qk[1], qf[ks], b1);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int i = warp * 16 + g + 8 * h, j = p * 16 + n * 8 + 2 * tq;
          float v[2], w[2];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float dec = j + e <= i ? expf(static_cast<float>(sm.b[i] - sm.b[j + e])) * sm.rk[j + e] : 0.f;
            v[e] = j + e < i ? sm.beta[i] * sm.rk[i] * dec * kk[n][2 * h + e] : 0.f;
            w[e] = sm.rq[i] * dec * qk[n][2 * h + e];
          }
          *reinterpret_cast<float2*>(sm.a + i * Sm::LDA + j) = make_float2(v[0], v[1]);
          uint32_t hi, mid, lo;
          split3(w[0], w[1], hi, mid, lo);
          const int at = (i * C + j) / 2;
          planes[3 * kPlane / 2 + at] = hi;
          planes[4 * kPlane / 2 + at] = mid;
          planes[5 * kPlane / 2 + at] = lo;
        }
    }
  }
  __syncthreads();
  // ---- (I + A)^-1, a column per thread by forward substitution; warp 1 starts at row 32
  if (tid < C) {
    const int j = tid;
    float x[C];
    const float beta = sm.beta[j];
    __nv_bfloat16* tp = reinterpret_cast<__nv_bfloat16*>(blob);
    auto rows = [&](auto lo_c) {
      constexpr int LO = decltype(lo_c)::value;
#pragma unroll
      for (int i = LO; i < C; ++i) {
        float s0 = i == j ? 1.f : 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
        for (int m = LO; m < i; m += 4) {
          const float4 r = *reinterpret_cast<const float4*>(sm.a + i * Sm::LDA + m);   // zero from the diagonal on
          s0 -= r.x * x[m];
          if (m + 1 < i) s1 -= r.y * x[m + 1];
          if (m + 2 < i) s2 -= r.z * x[m + 2];
          if (m + 3 < i) s3 -= r.w * x[m + 3];
        }
        x[i] = (s0 + s1) + (s2 + s3);
      }
#pragma unroll
      for (int i = LO; i < C; ++i) {
        const float v = x[i] * beta;
        const __nv_bfloat16 hi = __float2bfloat16_rn(v);
        const float r1 = v - __bfloat162float(hi);
        const __nv_bfloat16 mid = __float2bfloat16_rn(r1);
        tp[i * C + j] = hi;
        tp[kPlane + i * C + j] = mid;
        tp[2 * kPlane + i * C + j] = __float2bfloat16_rn(r1 - __bfloat162float(mid));
      }
    };
    if (warp == 0) rows(std::integral_constant<int, 0>{});
    else rows(std::integral_constant<int, 32>{});
  } else {
    // ---- factors per token: gamma rq, gamma rk, rk gamma_C / gamma; gamma_C
    const int t = tid - C;
    float* f = reinterpret_cast<float*>(blob + 6 * kPlane * 2);
    const float gamma = expf(static_cast<float>(sm.b[t]));
    f[t] = gamma * sm.rq[t];
    f[C + t] = gamma * sm.rk[t];
    f[2 * C + t] = sm.rk[t] * expf(static_cast<float>(sm.b[C - 1] - sm.b[t]));
    f[3 * C + t] = expf(static_cast<float>(sm.b[C - 1]));
  }
}

// Shared memory of one stage of the scan (elements of bf16, rows padded by 16 bytes)
template <int DK>
struct ScanLayout {
  static constexpr int ROWK = DK + 8, ROWP = C + 8;
  int rowv, k, q, v, p, f, bytes;      // byte offsets inside a stage
  __host__ __device__ explicit ScanLayout(int dv) {
    rowv = dv + 8;
    k = 0;
    q = k + C * ROWK * 2;
    v = q + C * ROWK * 2;
    p = v + C * rowv * 2;
    const int staged = C * (dv + 4) * 4;         // outputs are staged over K, Q and V
    if (p < staged) p = staged;
    f = p + 6 * C * ROWP * 2;
    bytes = f + 4 * C * 4;
  }
};

template <int DK>
__global__ void __launch_bounds__(256, 1) delta_scan_kernel(const ChunkArgs args) {
  using Lay = ScanLayout<DK>;
  constexpr int ROWK = Lay::ROWK, ROWP = Lay::ROWP, NK = DK / 8;
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ int s_first;
  const DeltaArgs& a = args.d;
  const int head = blockIdx.x, seq = blockIdx.y, kh = head / (a.H / a.G), dk = a.dk, dv = a.dv;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3, NT = blockDim.x;
  SeqInfo info;
  if (!sequence_info(a, seq, &info)) return;
  if (tid < 32) {
    const int first = first_segment(a.cu_q, C, seq);
    if (tid == 0) s_first = first;
  }
  __syncthreads();
  const Lay lay(dv);
  const int chunks = (info.len + C - 1) / C;
  const uint8_t* blob0 = args.blobs + (static_cast<size_t>(s_first) * a.H + head) * kBlobBytes;
  const uint32_t sbase = smem_u32(smem);

  auto fetch = [&](int j) {
    const uint32_t st = sbase + (j & 1) * lay.bytes;
    const int nt = min(C, info.len - j * C);
    const int64_t tok = info.tok0 + j * C;
    const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + tok * a.act_stride + kh * dk;
    const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + tok * a.act_stride + kh * dk;
    const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(a.v) + tok * a.act_stride + head * dv;
    for (int i = tid; i < C * (DK / 8); i += NT) {
      const int r = i / (DK / 8), c = i % (DK / 8);
      const bool ok = r < nt && c * 8 < dk;
      const int64_t off = ok ? r * a.act_stride + c * 8 : 0;
      cp_async16(st + lay.k + (r * ROWK + c * 8) * 2, kp + off, ok ? 16 : 0);
      cp_async16(st + lay.q + (r * ROWK + c * 8) * 2, qp + off, ok ? 16 : 0);
    }
    const int cv = dv / 8;
    for (int i = tid; i < C * cv; i += NT) {
      const int r = i / cv, c = i - r * cv;
      const bool ok = r < nt;
      cp_async16(st + lay.v + (r * lay.rowv + c * 8) * 2, vp + (ok ? r * a.act_stride + c * 8 : 0), ok ? 16 : 0);
    }
    const uint8_t* blob = blob0 + static_cast<size_t>(j) * a.H * kBlobBytes;
    for (int i = tid; i < 6 * C * (C / 8); i += NT) {
      const int r = i / (C / 8), c = i % (C / 8);       // r: row of one of the six parts
      // 16-column tiles above the diagonal are neither written nor read
      if (c / 2 <= (r % C) / 16) cp_async16(st + lay.p + (r * ROWP + c * 8) * 2, blob + (r * C + c * 8) * 2, 16);
    }
    for (int i = tid; i < C; i += NT) cp_async16(st + lay.f + i * 16, blob + 6 * kPlane * 2 + i * 16, 16);
    cp_async_commit();
  };

  // S^T: rows 16 warp + g (+ 8), columns 8 n + 2 tq (+ 1)
  float S[NK][4];
  float* pool = a.state + (info.slot * a.H + head) * static_cast<int64_t>(dk) * dv;
  const int vr = warp * 16 + g;
#pragma unroll
  for (int n = 0; n < NK; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = n * 8 + 2 * tq + (e & 1);
      S[n][e] = !info.fresh && d < dk ? pool[static_cast<int64_t>(d) * dv + vr + 8 * (e >> 1)] : 0.f;
    }

  fetch(0);
  const int r_in = (lane & 7) + (lane >> 4) * 8, bh = (lane >> 3) & 1;      // B operand, rows = n: (n lo, k lo) (n lo, k hi) (n hi, ...)
  const int t_in = (lane & 7) + ((lane >> 3) & 1) * 8, th = lane >> 4;      // B operand transposed, rows = k
  for (int j = 0; j < chunks; ++j) {
    cp_async_wait<0>();
    __syncthreads();                                   // chunk j has landed; everyone has left the other stage
    if (j + 1 < chunks) fetch(j + 1);
    uint8_t* stp = smem + (j & 1) * lay.bytes;
    const uint32_t st = sbase + (j & 1) * lay.bytes;
    const float* f = reinterpret_cast<const float*>(stp + lay.f);
    float D[8][4], O[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) D[n][e] = O[n][e] = 0.f;
    // ---- (K S)^T and (Q S)^T
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t h[4], m[4], l[4];
      split_a(S[2 * kk], S[2 * kk + 1], h, m, l);
#pragma unroll
      for (int np = 0; np < 4; np += 2) {
        uint32_t kf[2][4], qf[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          ldmatrix_x4(kf[u], st + lay.k + (((np + u) * 16 + r_in) * ROWK + kk * 16 + bh * 8) * 2);
          ldmatrix_x4(qf[u], st + lay.q + (((np + u) * 16 + r_in) * ROWK + kk * 16 + bh * 8) * 2);
        }
        auto part = [&](const uint32_t (&p)[4]) {        // eight accumulators between two uses of one
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const uint32_t k0[2] = {kf[u][0], kf[u][1]}, k1[2] = {kf[u][2], kf[u][3]};
            const uint32_t q0[2] = {qf[u][0], qf[u][1]}, q1[2] = {qf[u][2], qf[u][3]};
            mma_bf16_16816(D[2 * (np + u)], p, k0);
            mma_bf16_16816(D[2 * (np + u) + 1], p, k1);
            mma_bf16_16816(O[2 * (np + u)], p, q0);
            mma_bf16_16816(O[2 * (np + u) + 1], p, q1);
          }
        };
        part(l);
        part(m);
        part(h);
      }
    }
    // ---- D <- V^T - gamma rk D,  O <- gamma rq O
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      uint32_t vf[4];      // (tokens lo, columns lo) (tokens lo, columns hi) (tokens hi, ...)
      ldmatrix_x4_trans(vf, st + lay.v + ((np * 16 + (lane & 7) + (lane >> 4) * 8) * lay.rowv + warp * 16 + bh * 8) * 2);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int n = 2 * np + u;
        const float2 qs = *reinterpret_cast<const float2*>(f + n * 8 + 2 * tq);
        const float2 ks = *reinterpret_cast<const float2*>(f + C + n * 8 + 2 * tq);
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const uint32_t v = vf[2 * u + hh];
          D[n][2 * hh] = __uint_as_float(v << 16) - ks.x * D[n][2 * hh];
          D[n][2 * hh + 1] = __uint_as_float(v & 0xffff0000u) - ks.y * D[n][2 * hh + 1];
          O[n][2 * hh] *= qs.x;
          O[n][2 * hh + 1] *= qs.y;
        }
      }
    }
    // ---- U^T = D^T T^T, then O^T += U^T P^T: B rows are rows of T / P, lower triangle of 16-tiles
    float U[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) U[n][e] = 0.f;
    auto triangular = [&](const float (&in)[8][4], float (&acc)[8][4], int mat) {
      const uint32_t base = st + lay.p + mat * 3 * C * ROWP * 2;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t h[4], m[4], l[4];
        split_a(in[2 * kk], in[2 * kk + 1], h, m, l);
#pragma unroll
        for (int n0 = kk & ~1; n0 < 4; n0 += 2) {        // two tiles of 16 rows; the first may lie above the diagonal
          uint32_t b3[2][3][4];
#pragma unroll
          for (int u = 0; u < 2; ++u)
            if (n0 + u >= kk) {
              const uint32_t at = base + (((n0 + u) * 16 + r_in) * ROWP + kk * 16 + bh * 8) * 2;
#pragma unroll
              for (int p = 0; p < 3; ++p) ldmatrix_x4(b3[u][p], at + p * C * ROWP * 2);
            }
          auto part = [&](const uint32_t (&x)[4], int p) {
#pragma unroll
            for (int u = 0; u < 2; ++u)
              if (n0 + u >= kk) {
                const uint32_t b0[2] = {b3[u][p][0], b3[u][p][1]}, b1[2] = {b3[u][p][2], b3[u][p][3]};
                mma_bf16_16816(acc[2 * (n0 + u)], x, b0);
                mma_bf16_16816(acc[2 * (n0 + u) + 1], x, b1);
              }
          };
          part(l, 0);
          part(m, 1);
          part(h, 2);
          part(m, 0);
          part(h, 1);
          part(h, 0);
        }
      }
    };
    triangular(D, U, 0);
    triangular(U, O, 1);
    // ---- S^T = gamma_C S^T + (U rk gamma_C / gamma)^T K
    const float gc = f[3 * C];
#pragma unroll
    for (int n = 0; n < NK; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[n][e] *= gc;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const float2 cs = *reinterpret_cast<const float2*>(f + 2 * C + (2 * kk + u) * 8 + 2 * tq);
        U[2 * kk + u][0] *= cs.x;
        U[2 * kk + u][1] *= cs.y;
        U[2 * kk + u][2] *= cs.x;
        U[2 * kk + u][3] *= cs.y;
      }
      uint32_t h[4], m[4], l[4];
      split_a(U[2 * kk], U[2 * kk + 1], h, m, l);
#pragma unroll
      for (int c = 0; c < NK; c += 8) {
        uint32_t bf[4][4];
#pragma unroll
        for (int u = 0; u < 4; ++u)
          ldmatrix_x4_trans(bf[u], st + lay.k + ((kk * 16 + t_in) * ROWK + (c + 2 * u + th) * 8) * 2);
        auto part = [&](const uint32_t (&x)[4]) {
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            const uint32_t b0[2] = {bf[u][0], bf[u][1]}, b1[2] = {bf[u][2], bf[u][3]};
            mma_bf16_16816(S[c + 2 * u], x, b0);
            mma_bf16_16816(S[c + 2 * u + 1], x, b1);
          }
        };
        part(l);
        part(m);
        part(h);
      }
    }
    // ---- norm over the value columns, output gate
    // a warp takes the tokens warp, warp + NT / 32, ... in groups of eight; the gates of a group are loaded ahead
    const int nt = min(C, info.len - j * C), NW = NT / 32, c = lane * 4;
    const int64_t tok0 = info.tok0 + j * C;
    const __nv_bfloat16* gp = static_cast<const __nv_bfloat16*>(a.gate) + tok0 * a.proj_stride + head * dv + c;
    uint2 gate[8];
    auto load_gates = [&](int t0) {
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const int t = t0 + u * NW;
        gate[u] = c < dv && t < nt ? __ldg(reinterpret_cast<const uint2*>(gp + t * a.proj_stride)) : make_uint2(0u, 0u);
      }
    };
    load_gates(warp);
    __syncthreads();                                   // K, Q, V of this stage are done with
    float* so = reinterpret_cast<float*>(stp);
    const int ldo = dv + 4;
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) so[(n * 8 + 2 * tq + (e & 1)) * ldo + vr + 8 * (e >> 1)] = O[n][e];
    __syncthreads();
    float4 w = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < dv) w = make_float4(__ldg(a.norm_w + c), __ldg(a.norm_w + c + 1), __ldg(a.norm_w + c + 2), __ldg(a.norm_w + c + 3));
    for (int t0 = warp; t0 < nt; t0 += 8 * NW) {
      if (t0 != warp) load_gates(t0);
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const int t = t0 + u * NW;
        if (t >= nt) continue;                         // the same for the whole warp
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < dv) o = *reinterpret_cast<const float4*>(so + t * ldo + c);
        const float inv = rsqrtf(warp_sum(o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w) / static_cast<float>(dv) + a.eps);
        const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gate[u].x));
        const float2 g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gate[u].y));
        using bf16 = __nv_bfloat16;
        if (c < dv)
          *reinterpret_cast<uint2*>(static_cast<bf16*>(a.out) + ((tok0 + t) * a.H + head) * dv + c) =
              make_uint2(pack_bf16x2(o.x * inv * w.x * silu_for<bf16>(g0.x), o.y * inv * w.y * silu_for<bf16>(g0.y)),
                         pack_bf16x2(o.z * inv * w.z * silu_for<bf16>(g1.x), o.w * inv * w.w * silu_for<bf16>(g1.y)));
      }
    }
  }
#pragma unroll
  for (int n = 0; n < NK; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = n * 8 + 2 * tq + (e & 1);
      if (d < dk) pool[static_cast<int64_t>(d) * dv + vr + 8 * (e >> 1)] = S[n][e];
    }
}

inline int64_t chunk_count(int num_seqs, int64_t total_tokens) { return total_tokens / C + num_seqs; }

template <int DK>
int launch(const ChunkArgs& c, int64_t total_tokens, cudaStream_t s) {
  const size_t prep = sizeof(PrepSmem<DK>);
  const ScanLayout<DK> lay(c.d.dv);
  const size_t scan = 2 * static_cast<size_t>(lay.bytes);
  if (cudaFuncSetAttribute(delta_prepare_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(prep)) !=
          cudaSuccess ||
      cudaFuncSetAttribute(delta_scan_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(scan)) !=
          cudaSuccess)
    return B200_ERR_LAUNCH;
  delta_prepare_kernel<DK><<<dim3(static_cast<unsigned>(chunk_count(c.d.n, total_tokens)), c.d.H), kPrepThreads, prep, s>>>(c);
  delta_scan_kernel<DK><<<dim3(c.d.H, c.d.n), c.d.dv * 2, scan, s>>>(c);
  return launch_result();
}

}  // namespace

bool delta_chunk_shape(int dk, int dv) { return dk % 16 == 0 && dv % 16 == 0 && dk <= 128 && dv <= 128; }

size_t delta_chunk_workspace(int num_seqs, int64_t total_tokens, int H) {
  return static_cast<size_t>(chunk_count(num_seqs, total_tokens)) * H * kBlobBytes;
}

int delta_chunk_launch(const DeltaArgs& a, int64_t total_tokens, void* workspace, cudaStream_t s) {
  ChunkArgs c{a, static_cast<uint8_t*>(workspace)};
  return a.dk <= 64 ? launch<64>(c, total_tokens, s) : launch<128>(c, total_tokens, s);
}

}  // namespace b200
