// Talking-heads attention, bf16 tensor-core path for one query token per sequence (mathematics: talking_attention.cu).
//
// Bound by reading K and V once.  A CTA of four or eight warps owns one sequence, or one of `splits` equal shares of its
// visible keys, with all heads, and walks its keys in tiles of 32 through a ring of (K, V) tiles filled by cp.async:
//
//   QK    S^T[key, head] = K q^T per key head (the heads of a group are the N columns of mma.sync m16n8k16); soft
//         cap and distance bias on the accumulators, fp32 scores of all heads to shared memory
//   mix   lane = key, warp = every fourth (eighth) mixed head: the H x H mix, exponentials against a lazy reference
//         maximum (fp32, log2 domain; it moves only when a score exceeds it by 2^kSlack), bf16 weights to shared
//         memory; every lane keeps the sums of its own keys
//   PV    O^T[dv, head] += V^T P^T, fp32 accumulators in registers
//
// With more than one share the unnormalised partials (max, sum, O) are merged in fixed order by a second kernel, so
// the result does not depend on which CTA ran first.
#include "talking_attention.cuh"

namespace b200 {
namespace {

constexpr int BK = 32;
constexpr int kPRow = 40;             // bf16 per weight row: 32 keys + padding (odd multiple of 16 bytes)
constexpr int kSRow = 33;
constexpr int kMaxSplits = 32;
constexpr float kSlack = 30.f;         // log2 of how far a score may exceed the running reference
constexpr float kNoRef = -3.0e38f;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// cap tanh(x scale / cap) - bias; k = 2 log2(e) scale / cap
__device__ __forceinline__ float capped(float x, float k, float cap, float two_cap, float bias) {
  return (cap - bias) - two_cap * rcp_approx(1.f + fast_exp2(x * k));
}

struct DecodeParts {
  float* o;       // [n, splits, H, dv]
  float* ml;      // [n, splits, H, 2]
  int splits, stages;
};

__device__ __forceinline__ float gated(float o, const __nv_bfloat16* gp) {
  return gp ? o / (1.f + __expf(-__bfloat162float(*gp))) : o;
}

// HP: heads padded; NT: column tiles of 8 heads per key head; MAXU: row tiles of 16 value columns per warp
// NW: warps; COMMON: soft cap and bias table present
template <int HP, int NT, int MAXU, int NW, bool COMMON>
__global__ void __launch_bounds__(NW * 32, NW == 8 ? (NT * MAXU <= 4 ? 3 : NT * MAXU <= 8 ? 2 : 1) : 1)
talking_decode_kernel(const TalkArgs a, const DecodeParts parts) {
  constexpr int kWarps = NW, kThreads = NW * 32, kTpr = kThreads / BK;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float s_talk[HP * HP];     // talk * log2(e), zero-padded
  __shared__ float s_score[HP * kSRow];
  __shared__ __align__(16) __nv_bfloat16 s_p[(HP + 8 * NT) * kPRow];   // + rows that pad the last column tile
  __shared__ float s_cor[HP + 8 * NT], s_l[HP], s_m[HP];
  __shared__ int s_flag[2];             // tile parity: some head's reference moved
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int H = a.H, G = a.Hkv, Gs = H / G, dk = a.dk, dv = a.dv, seq = blockIdx.y;
  const int ctx = static_cast<int>(a.ctx_lens[seq]);
  if (ctx <= 0) return;
  const int klo = a.window > 0 ? max(0, ctx - a.window) : 0;
  const int tiles = (ctx - klo + BK - 1) / BK, per = (tiles + parts.splits - 1) / parts.splits;
  const int t0 = blockIdx.x * per, t1 = min(tiles, t0 + per);

  const int strQ = dk + 8, strK = G * dk + 8, strV = G * dv + 8;
  const uint32_t sQ = smem_u32(smem), sK = sQ + (H + 8 * NT) * strQ * 2;      // rows past the heads are padding
  const uint32_t stage_bytes = BK * (strK + strV) * 2;

  // which: 1 keys, 2 values, 3 both
  auto load_tile = [&](int t, int which) {
    const uint32_t kd = sK + (t - t0) % parts.stages * stage_bytes, vd = kd + BK * strK * 2;
    const int r = tid / kTpr, j = klo + t * BK + r;
    int64_t row = -1;
    if (j < ctx) {
      const int blk = a.bs_log2 >= 0 ? j >> a.bs_log2 : j / a.bs;
      const int id = blk < a.bt_stride ? __ldg(a.bt + static_cast<int64_t>(seq) * a.bt_stride + blk) : -1;
      if (id < 0 || id >= a.num_blocks) report(a.status, B200_ERR_BOUNDS);
      else row = static_cast<int64_t>(id) * a.bs + (j - blk * a.bs);
    }
    const int bytes = row >= 0 ? 16 : 0;
    const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.kc) + (row < 0 ? 0 : row) * G * dk;
    const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(a.vc) + (row < 0 ? 0 : row) * G * dv;
    if (which & 1)
      for (int c = tid % kTpr; c < G * dk / 8; c += kTpr) cp_async16(kd + (r * strK + c * 8) * 2, kp + c * 8, bytes);
    if (which & 2)
      for (int c = tid % kTpr; c < G * dv / 8; c += kTpr) cp_async16(vd + (r * strV + c * 8) * 2, vp + c * 8, bytes);
  };
  {
    const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + static_cast<int64_t>(seq) * a.q_stride;
    const int cpr = dk / 8;
    for (int i = tid; i < H * cpr; i += kThreads) {
      const int h = i / cpr, c = i - h * cpr;
      cp_async16(sQ + (h * strQ + c * 8) * 2, qp + h * dk + c * 8, 16);
    }
  }
  // one stage: the next keys arrive during mix and PV, the next values during QK and mix
  const bool single = parts.stages == 1;
  if (single) {
    if (t0 < t1) load_tile(t0, 1);
    cp_async_commit();
    if (t0 < t1) load_tile(t0, 2);
    cp_async_commit();
  }
  for (int i = 0; i < parts.stages - 1; ++i) {
    if (t0 + i < t1) load_tile(t0 + i, 3);
    cp_async_commit();
  }
  for (int i = tid; i < HP * HP; i += kThreads) {
    const int h = i / HP, k = i % HP;
    s_talk[i] = h < H && k < H ? a.talk[h * H + k] * kLog2e : 0.f;
  }
  for (int i = tid; i < HP * kSRow; i += kThreads) s_score[i] = 0.f;
  for (int i = tid; i < (HP + 8 * NT) * kPRow; i += kThreads) s_p[i] = __float2bfloat16_rn(0.f);
  if (tid < HP + 8 * NT) s_cor[tid] = 1.f;
  if (tid < 2) s_flag[tid] = 0;
  const float kx = a.cap > 0.f ? 2.f * kLog2e * a.scale / a.cap : 0.f;

  constexpr int HW = (HP + kWarps - 1) / kWarps;      // mixed heads per warp
  float m_run[HW], l_run[HW];
#pragma unroll
  for (int i = 0; i < HW; ++i) {
    m_run[i] = kNoRef;
    l_run[i] = 0.f;
  }
  float o[MAXU][NT][4];
#pragma unroll
  for (int u = 0; u < MAXU; ++u)
#pragma unroll
    for (int n = 0; n < NT; ++n) o[u][n][0] = o[u][n][1] = o[u][n][2] = o[u][n][3] = 0.f;
  const int mt_per_head = dv / 16, units = G * mt_per_head;
  // per row tile of this warp: byte offset of its value columns in a V row tile, of its heads' weights, first head
  uint32_t offV[MAXU], offP[MAXU];
  int head0[MAXU];
  {
    const int kr = (lane & 7) + (lane >> 4) * 8, vc = ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int u = 0; u < MAXU; ++u) {
      const int unit = warp + u * kWarps, c = unit / mt_per_head;
      offV[u] = (kr * strV + unit * 16 + vc) * 2;
      head0[u] = c * Gs;
      offP[u] = smem_u32(s_p) + ((c * Gs + (lane & 7)) * kPRow + ((lane >> 3) & 1) * 8) * 2;
    }
  }

  for (int t = t0; t < t1; ++t) {
    if (parts.stages == 2) cp_async_wait<0>();
    else cp_async_wait<1>();
    __syncthreads();
    if (!single) {
      if (t + parts.stages - 1 < t1) load_tile(t + parts.stages - 1, 3);
      cp_async_commit();
    }
    const uint32_t kt = sK + (t - t0) % parts.stages * stage_bytes, vt = kt + BK * strK * 2;
    const int j0 = klo + t * BK;

    // ---- QK, cap, bias ----
    for (int u = warp; u < 2 * G; u += kWarps) {
      const int mt = u & 1, c = u >> 1;
      // biases of the unit's 16 keys x Gs heads, requested ahead of the products
      constexpr int NB = 4 * NT;
      float bias[NB];
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        const int i = lane + b * 32;
        bias[b] = 0.f;
        if (i < 16 * Gs) {
          const int h = c * Gs + (i >> 4), dist = max(ctx - 1 - (j0 + mt * 16 + (i & 15)), 0);
          if (COMMON || a.bias_len > 0) bias[b] = __ldg(a.bias_table + h * a.bias_len + dist);
          else bias[b] = a.r1[h] * logf(1.f + a.r2[h] * static_cast<float>(dist));
        }
      }
      float s[NT][4];
#pragma unroll
      for (int n = 0; n < NT; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const uint32_t qa = sQ + ((c * Gs + (lane & 7)) * strQ + ((lane >> 3) & 1) * 8) * 2;
      const uint32_t ka = kt + ((mt * 16 + (lane & 15)) * strK + c * dk + (lane >> 4) * 8) * 2;
#pragma unroll 4
      for (int ks = 0; ks < dk / 16; ++ks) {
        uint32_t af[4];
        ldmatrix_x4(af, ka + ks * 32);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          uint32_t bf[2];
          ldmatrix_x2(bf, qa + n * 16 * strQ + ks * 32);
          mma_bf16_16816(s[n], af, bf);
        }
      }
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int hg = n * 8 + tq * 2 + (e & 1), key = mt * 16 + g + (e >> 1) * 8;
          if (hg < Gs) s_score[(c * Gs + hg) * kSRow + key] = s[n][e];
        }
      __syncwarp();
      // cap and bias of the unit's 16 keys x Gs heads, spread over all lanes
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        const int i = lane + b * 32;
        if (i < 16 * Gs) {
          float* sp = s_score + (c * Gs + (i >> 4)) * kSRow + mt * 16 + (i & 15);
          *sp = COMMON || a.cap > 0.f ? capped(*sp, kx, a.cap, 2.f * a.cap, bias[b]) : *sp * a.scale - bias[b];
        }
      }
    }
    __syncthreads();
    if (single) {
      if (t + 1 < t1) load_tile(t + 1, 1);
      cp_async_commit();
    }

    // ---- mix, weights ----
    {
      const float base = j0 + lane < ctx ? 0.f : -INFINITY;
      if (tid == 0) s_flag[(t + 1) & 1] = 0;      // read by the PV before this tile's first barrier
      float s[HP];
#pragma unroll
      for (int k = 0; k < HP; ++k) s[k] = s_score[k * kSRow + lane];
      float m[HW], top = -INFINITY;
#pragma unroll
      for (int i = 0; i < HW; ++i) {
        const float* w = s_talk + (warp + i * kWarps) * HP;
        m[i] = base;
#pragma unroll
        for (int k = 0; k < HP; k += 4) {
          const float4 x = *reinterpret_cast<const float4*>(w + k);
          m[i] = fmaf(x.x, s[k], m[i]);
          m[i] = fmaf(x.y, s[k + 1], m[i]);
          m[i] = fmaf(x.z, s[k + 2], m[i]);
          m[i] = fmaf(x.w, s[k + 3], m[i]);
        }
        if (warp + i * kWarps < H) top = fmaxf(top, m[i] - m_run[i]);
      }
      if (__any_sync(0xffffffffu, top > kSlack)) {
#pragma unroll
        for (int i = 0; i < HW; ++i) {
          const int h = warp + i * kWarps;
          const float mx = warp_max(m[i]);
          float cor = 1.f;
          if (mx > m_run[i] + kSlack && h < H) {
            cor = fast_exp2(m_run[i] - mx);        // no reference yet: 0
            m_run[i] = mx;
          }
          l_run[i] *= cor;
          if (lane == 0) s_cor[h] = cor;
        }
        if (lane == 0) s_flag[t & 1] = 1;
      } else if (lane < HW) {
        s_cor[warp + lane * kWarps] = 1.f;
      }
#pragma unroll
      for (int i = 0; i < HW; ++i) {
        const int h = warp + i * kWarps;
        if (h < H) {
          const __nv_bfloat16 p = __float2bfloat16_rn(fast_exp2(m[i] - m_run[i]));
          l_run[i] += __bfloat162float(p);
          s_p[h * kPRow + lane] = p;
        }
      }
    }
    if (single) cp_async_wait<1>();
    __syncthreads();

    // ---- PV ----
    const bool rescale = s_flag[t & 1] != 0;
#pragma unroll
    for (int u = 0; u < MAXU; ++u) {
      const int unit = warp + u * kWarps;
      if (unit < units) {
        if (rescale)
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            const float c0 = s_cor[head0[u] + n * 8 + tq * 2], c1 = s_cor[head0[u] + n * 8 + tq * 2 + 1];
            o[u][n][0] *= c0;
            o[u][n][1] *= c1;
            o[u][n][2] *= c0;
            o[u][n][3] *= c1;
          }
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
          // A = V^T: 16 value columns x 16 keys from rows of keys (transposing load)
          uint32_t af[4];
          ldmatrix_x4_trans(af, vt + offV[u] + kk * 32 * strV);
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            uint32_t bf[2];
            ldmatrix_x2(bf, offP[u] + n * (8 * kPRow * 2) + kk * 32);
            mma_bf16_16816(o[u][n], af, bf);
          }
        }
      }
    }
    if (single) {
      __syncthreads();
      if (t + 1 < t1) load_tile(t + 1, 2);
      cp_async_commit();
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < HW; ++i) {
    const int h = warp + i * kWarps;
    const float l = warp_sum(l_run[i]);
    if (h < H && lane == 0) {
      s_l[h] = l;
      s_m[h] = m_run[i];
    }
  }
  __syncthreads();
  const int64_t part = static_cast<int64_t>(seq) * parts.splits + blockIdx.x;
  if (parts.splits > 1)
    for (int h = tid; h < H; h += kThreads) {
      parts.ml[(part * H + h) * 2] = s_m[h];
      parts.ml[(part * H + h) * 2 + 1] = s_l[h];
    }
#pragma unroll
  for (int u = 0; u < MAXU; ++u) {
    const int unit = warp + u * kWarps;
    if (unit < units && t0 < t1) {
      const int c = unit / mt_per_head, mt = unit - c * mt_per_head;
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int hg = n * 8 + tq * 2 + (e & 1), d = mt * 16 + g + (e >> 1) * 8;
          if (hg < Gs) {
            const int h = c * Gs + hg;
            if (parts.splits > 1) {
              parts.o[(part * H + h) * dv + d] = o[u][n][e];
            } else {
              const __nv_bfloat16* gp = a.gate ? static_cast<const __nv_bfloat16*>(a.gate) +
                                                     static_cast<int64_t>(seq) * a.gate_stride + h * dv + d : nullptr;
              static_cast<__nv_bfloat16*>(a.out)[(static_cast<int64_t>(seq) * H + h) * dv + d] =
                  __float2bfloat16_rn(gated(o[u][n][e] / s_l[h], gp));
            }
          }
        }
    }
  }
}

// out[seq, h] = sum over shares of 2^(m_s - m) O_s / sum of 2^(m_s - m) l_s, gated; one warp per (sequence, head)
__global__ void __launch_bounds__(128) talking_merge_kernel(const TalkArgs a, const DecodeParts parts) {
  const int64_t w = static_cast<int64_t>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, H = a.H, dv = a.dv, n = parts.splits;
  if (w >= a.rows * H) return;
  const int64_t seq = w / H;
  const int h = static_cast<int>(w - seq * H);
  if (a.ctx_lens[seq] <= 0) return;
  const int64_t p = (seq * n + lane) * H + h;
  const float m = lane < n ? parts.ml[p * 2] : kNoRef, l = lane < n ? parts.ml[p * 2 + 1] : 0.f;
  const float mx = warp_max(m);
  const float f = m == kNoRef ? 0.f : fast_exp2(m - mx);
  const float inv = 1.f / warp_sum(f * l);
  for (int d0 = 0; d0 < dv; d0 += 32) {
    const int d = d0 + lane;
    float acc = 0.f;
    for (int s = 0; s < n; ++s) {
      const float fs = __shfl_sync(0xffffffffu, f, s);
      if (fs > 0.f && d < dv) acc += fs * parts.o[((seq * n + s) * H + h) * dv + d];
    }
    if (d >= dv) break;
    const __nv_bfloat16* gp =
        a.gate ? static_cast<const __nv_bfloat16*>(a.gate) + seq * a.gate_stride + h * dv + d : nullptr;
    static_cast<__nv_bfloat16*>(a.out)[(seq * H + h) * dv + d] = __float2bfloat16_rn(gated(acc * inv, gp));
  }
}

int splits_for(int n, int window) {
  // several CTAs per SM, shares of at least 128 keys
  const int sms = sm_count_cached();
  int s = (4 * (sms > 0 ? sms : 148) + n - 1) / n;
  if (window > 0) s = s < (window + 127) / 128 ? s : (window + 127) / 128;
  return s < 1 ? 1 : s > kMaxSplits ? kMaxSplits : s;
}

template <int HP, int NT, int MAXU, int NW, bool COMMON>
int launch_decode_as(const TalkArgs& a, const DecodeParts& parts, size_t smem, cudaStream_t s) {
  auto kern = talking_decode_kernel<HP, NT, MAXU, NW, COMMON>;
  static size_t configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64 || configured[dev] < smem) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
      return B200_ERR_LAUNCH;
    if (dev >= 0 && dev < 64) configured[dev] = smem;
  }
  kern<<<dim3(parts.splits, static_cast<unsigned>(a.rows)), NW * 32, smem, s>>>(a, parts);
  int rc = launch_result();
  if (rc != B200_OK || parts.splits == 1) return rc;
  talking_merge_kernel<<<static_cast<unsigned>((a.rows * a.H + 3) / 4), 128, 0, s>>>(a, parts);
  return launch_result();
}

template <int HP, int NT, int MAXU>
int launch_decode(const TalkArgs& a, const DecodeParts& parts, size_t smem, cudaStream_t s) {
  const bool common = a.cap > 0.f && a.window > 0 && a.bias_len >= a.window;
  if (HP >= 16 || smem > 76 * 1024) {
    constexpr int U = MAXU / 2;
    return common ? launch_decode_as<HP, NT, U, 8, true>(a, parts, smem, s)
                  : launch_decode_as<HP, NT, U, 8, false>(a, parts, smem, s);
  }
  return common ? launch_decode_as<HP, NT, MAXU, 4, true>(a, parts, smem, s)
                : launch_decode_as<HP, NT, MAXU, 4, false>(a, parts, smem, s);
}

template <int HP>
int dispatch_decode(const TalkArgs& a, const DecodeParts& parts, size_t smem, cudaStream_t s) {
  const int nt = (a.H / a.Hkv + 7) / 8, u = (a.Hkv * a.dv / 16 + 3) / 4;    // row tiles per warp of four
  if (nt == 1) {
    if (u <= 4) return launch_decode<HP, 1, 4>(a, parts, smem, s);
    if (u <= 8) return launch_decode<HP, 1, 8>(a, parts, smem, s);
    if (u <= 16) return launch_decode<HP, 1, 16>(a, parts, smem, s);
    if (u <= 32) return launch_decode<HP, 1, 32>(a, parts, smem, s);
  } else if (nt == 2 && HP >= 16) {
    if (u <= 8) return launch_decode<HP, HP >= 16 ? 2 : 1, 8>(a, parts, smem, s);
    if (u <= 16) return launch_decode<HP, HP >= 16 ? 2 : 1, 16>(a, parts, smem, s);
  } else if (nt == 4 && HP >= 32) {
    if (u <= 8) return launch_decode<HP, HP >= 32 ? 4 : 1, 8>(a, parts, smem, s);
  }
  return B200_ERR_UNSUPPORTED;
}

}  // namespace

size_t talking_decode_workspace_bytes(int n, int H, int dv, int window) {
  const int splits = splits_for(n, window);
  return splits == 1 ? 0 : static_cast<size_t>(n) * splits * H * (dv + 2) * sizeof(float);
}

int talking_decode_mma_launch(const TalkArgs& a, cudaStream_t s) {
  if (!a.talk_host || a.cu_q || a.H > 32 || a.dk % 16 || a.dv % 16 || a.rows > 65535) return B200_ERR_UNSUPPORTED;
  if (a.q_stride % 8 || !aligned16(a.q) || !aligned16(a.kc) || !aligned16(a.vc)) return B200_ERR_UNSUPPORTED;
  DecodeParts parts{};
  parts.splits = splits_for(static_cast<int>(a.rows), a.window);
  if (parts.splits > 1) {
    if (a.workspace_bytes < talking_decode_workspace_bytes(static_cast<int>(a.rows), a.H, a.dv, a.window))
      return B200_ERR_WORKSPACE;
    parts.ml = static_cast<float*>(a.workspace);
    parts.o = parts.ml + static_cast<size_t>(a.rows) * parts.splits * a.H * 2;
  }
  const size_t q_bytes = size_t(a.H + (a.H / a.Hkv + 7) / 8 * 8) * (a.dk + 8) * 2;
  const size_t stage = size_t(BK) * (a.Hkv * a.dk + 8 + a.Hkv * a.dv + 8) * 2;
  parts.stages = q_bytes + 3 * stage <= 50 * 1024 ? 3 : 2;
  if (q_bytes + 2 * stage > 76 * 1024) parts.stages = 1;      // other CTAs of the SM hide the loads
  const size_t smem = q_bytes + parts.stages * stage;
  if (smem > 208 * 1024) return B200_ERR_UNSUPPORTED;
  if (a.H <= 8) return dispatch_decode<8>(a, parts, smem, s);
  if (a.H <= 16) return dispatch_decode<16>(a, parts, smem, s);
  return dispatch_decode<32>(a, parts, smem, s);
}

}  // namespace b200
