// Attention prologue of layers whose queries and keys pass a short causal convolution, a norm over the whole projection and a
// rotation of channel halves, and whose values are the convolved keys themselves.  One launch behind the projection:
//
//   u[t] = sum_m w[m] in[t - (taps - 1) + m]       per channel of q and k, zeros before the sequence's start
//   v    = u_k
//   q    = rot(u_q / sqrt(mean(u_q^2) + eps) wq),  k = rot(u_k / sqrt(mean(u_k^2) + eps) wk)     means over all heads, fp32
//   rot: channels (i, i + half), i < half, of every head turn by position * freq[i], the others pass
//
// with the scatter of k and v into the paged pool.  The last taps - 1 inputs of every sequence are its state (position p in row
// p mod (taps - 1) of the slot, channels [q | k]).  A CTA owns a segment of one sequence with all its channels; the CTA of the
// first segment, the only one that reads the state, is the one that moves it on, each thread its own channels.
#include <initializer_list>

#include "rotary.cuh"
#include "sequences.cuh"

namespace b200 {
namespace {

struct CnArgs {
  const void* q;             // [T, Cq] (token stride free)
  const void* k;             // [T, Ck]
  int64_t stride;
  const float* wq;           // [taps, Cq], the last row weighs the current token
  const float* wk;           // [taps, Ck]
  int taps;
  float* ring;               // [slots, taps - 1, Cq + Ck] or null (one tap)
  const int64_t* slots;
  int64_t num_slots;
  const int32_t* cu_q;       // [n + 1], or null: row i is sequence i
  const int32_t* cu_k;
  const int64_t* ctx_lens;
  int n;
  const float* nq;           // [Cq] norm weights
  const float* nk;           // [Ck]
  float eps;
  const double* freq;        // [half]
  int half;
  const int64_t* positions;  // [T]
  void* q_out;               // [T, Cq]
  void* k_out;               // [T, Ck] or null
  void* v_out;               // [T, Ck] or null
  void* kc;                  // pools [slots, Ck] or null
  void* vc;
  const int64_t* slot_map;   // [T], < 0: not stored
  int64_t pool_slots, T;
  int Cq, Ck, D;
  int seg_len;               // tokens per CTA, at least taps - 1
  int32_t* status;
};

constexpr int kSegment = 16, kMaxSegment = 64;

// slot in the pool of a token, -1: none
__device__ __forceinline__ int64_t pool_slot(const CnArgs& a, int64_t tok) {
  if (a.kc == nullptr) return -1;
  const int64_t s = a.slot_map[tok];
  if (s >= a.pool_slots) {
    if (threadIdx.x == 0) report(a.status, B200_ERR_BOUNDS);
    return -1;
  }
  return s;
}

__device__ __forceinline__ void angles(const CnArgs& a, const Segment& g, float2* cs) {
  for (int i = threadIdx.x; i < g.count * a.half; i += blockDim.x) {
    const int t = i / a.half, j = i - t * a.half;
    cs[i] = rotary_angle(a.positions[g.first + t], a.freq[j]);
  }
}

// ---- eight channels per thread (bf16), as four packed fp32 pairs ----
__device__ __forceinline__ void load_pairs(const float* p, f32x2 (&v)[4]) {
  const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(p), b = *reinterpret_cast<const ulonglong2*>(p + 4);
  v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
}
__device__ __forceinline__ void store_pairs(float* p, const f32x2 (&v)[4]) {
  *reinterpret_cast<ulonglong2*>(p) = make_ulonglong2(v[0], v[1]);
  *reinterpret_cast<ulonglong2*>(p + 4) = make_ulonglong2(v[2], v[3]);
}
__device__ __forceinline__ void unpack_pairs(uint4 u, f32x2 (&v)[4]) {
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) v[e] = pack2(__uint_as_float(w[e] << 16), __uint_as_float(w[e] & 0xffff0000u));
}
__device__ __forceinline__ uint4 round_pairs(const f32x2 (&v)[4]) {
  uint32_t w[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 f = unpack2(v[e]);
    w[e] = pack_bf16x2(f.x, f.y);
  }
  return make_uint4(w[0], w[1], w[2], w[3]);
}

// Shared-memory rows that threads read in pieces of eight floats are kept as two planes of four, so that neighbouring threads'
// 16-byte accesses lie side by side.
__device__ __forceinline__ void load_planes(const float* p, int plane, f32x2 (&v)[4]) {
  const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(p), b = *reinterpret_cast<const ulonglong2*>(p + plane);
  v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
}

// half a multiple of eight, so that a thread's partner channels are one thread's.  SHFL: that thread is in the same warp; else
// the values pass through shared memory.
template <int TAPS, bool SHFL, int THREADS>
__global__ void __launch_bounds__(THREADS, 640 / THREADS > 0 ? 640 / THREADS : 1) conv_norm_rope_kernel(const CnArgs a) {
  extern __shared__ float4 smem4[];
  __shared__ float sums[2][2][32];                                          // squares of every warp's channels of q and k
  __shared__ int64_t s_slot[kMaxSegment];
  Segment g;
  if (!segment_of(a, a.seg_len, &g)) return;
  const int C = a.Cq + a.Ck, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  float* cos_t = reinterpret_cast<float*>(smem4);                           // [seg_len][2 planes][half / 2]
  float* sin_t = cos_t + a.seg_len * a.half;
  float* swap = sin_t + a.seg_len * a.half;                                 // [2][2 planes][C / 2] weighted values, for the partners
  const int c = threadIdx.x * 8;                                            // channel of [q | k]
  const bool in = c < C, is_k = c >= a.Cq;
  const int cc = is_k ? c - a.Cq : c, width = is_k ? a.Ck : a.Cq;           // channel of q or k
  const int ch = cc % a.D;                                                  // and of the head
  const int partner = ch < a.half ? a.half : ch < 2 * a.half ? -a.half : 0;
  const bool mixed = a.Cq % 256 != 0;                                       // a warp holds channels of both
  const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(is_k ? a.k : a.q) + g.first * a.stride + cc;
  auto input = [&](int t) {                                                 // loads run two tokens ahead
    return in && t < g.count ? *reinterpret_cast<const uint4*>(src + t * a.stride) : make_uint4(0, 0, 0, 0);
  };
  uint4 next = input(0), after = input(1);
  f32x2 w[TAPS][4];
  uint4 hist[TAPS - 1];                                                     // hist[m]: input TAPS - 1 - m tokens back
#pragma unroll
  for (int m = 0; m < TAPS; ++m)
#pragma unroll
    for (int e = 0; e < 4; ++e) w[m][e] = 0;
#pragma unroll
  for (int m = 0; m < TAPS - 1; ++m) hist[m] = make_uint4(0, 0, 0, 0);
  if (in) {
#pragma unroll
    for (int m = 0; m < TAPS; ++m) load_pairs((is_k ? a.wk : a.wq) + static_cast<int64_t>(m) * width + cc, w[m]);
#pragma unroll
    for (int m = 0; m < TAPS - 1; ++m) {
      const int back = TAPS - 1 - m;                                        // tokens before the segment's first
      if (g.index > 0) {
        hist[m] = *reinterpret_cast<const uint4*>(src - back * a.stride);
      } else if (g.slot >= 0 && g.pos0 - back >= 0) {
        f32x2 v[4];
        load_pairs(a.ring + (g.slot * (TAPS - 1) + (g.pos0 - back) % (TAPS - 1)) * C + c, v);
        hist[m] = round_pairs(v);                                           // the state holds rounded values
      }
    }
    if (g.index == 0 && g.slot >= 0) {
      for (int m = 0; m < min(TAPS - 1, g.len); ++m) {
        const int t = g.len - 1 - m;
        f32x2 v[4];
        unpack_pairs(*reinterpret_cast<const uint4*>(src + t * a.stride), v);
        store_pairs(a.ring + (g.slot * (TAPS - 1) + (g.pos0 + t) % (TAPS - 1)) * C + c, v);
      }
    }
  }
  for (int i = threadIdx.x; i < 4 * 32; i += blockDim.x)
    if ((i & 31) >= nw) (&sums[0][0][0])[i] = 0.f;
  for (int t = threadIdx.x; t < g.count; t += blockDim.x) s_slot[t] = pool_slot(a, g.first + t);
  for (int i = threadIdx.x; i < g.count * a.half; i += blockDim.x) {
    const int t = i / a.half, j = i - t * a.half;
    const float2 r = rotary_angle(a.positions[g.first + t], a.freq[j]);
    const int at = t * a.half + (j >> 2 & 1) * (a.half / 2) + (j >> 3) * 4 + (j & 3);
    cos_t[at] = r.x;
    sin_t[at] = r.y;
  }
  const float per = 1.f / static_cast<float>(width);
  const float* norm = (is_k ? a.nk : a.nq) + cc;
  const f32x2 sign = pack2(partner < 0 ? -1.f : 1.f, partner < 0 ? -1.f : 1.f);
  const int angle = (partner > 0 ? ch : ch - a.half) / 2, to = threadIdx.x * 4 + partner / 2, other = lane + partner / 8;
  for (int t = 0; t < g.count; ++t) {
    const uint4 cur = next;
    next = after;
    after = input(t + 2);
    f32x2 y[4], z[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] = 0;
#pragma unroll
    for (int m = 0; m < TAPS; ++m) {
      f32x2 v[4];
      unpack_pairs(m < TAPS - 1 ? hist[m] : cur, v);
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = fma2(w[m][e], v[e], y[e]);
    }
#pragma unroll
    for (int m = 0; m < TAPS - 1; ++m) hist[m] = m + 1 < TAPS - 1 ? hist[m + 1 < TAPS - 1 ? m + 1 : 0] : cur;
    f32x2 sq = 0;
#pragma unroll
    for (int e = 0; e < 4; ++e) sq = fma2(y[e], y[e], sq);
    const float2 f = unpack2(sq);
    float* part = sums[t & 1][0];
    if (mixed) {
      const float sq_q = warp_sum(is_k ? 0.f : f.x + f.y), sq_k = warp_sum(is_k ? f.x + f.y : 0.f);
      if (lane == 0) {
        part[warp] = sq_q;
        part[32 + warp] = sq_k;
      }
    } else {
      const float sum = warp_sum(f.x + f.y);
      if (lane == 0) {
        part[is_k * 32 + warp] = sum;
        part[!is_k * 32 + warp] = 0.f;
      }
    }
    uint4 raw = make_uint4(0, 0, 0, 0);
    if (is_k) raw = round_pairs(y);
    if (in) {
      f32x2 weight[4];
      load_pairs(norm, weight);
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = mul2(y[e], weight[e]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) z[e] = mul2(y[e], sign);                  // the upper half's values enter with a minus
    float* ex = swap + (t & 1) * C;
    if constexpr (SHFL) {
#pragma unroll
      for (int e = 0; e < 4; ++e) z[e] = __shfl_sync(0xffffffffu, z[e], other);
    } else if (partner != 0 && in) {
      *reinterpret_cast<ulonglong2*>(ex + threadIdx.x * 4) = make_ulonglong2(z[0], z[1]);
      *reinterpret_cast<ulonglong2*>(ex + C / 2 + threadIdx.x * 4) = make_ulonglong2(z[2], z[3]);
    }
    __syncthreads();
    float total = warp_sum(part[(mixed ? 0 : is_k) * 32 + lane]);
    if (mixed) {
      const float total_k = warp_sum(part[32 + lane]);
      if (is_k) total = total_k;
    }
    if (!in) continue;
    const float r = rsqrtf(total * per + a.eps);
    const f32x2 inv = pack2(r, r);
    if (partner != 0) {
      f32x2 cs[4], sn[4];
      if constexpr (!SHFL) load_planes(ex + to, C / 2, z);
      load_planes(cos_t + t * a.half + angle, a.half / 2, cs);
      load_planes(sin_t + t * a.half + angle, a.half / 2, sn);
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = fma2(z[e], sn[e], mul2(y[e], cs[e]));
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] = mul2(y[e], inv);
    const uint4 o = round_pairs(y);
    const int64_t at = (g.first + t) * width + cc;
    if (!is_k) {
      *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.q_out) + at) = o;
      continue;
    }
    if (a.k_out != nullptr) {
      *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.k_out) + at) = o;
      *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.v_out) + at) = raw;
    }
    const int64_t slot = s_slot[t];
    if (slot >= 0) {
      *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.kc) + slot * a.Ck + cc) = o;
      *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.vc) + slot * a.Ck + cc) = raw;
    }
  }
}

// ---- any sizes and dtype, a token at a time ----
template <typename T>
__global__ void __launch_bounds__(256) conv_norm_rope_any_kernel(const CnArgs a) {
  extern __shared__ float4 smem4[];
  __shared__ float sums[2][8];
  Segment g;
  if (!segment_of(a, a.seg_len, &g)) return;
  const int C = a.Cq + a.Ck, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, back = a.taps - 1;
  float2* cs = reinterpret_cast<float2*>(smem4);                            // [seg_len][half]
  float* y = reinterpret_cast<float*>(cs + a.seg_len * a.half);             // [C]
  angles(a, g, cs);
  // projected value of channel c, t tokens from the segment's first (t < 0: before it)
  auto source = [&](int c, int t) -> const T* {
    return c < a.Cq ? static_cast<const T*>(a.q) + (g.first + t) * a.stride + c
                    : static_cast<const T*>(a.k) + (g.first + t) * a.stride + c - a.Cq;
  };
  auto input = [&](int c, int t) -> float {
    if (t >= 0 || g.index > 0) return to_float<T>(*source(c, t));
    if (g.slot < 0 || g.pos0 + t < 0) return 0.f;
    return a.ring[(g.slot * back + (g.pos0 + t) % back) * C + c];
  };
  for (int t = 0; t < g.count; ++t) {
    const int64_t tok = g.first + t, slot = pool_slot(a, tok);
    float sq = 0.f, sk = 0.f;
    __syncthreads();                                                        // y and the sums are free
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
      const bool is_k = c >= a.Cq;
      const float* w = is_k ? a.wk + c - a.Cq : a.wq + c;
      const int width = is_k ? a.Ck : a.Cq;
      float v = 0.f;
      for (int m = 0; m < a.taps; ++m) v = fmaf(w[static_cast<int64_t>(m) * width], input(c, t - back + m), v);
      y[c] = v;
      if (is_k) sk += v * v;
      else sq += v * v;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) {
      sums[0][warp] = sq;
      sums[1][warp] = sk;
    }
    __syncthreads();
    float total[2] = {0.f, 0.f};
    for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) {
      total[0] += sums[0][i];
      total[1] += sums[1][i];
    }
    const float inv_q = rsqrtf(total[0] / static_cast<float>(a.Cq) + a.eps), inv_k = rsqrtf(total[1] / static_cast<float>(a.Ck) + a.eps);
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
      const bool is_k = c >= a.Cq;
      const int cc = is_k ? c - a.Cq : c, ch = cc % a.D;
      const float inv = is_k ? inv_k : inv_q;
      const float* norm = is_k ? a.nk : a.nq;
      float o = y[c] * inv * norm[cc];
      if (ch < 2 * a.half) {
        const int p = ch < a.half ? a.half : -a.half;
        const float z = y[c + p] * inv * norm[cc + p];
        const float2 r = cs[t * a.half + (p > 0 ? ch : ch - a.half)];
        o = p > 0 ? o * r.x - z * r.y : o * r.x + z * r.y;
      }
      if (!is_k) {
        static_cast<T*>(a.q_out)[tok * a.Cq + cc] = from_float<T>(o);
        continue;
      }
      if (a.k_out != nullptr) {
        static_cast<T*>(a.k_out)[tok * a.Ck + cc] = from_float<T>(o);
        static_cast<T*>(a.v_out)[tok * a.Ck + cc] = from_float<T>(y[c]);
      }
      if (slot >= 0) {
        static_cast<T*>(a.kc)[slot * a.Ck + cc] = from_float<T>(o);
        static_cast<T*>(a.vc)[slot * a.Ck + cc] = from_float<T>(y[c]);
      }
    }
  }
  if (g.index == 0 && g.slot >= 0)
    for (int m = 0; m < min(back, g.len); ++m) {
      const int t = g.len - 1 - m;
      for (int c = threadIdx.x; c < C; c += blockDim.x)
        a.ring[(g.slot * back + (g.pos0 + t) % back) * C + c] = to_float<T>(*source(c, t));
    }
}

constexpr size_t kMaxShared = 200 * 1024;

// lifts a kernel's limit of dynamic shared memory, once per device
template <typename Kernel>
bool allow_shared(Kernel kern, bool* configured) {
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return false;
  if (!configured[dev]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kMaxShared)) != cudaSuccess)
      return false;
    configured[dev] = true;
  }
  return true;
}

template <int TAPS, bool SHFL, int THREADS>
int launch_wide(const CnArgs& a, unsigned grid, int threads, cudaStream_t s) {
  const size_t smem = (static_cast<size_t>(2 * a.seg_len) * a.half + (SHFL ? 0 : 2 * (a.Cq + a.Ck))) * sizeof(float);
  if (smem > kMaxShared) return B200_ERR_UNSUPPORTED;
  auto kern = conv_norm_rope_kernel<TAPS, SHFL, THREADS>;
  static bool configured[64] = {};
  if (smem > 40 * 1024 && !allow_shared(kern, configured)) return B200_ERR_LAUNCH;
  kern<<<grid, threads, smem, s>>>(a);
  return launch_result();
}

template <int TAPS>
int launch_taps(CnArgs a, cudaStream_t s) {
  const int threads = ((a.Cq + a.Ck) / 8 + 31) / 32 * 32;
  unsigned grid = static_cast<unsigned>(a.T);
  if (a.cu_q != nullptr) {
    // one wave: a CTA's start (weights, angles, inputs before its segment) costs as much as a few tokens
    const int64_t ctas = static_cast<int64_t>(sm_count_cached()) * (threads > 640 ? 1 : 640 / threads);
    const int64_t fit = ctas > a.n ? (a.T + ctas - a.n - 1) / (ctas - a.n) : kMaxSegment;
    a.seg_len = static_cast<int>(fit < 4 ? 4 : fit < kMaxSegment ? fit : kMaxSegment);
    grid = static_cast<unsigned>(a.T / a.seg_len + a.n + 1);
  }
  const bool shfl = 32 % (a.D / 8) == 0;          // a head lies inside one warp
  if (threads <= 320) return shfl ? launch_wide<TAPS, true, 320>(a, grid, threads, s) : launch_wide<TAPS, false, 320>(a, grid, threads, s);
  if (threads <= 640) return shfl ? launch_wide<TAPS, true, 640>(a, grid, threads, s) : launch_wide<TAPS, false, 640>(a, grid, threads, s);
  return shfl ? launch_wide<TAPS, true, 1024>(a, grid, threads, s) : launch_wide<TAPS, false, 1024>(a, grid, threads, s);
}

template <typename T>
int launch_any(const CnArgs& a, unsigned grid, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(a.seg_len) * a.half * sizeof(float2) + static_cast<size_t>(a.Cq + a.Ck) * sizeof(float);
  if (smem > kMaxShared) return B200_ERR_TOO_LARGE;
  static bool configured[64] = {};
  if (smem > 40 * 1024 && !allow_shared(conv_norm_rope_any_kernel<T>, configured)) return B200_ERR_LAUNCH;
  conv_norm_rope_any_kernel<T><<<grid, 256, smem, s>>>(a);
  return launch_result();
}

}  // namespace
}  // namespace b200

extern "C" int b200_conv_norm_rope_store(
    const void* q, const void* k, int64_t token_stride, const float* conv_q, const float* conv_k, int32_t taps, float* ring,
    int64_t num_slots, const int64_t* state_slots, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
    const int64_t* context_lens, int32_t num_seqs, const float* q_norm_w, const float* k_norm_w, float eps, const double* freq,
    int32_t rot_dims, const int64_t* positions, void* q_out, void* k_out, void* v_out, void* k_cache, void* v_cache,
    const int64_t* slot_mapping, int64_t pool_slots, int64_t num_tokens, int32_t num_q_heads, int32_t num_kv_heads,
    int32_t head_dim, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (num_tokens < 0 || num_seqs < 0 || num_slots < 0 || taps <= 0 || num_q_heads <= 0 || num_kv_heads <= 0 || head_dim <= 0 ||
      rot_dims < 0 || rot_dims % 2 || rot_dims > head_dim)
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_tokens == 0) return B200_OK;
  if (!q || !k || !conv_q || !conv_k || !q_norm_w || !k_norm_w || (rot_dims && !freq) || !positions || !q_out || !state_slots ||
      (taps > 1 && !ring))
    return B200_ERR_ARG;
  if ((k_out != nullptr) != (v_out != nullptr) || (k_cache != nullptr) != (v_cache != nullptr) || (k_cache && !slot_mapping))
    return B200_ERR_ARG;
  if (cu_seqlens_q ? !cu_seqlens_k : !context_lens || num_seqs != num_tokens) return B200_ERR_ARG;
  if (num_tokens > 2147483647 - num_seqs) return B200_ERR_TOO_LARGE;
  if (taps == 1) state_slots = nullptr;      // no state
  CnArgs a{q, k, token_stride, conv_q, conv_k, taps, ring, state_slots, num_slots, cu_seqlens_q, cu_seqlens_k, context_lens,
           num_seqs, q_norm_w, k_norm_w, eps, freq, rot_dims / 2, positions, q_out, k_out, v_out, k_cache, v_cache, slot_mapping,
           pool_slots, num_tokens, num_q_heads * head_dim, num_kv_heads * head_dim, head_dim,
           taps - 1 > kSegment ? taps - 1 : kSegment, status};
  if (!cu_seqlens_q) a.seg_len = 1;
  const unsigned grid = static_cast<unsigned>(cu_seqlens_q ? num_tokens / a.seg_len + num_seqs + 1 : num_tokens);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_F32) return launch_any<float>(a, grid, s);
  bool wide = head_dim % 8 == 0 && a.half % 8 == 0 && token_stride % 8 == 0 && a.Cq + a.Ck <= 8192;
  for (const void* p : {q, k, static_cast<const void*>(conv_q), static_cast<const void*>(conv_k), static_cast<const void*>(ring),
                        static_cast<const void*>(q_norm_w), static_cast<const void*>(k_norm_w), static_cast<const void*>(q_out),
                        static_cast<const void*>(k_out), static_cast<const void*>(v_out), static_cast<const void*>(k_cache),
                        static_cast<const void*>(v_cache)})
    wide = wide && aligned16(p);
  if (wide) {
    const int rc = taps == 2 ? launch_taps<2>(a, s) : taps == 3 ? launch_taps<3>(a, s)
                   : taps == 4 ? launch_taps<4>(a, s) : B200_ERR_UNSUPPORTED;
    if (rc != B200_ERR_UNSUPPORTED) return rc;
  }
  return launch_any<__nv_bfloat16>(a, grid, s);
}
