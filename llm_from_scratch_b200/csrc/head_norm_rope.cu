// Attention prologue for models that norm every query / key head on its own and rotate neighbouring channels:
//
//   q[h] = rot(rms(q_in[h]) wq),  k[g] = rot(rms(k_in[g]) wk)     rms over the head, fp32
//   rot: channels (2i, 2i + 1) of the first `rot_dims` turn by position * freq[i], the others pass
//
// in one launch with the scatter of k and v into the paged pool.  A CTA computes the angles once per token for all heads.
#include <initializer_list>

#include "rotary.cuh"

namespace b200 {
namespace {

constexpr int kThreads = 256, kTokens = 4;

struct HnArgs {
  const void* q;             // [T, Hq, D] (token stride free)
  const void* k;             // [T, Hkv, D]
  const void* v;             // [T, Hkv, Dv]
  int64_t stride;
  const float* wq;           // [D]
  const float* wk;
  float eps;
  const double* freq;        // [rot_dims / 2]
  int half;                  // rot_dims / 2
  const int64_t* positions;  // [T]
  void* q_out;               // [T, Hq, D]
  void* k_out;               // [T, Hkv, D]
  void* kc;                  // pools or null
  void* vc;
  const int64_t* slots;      // [T], < 0: not stored
  int64_t num_slots, T;
  int Hq, Hkv, D, Dv;
  int32_t* status;
};

template <typename T, int V>
__device__ __forceinline__ void load_pairs(const T* p, int left, float (&x)[V]) {
  if constexpr (V == 4) {
    if constexpr (sizeof(T) == 2) {
      const uint2 a = *reinterpret_cast<const uint2*>(p);
      const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.x));
      const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.y));
      x[0] = lo.x, x[1] = lo.y, x[2] = hi.x, x[3] = hi.y;
    } else {
      const float4 a = *reinterpret_cast<const float4*>(p);
      x[0] = a.x, x[1] = a.y, x[2] = a.z, x[3] = a.w;
    }
  } else {
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = e < left ? to_float<T>(p[e]) : 0.f;
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_pairs(T* p, int left, const float (&x)[V]) {
  if constexpr (V == 4) {
    if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]));
    else *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  } else {
#pragma unroll
    for (int e = 0; e < V; ++e)
      if (e < left) p[e] = from_float<T>(x[e]);
  }
}

// A warp per (token, query or key head), V consecutive channels per lane and trip, N trips.
template <typename T, int V, int N>
__global__ void __launch_bounds__(kThreads) head_norm_rope_kernel(const HnArgs a) {
  extern __shared__ float2 cs[];     // [kTokens][half] (cos, sin)
  const int64_t t0 = static_cast<int64_t>(blockIdx.x) * kTokens;
  const int nt = static_cast<int>(a.T - t0 < kTokens ? a.T - t0 : kTokens);
  for (int i = threadIdx.x; i < nt * a.half; i += kThreads) {
    const int t = i / a.half, j = i - t * a.half;
    cs[i] = rotary_angle(a.positions[t0 + t], a.freq[j]);
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, heads = a.Hq + a.Hkv;
  for (int task = warp; task < nt * heads; task += kThreads / 32) {
    const int t = task / heads, h = task - t * heads;
    const int64_t tok = t0 + t;
    const bool is_q = h < a.Hq;
    const int hh = is_q ? h : h - a.Hq;
    const T* src = static_cast<const T*>(is_q ? a.q : a.k) + tok * a.stride + static_cast<int64_t>(hh) * a.D;
    const float* w = is_q ? a.wq : a.wk;
    float x[N][V];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * 32 + lane) * V;
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = 0.f;
      if (c < a.D) load_pairs<T, V>(src + c, a.D - c, x[i]);
#pragma unroll
      for (int e = 0; e < V; ++e) ss += x[i][e] * x[i][e];
    }
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(a.D) + a.eps);
    T* out = static_cast<T*>(is_q ? a.q_out : a.k_out) + (tok * (is_q ? a.Hq : a.Hkv) + hh) * a.D;
    T* pool = nullptr;
    if (!is_q && a.kc != nullptr) {
      const int64_t slot = a.slots[tok];
      if (slot >= a.num_slots) {
        if (lane == 0) report(a.status, B200_ERR_BOUNDS);
      } else if (slot >= 0) {
        pool = static_cast<T*>(a.kc) + (slot * a.Hkv + hh) * a.D;
      }
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * 32 + lane) * V;
      if (c >= a.D) continue;
#pragma unroll
      for (int e = 0; e < V; e += 2) {
        float u = x[i][e] * inv * (c + e < a.D ? w[c + e] : 0.f), v = x[i][e + 1] * inv * (c + e + 1 < a.D ? w[c + e + 1] : 0.f);
        const int pair = (c + e) >> 1;
        if (pair < a.half) {
          const float2 r = cs[t * a.half + pair];
          const float nu = u * r.x - v * r.y, nv = v * r.x + u * r.y;
          u = nu;
          v = nv;
        }
        x[i][e] = u;
        x[i][e + 1] = v;
      }
      store_pairs<T, V>(out + c, a.D - c, x[i]);
      if (pool != nullptr) store_pairs<T, V>(pool + c, a.D - c, x[i]);
    }
  }
  if (a.vc != nullptr) {
    const int W = a.Hkv * a.Dv;
    constexpr int E = 16 / sizeof(T);
    const bool wide = W % E == 0 && a.stride % E == 0 && (reinterpret_cast<uintptr_t>(a.v) & 15) == 0 &&
                      (reinterpret_cast<uintptr_t>(a.vc) & 15) == 0;
    const int per = wide ? W / E : W;
    for (int i = threadIdx.x; i < nt * per; i += kThreads) {
      const int t = i / per, c = i - t * per;
      const int64_t slot = a.slots[t0 + t];
      if (slot < 0 || slot >= a.num_slots) continue;
      const T* vs = static_cast<const T*>(a.v) + (t0 + t) * a.stride;
      T* vd = static_cast<T*>(a.vc) + slot * W;
      if (wide) reinterpret_cast<uint4*>(vd)[c] = reinterpret_cast<const uint4*>(vs)[c];
      else vd[c] = vs[c];
    }
  }
}

// bf16 heads of 8 * LPH channels (LPH a power of two up to 32): LPH lanes per head, 16 bytes per lane, 32 / LPH heads per warp
template <int LPH>
__global__ void __launch_bounds__(kThreads) head_norm_rope_wide_kernel(const HnArgs a) {
  extern __shared__ float2 cs[];     // [kTokens][half] (cos, sin)
  constexpr int HPW = 32 / LPH, D = 8 * LPH;
  const int64_t t0 = static_cast<int64_t>(blockIdx.x) * kTokens;
  const int nt = static_cast<int>(a.T - t0 < kTokens ? a.T - t0 : kTokens);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, heads = a.Hq + a.Hkv, c = (lane % LPH) * 8;
  for (int i = threadIdx.x; i < nt * a.half; i += kThreads) {
    const int t = i / a.half, j = i - t * a.half;
    cs[i] = rotary_angle(a.positions[t0 + t], a.freq[j]);
  }
  const bool turns = c < 2 * a.half;             // whole 8-channel groups turn or pass (half a multiple of four)
  __syncthreads();
  union Pack {
    uint4 u;
    __nv_bfloat162 p[4];
  };
  for (int task = warp * HPW + lane / LPH; task < (nt * heads + HPW - 1) / HPW * HPW; task += kThreads / 32 * HPW) {
    const bool live = task < nt * heads;
    const int t = live ? task / heads : 0, h = live ? task - t * heads : 0;
    const int64_t tok = t0 + t;
    const bool is_q = h < a.Hq;
    const int hh = is_q ? h : h - a.Hq;
    Pack x;
    x.u = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(is_q ? a.q : a.k) + tok * a.stride + hh * D + c);
    float v[8], ss = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(x.p[e]);
      v[2 * e] = f.x;
      v[2 * e + 1] = f.y;
      ss += f.x * f.x + f.y * f.y;
    }
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = rsqrtf(ss / static_cast<float>(D) + a.eps);
    const float* w = (is_q ? a.wq : a.wk) + c;
    const float4 w0 = *reinterpret_cast<const float4*>(w), w1 = *reinterpret_cast<const float4*>(w + 4);
    const float ww[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float u = v[2 * e] * inv * ww[2 * e], z = v[2 * e + 1] * inv * ww[2 * e + 1];
      if (turns) {
        const float2 r = cs[t * a.half + c / 2 + e];
        const float nu = u * r.x - z * r.y;
        z = z * r.x + u * r.y;
        u = nu;
      }
      x.p[e] = __floats2bfloat162_rn(u, z);
    }
    if (!live) continue;
    *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(is_q ? a.q_out : a.k_out) + (tok * (is_q ? a.Hq : a.Hkv) + hh) * D + c) = x.u;
    if (!is_q && a.kc != nullptr) {
      const int64_t slot = a.slots[tok];
      if (slot >= a.num_slots) report(a.status, B200_ERR_BOUNDS);
      else if (slot >= 0)
        *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.kc) + (slot * a.Hkv + hh) * D + c) = x.u;
    }
  }
  if (a.vc != nullptr) {
    const int per = a.Hkv * a.Dv / 8;
    for (int i = threadIdx.x; i < nt * per; i += kThreads) {
      const int t = i / per, j = i - t * per;
      const int64_t slot = a.slots[t0 + t];
      if (slot < 0 || slot >= a.num_slots) continue;
      reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.vc) + slot * a.Hkv * a.Dv)[j] =
          reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.v) + (t0 + t) * a.stride)[j];
    }
  }
}

// whether the wide kernel takes the call, and its launch
bool launch_wide(const HnArgs& a, cudaStream_t s) {
  const int lph = a.D / 8;
  if (a.D % 8 || a.Dv % 8 || (lph & (lph - 1)) || lph > 32 || a.half % 4 || a.stride % 8) return false;
  for (const void* p : {a.q, a.k, a.v, static_cast<const void*>(a.wq), static_cast<const void*>(a.wk),
                        static_cast<const void*>(a.q_out), static_cast<const void*>(a.k_out), static_cast<const void*>(a.kc),
                        static_cast<const void*>(a.vc)})
    if (!aligned16(p)) return false;
  const unsigned grid = static_cast<unsigned>((a.T + kTokens - 1) / kTokens);
  const size_t smem = static_cast<size_t>(kTokens) * a.half * sizeof(float2);
  switch (lph) {
    case 4: head_norm_rope_wide_kernel<4><<<grid, kThreads, smem, s>>>(a); break;
    case 8: head_norm_rope_wide_kernel<8><<<grid, kThreads, smem, s>>>(a); break;
    case 16: head_norm_rope_wide_kernel<16><<<grid, kThreads, smem, s>>>(a); break;
    case 32: head_norm_rope_wide_kernel<32><<<grid, kThreads, smem, s>>>(a); break;
    default: return false;
  }
  return true;
}

template <typename T>
int launch(const HnArgs& a, cudaStream_t s) {
  if (sizeof(T) == 2 && launch_wide(a, s)) return launch_result();
  const unsigned grid = static_cast<unsigned>((a.T + kTokens - 1) / kTokens);
  const size_t smem = static_cast<size_t>(kTokens) * a.half * sizeof(float2);
  const bool vec = a.D % 4 == 0 && a.D > 64 && a.stride % 4 == 0 && aligned16(a.q) && aligned16(a.k) && aligned16(a.q_out) &&
                   aligned16(a.k_out) && (!a.kc || aligned16(a.kc));
  if (vec && a.D <= 128) head_norm_rope_kernel<T, 4, 1><<<grid, kThreads, smem, s>>>(a);
  else if (vec && a.D <= 256) head_norm_rope_kernel<T, 4, 2><<<grid, kThreads, smem, s>>>(a);
  else if (a.D <= 64) head_norm_rope_kernel<T, 2, 1><<<grid, kThreads, smem, s>>>(a);
  else head_norm_rope_kernel<T, 2, 8><<<grid, kThreads, smem, s>>>(a);
  return launch_result();
}

}  // namespace
}  // namespace b200

extern "C" int b200_head_norm_rope_store(const void* q, const void* k, const void* v, int64_t token_stride,
                                         const float* q_norm_w, const float* k_norm_w, float eps, const double* freq,
                                         int32_t rot_dims, const int64_t* positions, void* q_out, void* k_out, void* k_cache,
                                         void* v_cache, const int64_t* slot_mapping, int64_t num_slots, int64_t num_tokens,
                                         int32_t num_q_heads, int32_t num_kv_heads, int32_t dim_k, int32_t dim_v,
                                         int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (num_tokens < 0 || num_q_heads <= 0 || num_kv_heads <= 0 || dim_k <= 0 || dim_v <= 0 || rot_dims < 0 ||
      rot_dims % 2 || rot_dims > dim_k)
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (dim_k > 512) return B200_ERR_UNSUPPORTED;
  if (num_tokens == 0) return B200_OK;
  if (!q || !k || !v || !q_norm_w || !k_norm_w || (rot_dims && !freq) || !positions || !q_out || !k_out) return B200_ERR_ARG;
  if ((k_cache != nullptr) != (v_cache != nullptr) || (k_cache && !slot_mapping)) return B200_ERR_ARG;
  if (num_tokens > 2147483647) return B200_ERR_TOO_LARGE;
  HnArgs a{q, k, v, token_stride, q_norm_w, k_norm_w, eps, freq, rot_dims / 2, positions, q_out, k_out, k_cache, v_cache,
           slot_mapping, num_slots, num_tokens, num_q_heads, num_kv_heads, dim_k, dim_v, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == B200_DTYPE_F32 ? launch<float>(a, s) : launch<__nv_bfloat16>(a, s);
}
