// Hyper-connected residual streams, one launch per sublayer boundary.
//
// A decoder with S residual streams keeps x [T, S, d] in fp32.  Between two sublayers it needs
//
//   y      the result of the sublayer that just ran, per channel times an optional layer scale; the result
//          is one tensor, or the join of two side-by-side mixers  (rms(y0) w0 + rms(y1) w1) / 2
//   x'[t]  = sum_s mix[s][t] x[s] + out[t] y                       (all streams at once from the old ones)
//   u      = sum_t in[t] x'[t]                                     (input weights of the next sublayer)
//   h      = u / sqrt(mean(u^2) + eps) * (w + plus_one)            (its norm, in the activation dtype)
//
// The first boundary starts the streams from the embedding row instead (no update), the last one reads the
// plain sum of the streams (in = NULL) for the final norm.  One CTA per token row: the S streams of a channel
// pass through one thread, u stays in shared memory between the two passes of the norm.  Everything is fp32;
// only h is rounded.
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kMaxStreams = 8;

struct StreamArgs {
  float* x;                  // [T, S, d]
  const int64_t* tokens;     // [T] with embed, else null
  const void* embed;         // [vocab, d]
  int64_t vocab;
  const void* y0;            // [T, d] or null: no update
  const void* y1;            // second mixer of a parallel pair or null
  const float* w0;           // [d] norm weights of the join
  const float* w1;
  float join_eps;
  const float* scale;        // [d] layer scale or null
  const float* mix;          // [S, S], from-to
  const float* out;          // [S]
  const float* in;           // [S] or null = ones
  const float* norm_w;       // [d]
  float plus_one, eps;
  void* h;                   // [T, d]
  int S, d;
  int32_t* status;
};

__device__ __forceinline__ float cta_sum(float v, float* scratch) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < (blockDim.x >> 5); ++w) t += scratch[w];
  return t;
}

template <int V>
struct Pack {
  float v[V];
};
template <int V>
__device__ __forceinline__ Pack<V> load_f(const float* p) {
  Pack<V> r;
  if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    r.v[0] = a.x, r.v[1] = a.y, r.v[2] = a.z, r.v[3] = a.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int V>
__device__ __forceinline__ void store_f(float* p, const Pack<V>& a) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]);
  else *p = a.v[0];
}
template <typename T, int V>
__device__ __forceinline__ Pack<V> load_t(const T* p) {
  Pack<V> r;
  if constexpr (V == 4 && sizeof(T) == 2) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.y));
    r.v[0] = lo.x, r.v[1] = lo.y, r.v[2] = hi.x, r.v[3] = hi.y;
  } else if constexpr (V == 4) {
    r = load_f<4>(reinterpret_cast<const float*>(p));
  } else {
    r.v[0] = to_float<T>(*p);
  }
  return r;
}
template <typename T, int V>
__device__ __forceinline__ void store_t(T* p, const Pack<V>& a) {
  if constexpr (V == 4 && sizeof(T) == 2)
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(a.v[0], a.v[1]), pack_bf16x2(a.v[2], a.v[3]));
  else if constexpr (V == 4) store_f<4>(reinterpret_cast<float*>(p), a);
  else *p = from_float<T>(a.v[0]);
}

// SC: number of streams when known at compile time, 0 = read it from the arguments (<= kMaxStreams)
template <typename T, int V, int SC>
__global__ void __launch_bounds__(512) stream_update_kernel(const StreamArgs a) {
  extern __shared__ float u_row[];     // [d]
  __shared__ float scratch[16];
  constexpr int SM = SC > 0 ? SC : kMaxStreams;
  const int S = SC > 0 ? SC : a.S;
  const int d = a.d;
  const int64_t row = blockIdx.x;
  float* xr = a.x + row * S * d;
  const int step = blockDim.x * V, first = threadIdx.x * V;

  float win[SM];
#pragma unroll
  for (int s = 0; s < SM; ++s) win[s] = s < S ? (a.in ? a.in[s] : 1.f) : 0.f;

  float ss = 0.f;
  if (a.embed != nullptr) {
    int64_t tok = a.tokens[row];
    if (tok < 0 || tok >= a.vocab) {
      if (threadIdx.x == 0) report(a.status, B200_ERR_BOUNDS);
      tok = 0;
    }
    const T* e = static_cast<const T*>(a.embed) + tok * d;
    float wsum = 0.f;
#pragma unroll
    for (int s = 0; s < SM; ++s) wsum += win[s];
    for (int i = first; i < d; i += step) {
      Pack<V> x = load_t<T, V>(e + i), u;
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) store_f<V>(xr + static_cast<int64_t>(s) * d + i, x);
#pragma unroll
      for (int k = 0; k < V; ++k) {
        u.v[k] = wsum * x.v[k];
        ss += u.v[k] * u.v[k];
      }
      store_f<V>(u_row + i, u);
    }
  } else {
    const T* y0 = a.y0 ? static_cast<const T*>(a.y0) + row * d : nullptr;
    const T* y1 = a.y1 ? static_cast<const T*>(a.y1) + row * d : nullptr;
    float n0 = 1.f, n1 = 0.f;
    if (y1 != nullptr) {
      float s0 = 0.f, s1 = 0.f;
      for (int i = first; i < d; i += step) {
        const Pack<V> p0 = load_t<T, V>(y0 + i), p1 = load_t<T, V>(y1 + i);
#pragma unroll
        for (int k = 0; k < V; ++k) {
          s0 += p0.v[k] * p0.v[k];
          s1 += p1.v[k] * p1.v[k];
        }
      }
      n0 = 0.5f * rsqrtf(cta_sum(s0, scratch) / static_cast<float>(d) + a.join_eps);
      n1 = 0.5f * rsqrtf(cta_sum(s1, scratch) / static_cast<float>(d) + a.join_eps);
    }
    float mix[SM * SM], wout[SM];
    if (y0 != nullptr) {
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        wout[s] = s < S ? a.out[s] : 0.f;
#pragma unroll
        for (int t = 0; t < SM; ++t) mix[s * SM + t] = (s < S && t < S) ? a.mix[s * S + t] : 0.f;
      }
    }
    for (int i = first; i < d; i += step) {
      Pack<V> x[SM];
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) x[s] = load_f<V>(xr + static_cast<int64_t>(s) * d + i);
        else
          for (int k = 0; k < V; ++k) x[s].v[k] = 0.f;
      Pack<V> u;
#pragma unroll
      for (int k = 0; k < V; ++k) u.v[k] = 0.f;
      if (y0 != nullptr) {
        Pack<V> y = load_t<T, V>(y0 + i);
        if (y1 != nullptr) {
          const Pack<V> p1 = load_t<T, V>(y1 + i), g0 = load_f<V>(a.w0 + i), g1 = load_f<V>(a.w1 + i);
#pragma unroll
          for (int k = 0; k < V; ++k) y.v[k] = y.v[k] * n0 * g0.v[k] + p1.v[k] * n1 * g1.v[k];
        }
        if (a.scale != nullptr) {
          const Pack<V> ls = load_f<V>(a.scale + i);
#pragma unroll
          for (int k = 0; k < V; ++k) y.v[k] *= ls.v[k];
        }
#pragma unroll
        for (int t = 0; t < SM; ++t) {
          if (t >= S) continue;
          Pack<V> z;
#pragma unroll
          for (int k = 0; k < V; ++k) {
            float acc = wout[t] * y.v[k];
#pragma unroll
            for (int s = 0; s < SM; ++s) acc += mix[s * SM + t] * x[s].v[k];
            z.v[k] = acc;
            u.v[k] += win[t] * acc;
          }
          store_f<V>(xr + static_cast<int64_t>(t) * d + i, z);
        }
      } else {
#pragma unroll
        for (int s = 0; s < SM; ++s)
#pragma unroll
          for (int k = 0; k < V; ++k) u.v[k] += win[s] * x[s].v[k];
      }
#pragma unroll
      for (int k = 0; k < V; ++k) ss += u.v[k] * u.v[k];
      store_f<V>(u_row + i, u);
    }
  }
  if (a.h == nullptr) return;
  const float inv = rsqrtf(cta_sum(ss, scratch) / static_cast<float>(d) + a.eps);
  T* h = static_cast<T*>(a.h) + row * d;
  for (int i = first; i < d; i += step) {
    const Pack<V> u = load_f<V>(u_row + i), w = load_f<V>(a.norm_w + i);
    Pack<V> r;
#pragma unroll
    for (int k = 0; k < V; ++k) r.v[k] = u.v[k] * inv * (w.v[k] + a.plus_one);
    store_t<T, V>(h + i, r);
  }
}

// The same boundary when a row is one Pack of four channels per thread (d / 4 threads): every load of the row is
// issued before the first reduction and nothing is read twice.
template <typename T, int SC>
__global__ void __launch_bounds__(1024, 1) stream_update_row_kernel(const StreamArgs a) {
  constexpr int V = 4;
  __shared__ float2 scratch[2][32];
  const int d = a.d, i = threadIdx.x * V, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int64_t row = blockIdx.x;
  float* xr = a.x + row * SC * d + i;
  auto sum2 = [&](float p, float q, int use) {           // CTA sums of two values; `use` picks the scratch row
    p = warp_sum(p);
    q = warp_sum(q);
    if (lane == 0) scratch[use][warp] = make_float2(p, q);
    __syncthreads();
    float2 t = lane < warps ? scratch[use][lane] : make_float2(0.f, 0.f);
    return make_float2(warp_sum(t.x), warp_sum(t.y));
  };
  Pack<V> x[SC];
#pragma unroll
  for (int s = 0; s < SC; ++s) x[s] = load_f<V>(xr + static_cast<int64_t>(s) * d);
  Pack<V> y = load_t<T, V>(static_cast<const T*>(a.y0) + row * d + i);
  const Pack<V> nw = load_f<V>(a.norm_w + i);
  Pack<V> ls;
#pragma unroll
  for (int k = 0; k < V; ++k) ls.v[k] = 1.f;
  if (a.scale != nullptr) ls = load_f<V>(a.scale + i);
  if (a.y1 != nullptr) {
    const Pack<V> y1 = load_t<T, V>(static_cast<const T*>(a.y1) + row * d + i);
    const Pack<V> g0 = load_f<V>(a.w0 + i), g1 = load_f<V>(a.w1 + i);
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int k = 0; k < V; ++k) {
      s0 += y.v[k] * y.v[k];
      s1 += y1.v[k] * y1.v[k];
    }
    const float2 t = sum2(s0, s1, 0);
    const float n0 = 0.5f * rsqrtf(t.x / static_cast<float>(d) + a.join_eps);
    const float n1 = 0.5f * rsqrtf(t.y / static_cast<float>(d) + a.join_eps);
#pragma unroll
    for (int k = 0; k < V; ++k) y.v[k] = y.v[k] * n0 * g0.v[k] + y1.v[k] * n1 * g1.v[k];
  }
  Pack<V> u;
#pragma unroll
  for (int k = 0; k < V; ++k) {
    y.v[k] *= ls.v[k];
    u.v[k] = 0.f;
  }
#pragma unroll
  for (int t = 0; t < SC; ++t) {
    const float wo = __ldg(a.out + t), wi = a.in ? __ldg(a.in + t) : 1.f;
    Pack<V> z;
#pragma unroll
    for (int k = 0; k < V; ++k) z.v[k] = wo * y.v[k];
#pragma unroll
    for (int s = 0; s < SC; ++s) {
      const float m = __ldg(a.mix + s * SC + t);
#pragma unroll
      for (int k = 0; k < V; ++k) z.v[k] += m * x[s].v[k];
    }
#pragma unroll
    for (int k = 0; k < V; ++k) u.v[k] += wi * z.v[k];
    store_f<V>(xr + static_cast<int64_t>(t) * d, z);
  }
  if (a.h == nullptr) return;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < V; ++k) ss += u.v[k] * u.v[k];
  const float inv = rsqrtf(sum2(ss, 0.f, 1).x / static_cast<float>(d) + a.eps);
#pragma unroll
  for (int k = 0; k < V; ++k) u.v[k] = u.v[k] * inv * (nw.v[k] + a.plus_one);
  store_t<T, V>(static_cast<T*>(a.h) + row * d + i, u);
}

template <typename T>
int launch_stream_rows(const StreamArgs& a, int64_t rows, cudaStream_t s) {
  auto kern = stream_update_row_kernel<T, 1>;
  if (a.S == 2) kern = stream_update_row_kernel<T, 2>;
  if (a.S == 3) kern = stream_update_row_kernel<T, 3>;
  if (a.S == 4) kern = stream_update_row_kernel<T, 4>;
  kern<<<static_cast<unsigned>(rows), a.d / 4, 0, s>>>(a);
  return launch_result();
}

template <typename T, int V>
int launch_streams(const StreamArgs& a, int64_t rows, cudaStream_t s) {
  if (V == 4 && a.S <= 4 && a.y0 != nullptr && a.norm_w != nullptr && a.d % 128 == 0 && a.d <= 4096)
    return launch_stream_rows<T>(a, rows, s);
  const size_t smem = static_cast<size_t>(a.d) * sizeof(float);
  int threads = (a.d / V + 31) / 32 * 32;
  threads = threads < 64 ? 64 : threads > 512 ? 512 : threads;
  auto kern = stream_update_kernel<T, V, 0>;
  switch (a.S) {
    case 1: kern = stream_update_kernel<T, V, 1>; break;
    case 2: kern = stream_update_kernel<T, V, 2>; break;
    case 3: kern = stream_update_kernel<T, V, 3>; break;
    case 4: kern = stream_update_kernel<T, V, 4>; break;
    default: break;
  }
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem)) != cudaSuccess)
    return B200_ERR_LAUNCH;
  kern<<<static_cast<unsigned>(rows), threads, smem, s>>>(a);
  return launch_result();
}

// ---------------------------------------------------------------------------------------------
// Clamped gated linear unit: act = g sigmoid(slope g) (u + 1), g = min(gate, limit), u = clamp(up, +-limit).
// ---------------------------------------------------------------------------------------------
template <typename T, int V>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const T* __restrict__ h, T* __restrict__ act, int64_t total,
                                                          int F, float limit, float slope) {
  // one unit = V consecutive channels of one row
  const int per_row = F / V;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t row = i / per_row;
    const int c = static_cast<int>(i - row * per_row) * V;
    const T* g = h + row * 2 * F + c;
    T* o = act + row * F + c;
    if constexpr (V == 8) {
      const uint4 ga = *reinterpret_cast<const uint4*>(g), ua = *reinterpret_cast<const uint4*>(g + F);
      const uint32_t gw[4] = {ga.x, ga.y, ga.z, ga.w}, uw[4] = {ua.x, ua.y, ua.z, ua.w};
      uint32_t r[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 gf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[k]));
        const float2 uf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&uw[k]));
        r[k] = pack_bf16x2(clamped_glu_f(gf.x, uf.x, limit, slope), clamped_glu_f(gf.y, uf.y, limit, slope));
      }
      *reinterpret_cast<uint4*>(o) = make_uint4(r[0], r[1], r[2], r[3]);
    } else {
      *o = from_float<T>(clamped_glu_f(to_float<T>(g[0]), to_float<T>(g[F]), limit, slope));
    }
  }
}

}  // namespace
}  // namespace b200

extern "C" int b200_stream_update(float* x, const int64_t* tokens, const void* embed, int64_t vocab, const void* y0,
                                  const void* y1, const float* join_w0, const float* join_w1, float join_eps,
                                  const float* layer_scale, const float* mix, const float* out_w, const float* in_w,
                                  const float* norm_w, int32_t norm_plus_one, float eps, void* h, int64_t rows,
                                  int32_t streams, int32_t dim, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (rows < 0 || streams <= 0 || dim <= 0) return B200_ERR_ARG;
  if (streams > kMaxStreams || (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16)) return B200_ERR_UNSUPPORTED;
  if (static_cast<size_t>(dim) * sizeof(float) > 200 * 1024 || rows > 2147483647LL) return B200_ERR_TOO_LARGE;
  if (rows == 0) return B200_OK;
  if (!x || (embed && !tokens) || (embed && y0) || (y1 && !(y0 && join_w0 && join_w1)) || (y0 && !(mix && out_w)) ||
      (h && !norm_w))
    return B200_ERR_ARG;
  StreamArgs a{x, tokens, embed, vocab, y0, y1, join_w0, join_w1, join_eps, layer_scale, mix, out_w, in_w, norm_w,
               norm_plus_one ? 1.f : 0.f, eps, h, streams, dim, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto al = [](const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const size_t ts = dtype == B200_DTYPE_F32 ? 16 : 8;
  const bool vec = dim % 4 == 0 && al(x, 16) && al(embed, ts) && al(y0, ts) && al(y1, ts) && al(h, ts) &&
                   al(join_w0, 16) && al(join_w1, 16) && al(layer_scale, 16) && al(norm_w, 16);
  if (dtype == B200_DTYPE_F32)
    return vec ? launch_streams<float, 4>(a, rows, s) : launch_streams<float, 1>(a, rows, s);
  return vec ? launch_streams<__nv_bfloat16, 4>(a, rows, s) : launch_streams<__nv_bfloat16, 1>(a, rows, s);
}

extern "C" int b200_clamped_glu(const void* h, void* act, int64_t rows, int32_t d_ff, float limit, float slope,
                                int32_t dtype, void* stream) {
  using namespace b200;
  if (rows < 0 || d_ff <= 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (!h || !act) return B200_ERR_ARG;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int sms = sm_count_cached();
  if (sms <= 0) return B200_ERR_NO_DEVICE;
  const bool vec = dtype == B200_DTYPE_BF16 && d_ff % 8 == 0 && aligned16(h) && aligned16(act);
  const int64_t total = vec ? rows * (d_ff / 8) : rows * d_ff;
  int64_t grid = (total + 255) / 256;
  if (grid > int64_t(sms) * 16) grid = int64_t(sms) * 16;
  const unsigned g = static_cast<unsigned>(grid);
  if (vec)
    clamped_glu_kernel<__nv_bfloat16, 8><<<g, 256, 0, s>>>(static_cast<const __nv_bfloat16*>(h),
                                                           static_cast<__nv_bfloat16*>(act), total, d_ff, limit, slope);
  else if (dtype == B200_DTYPE_BF16)
    clamped_glu_kernel<__nv_bfloat16, 1><<<g, 256, 0, s>>>(static_cast<const __nv_bfloat16*>(h),
                                                           static_cast<__nv_bfloat16*>(act), total, d_ff, limit, slope);
  else
    clamped_glu_kernel<float, 1><<<g, 256, 0, s>>>(static_cast<const float*>(h), static_cast<float*>(act), total, d_ff,
                                                   limit, slope);
  return launch_result();
}
