// Gated delta rule over per-sequence states.  Per value head h with key head floor(h / (H / G)):
//
//   q, k, v   projections behind a short causal convolution per channel and silu
//   q^ = q / sqrt(sum q^2 + 1e-6) dk^-1/2,  k^ = k / sqrt(sum k^2 + 1e-6)
//   beta = sigmoid(b),  g = exp(-exp(A) softplus(a + dt))
//   S <- g S,  u = beta (v - S^T k^),  S <- S + k^ u^T,  o = S^T q^
//   out = o / sqrt(mean(o^2) + eps) norm_w silu(gate)
//
// q, k, v behind the activation are in the activation dtype, everything after that is fp32.  The state S [dk, dv] of every
// (slot, head) and the convolution's last inputs live in fp32 pools.  The inputs are kept as a ring, position p in row
// p mod taps: a step reads the rows of the positions before it and writes its own, which nobody reads in that step, so
// the CTAs of heads that share a key head need no order among themselves.  A sequence whose first token of the call is at
// position 0 starts from zero whatever its slot holds.
//
// delta_conv_kernel    convolution + silu of prompts and portions
// delta_serial_kernel  one CTA per (sequence, value head), tokens in order: decode (with the convolution in front), fp32, and
//                      sizes the chunked kernels (delta_chunk.cu) do not take.  One pass over the state yields both S^T k^
//                      and S^T q^: with k^, q^ as they are, o = g S^T q^ + (k^ . q^) u.
// delta_step_kernel    the same for one token per sequence and heads of 64 or 128 channels
#include "delta_common.cuh"

namespace b200 {
namespace {

// ---------------------------------------------------------------------------------------------
// convolution of prompts
// ---------------------------------------------------------------------------------------------
constexpr int kConvTokens = 32, kConvThreads = 128;

struct ConvArgs {
  const void* x;             // [T, C], token stride
  int64_t stride;
  const float* w;            // [taps, C], the last row weighs the current token
  float* ring;               // [slots, taps, C]
  const int64_t* slots;
  int64_t num_slots;
  const int32_t* cu_q;
  const int32_t* cu_k;
  const int64_t* ctx_lens;   // null
  void* out;                 // [T, C]
  int C, taps, n;
  int32_t* status;
};

template <typename T>
__device__ __forceinline__ float4 load4(const T* p) {
  if constexpr (sizeof(T) == 2) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
  } else {
    return *reinterpret_cast<const float4*>(p);
  }
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v) {
  if constexpr (sizeof(T) == 2)
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  else
    *reinterpret_cast<float4*>(p) = v;
}
__device__ __forceinline__ void fma4(float4& acc, float4 w, float4 x) {
  acc.x += w.x * x.x;
  acc.y += w.y * x.y;
  acc.z += w.z * x.z;
  acc.w += w.w * x.w;
}

// A thread takes four channels through a segment of a sequence.  TAPS > 0: the inputs before the current one stay in
// registers; 0: any number of taps, read again for every token.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads) delta_conv_kernel(const ConvArgs a) {
  int seq, index;
  if (!find_segment(a.cu_q, a.n, kConvTokens, blockIdx.x, &seq, &index)) return;
  SeqInfo info;
  if (!sequence_info(a, seq, &info)) return;
  const int c = (blockIdx.y * kConvThreads + threadIdx.x) * 4;
  if (c >= a.C) return;
  const int taps = TAPS > 0 ? TAPS : a.taps;
  const int lo = index * kConvTokens, nt = min(kConvTokens, info.len - lo);
  const T* x = static_cast<const T*>(a.x) + info.tok0 * a.stride + c;
  float* ring = a.ring + info.slot * taps * a.C + c;
  T* out = static_cast<T*>(a.out) + info.tok0 * a.C + c;
  // input of token t of the portion, also before its start and before position 0
  auto input = [&](int t) -> float4 {
    if (t >= 0) return load4<T>(x + static_cast<int64_t>(t) * a.stride);
    const int64_t p = info.pos0 + t;
    if (p < 0) return make_float4(0.f, 0.f, 0.f, 0.f);
    return *reinterpret_cast<const float4*>(ring + (p % taps) * a.C);
  };
  if constexpr (TAPS > 0) {
    float4 w[TAPS], h[TAPS];       // h[m]: input TAPS - 1 - m tokens back
#pragma unroll
    for (int m = 0; m < TAPS; ++m) {
      w[m] = *reinterpret_cast<const float4*>(a.w + static_cast<int64_t>(m) * a.C + c);
      if (m > 0) h[m] = input(lo - TAPS + m);
    }
    constexpr int B = 8;           // loads in flight
    float4 x8[B];
    for (int t0 = lo; t0 < lo + nt; t0 += B) {
#pragma unroll
      for (int u = 0; u < B; ++u) x8[u] = load4<T>(x + static_cast<int64_t>(min(t0 + u, lo + nt - 1)) * a.stride);
#pragma unroll
      for (int u = 0; u < B; ++u) {
        const int t = t0 + u;
        if (t >= lo + nt) break;
#pragma unroll
        for (int m = 0; m + 1 < TAPS; ++m) h[m] = h[m + 1];
        h[TAPS - 1] = x8[u];
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int m = 0; m < TAPS; ++m) fma4(y, w[m], h[m]);
        store4<T>(out + static_cast<int64_t>(t) * a.C, make_float4(silu_for<T>(y.x), silu_for<T>(y.y), silu_for<T>(y.z), silu_for<T>(y.w)));
      }
    }
  } else {
    for (int t = lo; t < lo + nt; ++t) {
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int m = 0; m < taps; ++m)
        fma4(y, *reinterpret_cast<const float4*>(a.w + static_cast<int64_t>(m) * a.C + c), input(t - (taps - 1) + m));
      store4<T>(out + static_cast<int64_t>(t) * a.C, make_float4(silu_for<T>(y.x), silu_for<T>(y.y), silu_for<T>(y.z), silu_for<T>(y.w)));
    }
  }
  // The thread that has read the ring is the one that moves it on: the last taps - 1 inputs of the portion.
  if (index == 0)
    for (int m = 0; m < min(taps - 1, info.len); ++m) {
      const int t = info.len - 1 - m;
      *reinterpret_cast<float4*>(ring + ((info.pos0 + t) % taps) * a.C) = load4<T>(x + static_cast<int64_t>(t) * a.stride);
    }
}

// ---------------------------------------------------------------------------------------------
// tokens in order
// ---------------------------------------------------------------------------------------------

// Threads are RG row groups x CL column units of V columns.  R > 0: a thread keeps its rows rg, rg + RG, ... of a column
// unit in registers (R * RG >= dk); R == 0: the state is read twice.  CONV: one token per sequence, convolution first.
template <typename T, bool CONV, int V, int R>
__global__ void __launch_bounds__(512) delta_serial_kernel(const DeltaArgs a, int CL) {
  extern __shared__ float sm[];
  const int dk = a.dk, dv = a.dv, head = blockIdx.x, kh = head / (a.H / a.G), NT = blockDim.x;
  const int RG = NT / CL, cu = threadIdx.x % CL, rg = threadIdx.x / CL, lane = threadIdx.x & 31;
  float* sq = sm;                 // [dk]
  float* sk = sq + dk;            // [dk]
  float* sv = sk + dk;            // [dv]
  float* su = sv + dv;            // [dv] the write u
  float* so = su + dv;            // [dv]
  float* red = so + dv;           // [2][RG][CL * V]
  SeqInfo info;
  if (!sequence_info(a, blockIdx.y, &info)) return;
  const int units = (dv + V - 1) / V, W = CL * V;
  const bool resident = R > 0 && units <= CL;        // the state stays in registers between tokens
  float* S = a.state + (info.slot * a.H + head) * static_cast<int64_t>(dk) * dv;
  float* ring = CONV ? a.conv_ring + info.slot * a.taps * a.conv_width : nullptr;
  const int ring0 = CONV ? static_cast<int>(info.pos0 % a.taps) : 0;      // ring row of the current position
  const float scale = rsqrtf(static_cast<float>(dk));
  float s[R > 0 ? R : 1][V];
  auto load_state = [&](int c, bool zero) {
    if constexpr (R > 0) {
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int r = rg + i * RG;
        const float* sp = S + static_cast<int64_t>(r) * dv + c * V;
        if constexpr (V == 4) {
          const float4 x = zero || r >= dk ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(sp);
          s[i][0] = x.x, s[i][1] = x.y, s[i][2] = x.z, s[i][3] = x.w;
        } else {
          s[i][0] = zero || r >= dk ? 0.f : *sp;
        }
      }
    }
  };
  if (cu < units) load_state(cu, info.fresh);        // in flight while the inputs are gathered
  const float dt_bias = a.dt_bias[head], a_log = a.a_log[head];
  const float my_norm = threadIdx.x < dv ? a.norm_w[threadIdx.x] : 0.f;
  for (int t = 0; t < (CONV ? 1 : info.len); ++t) {
    const int64_t tok = info.tok0 + t, prow = tok * a.proj_stride + head;
    const T* gp = static_cast<const T*>(a.gate) + tok * a.proj_stride + head * dv;
    const T raw_b = static_cast<const T*>(a.b)[prow], raw_a = static_cast<const T*>(a.a)[prow];
    const T my_gate = threadIdx.x < dv ? gp[threadIdx.x] : from_float<T>(0.f);
    const T* qp = static_cast<const T*>(a.q) + tok * a.act_stride + kh * dk;
    const T* kp = static_cast<const T*>(a.k) + tok * a.act_stride + kh * dk;
    const T* vp = static_cast<const T*>(a.v) + tok * a.act_stride + head * dv;
    for (int i = threadIdx.x; i < 2 * dk + dv; i += NT) {
      const bool is_q = i < dk, is_k = !is_q && i < 2 * dk;
      const int j = is_q ? i : is_k ? i - dk : i - 2 * dk;
      float x = to_float<T>((is_q ? qp : is_k ? kp : vp)[j]);
      if constexpr (CONV) {
        const int col = (is_q ? a.col_q + kh * dk : is_k ? a.col_k + kh * dk : a.col_v + head * dv) + j;
        float y = a.conv_w[(a.taps - 1) * a.conv_width + col] * x;
        float* rc = ring + col;
        for (int m = 1; m < a.taps; ++m)
          if (m <= info.pos0)
            y += a.conv_w[(a.taps - 1 - m) * a.conv_width + col] * rc[(ring0 >= m ? ring0 - m : ring0 - m + a.taps) * a.conv_width];
        rc[ring0 * a.conv_width] = x;
        x = to_float<T>(from_float<T>(silu_for<T>(y)));
      }
      sm[i] = x;                  // q | k | v
    }
    __syncthreads();
    // norms and k^ . q^: every warp for itself
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int i = lane; i < dk; i += 32) {
      const float x = sq[i], y = sk[i];
      qq += x * x;
      kk += y * y;
      kq += x * y;
    }
    const float rq = rsqrtf(warp_sum(qq) + 1e-6f) * scale, rk = rsqrtf(warp_sum(kk) + 1e-6f);
    kq = warp_sum(kq) * rq * rk;
    const float beta = sigmoid_f(to_float<T>(raw_b));
    const float g = expf(log_decay(to_float<T>(raw_a) + dt_bias, a_log));
    const bool zero = info.fresh && t == 0;
    for (int c0 = 0; c0 < units; c0 += CL) {
      const int c = c0 + cu;
      float pk[V], pq[V];
#pragma unroll
      for (int e = 0; e < V; ++e) pk[e] = pq[e] = 0.f;
      if (c < units) {
        if constexpr (R > 0) {
          if (t > 0 ? !resident : c0 > 0) load_state(c, zero);
#pragma unroll
          for (int i = 0; i < R; ++i) {
            const int r = rg + i * RG;
            const float x = r < dk ? sk[r] : 0.f, y = r < dk ? sq[r] : 0.f;
#pragma unroll
            for (int e = 0; e < V; ++e) {
              pk[e] += s[i][e] * x;
              pq[e] += s[i][e] * y;
            }
          }
        } else if (!zero) {
          for (int r = rg; r < dk; r += RG) {
            const float x = sk[r], y = sq[r];
#pragma unroll
            for (int e = 0; e < V; ++e) {
              const float v = S[static_cast<int64_t>(r) * dv + c * V + e];
              pk[e] += v * x;
              pq[e] += v * y;
            }
          }
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) {
        red[rg * W + cu * V + e] = pk[e];
        red[(RG + rg) * W + cu * V + e] = pq[e];
      }
      __syncthreads();
      const int cols = min(W, dv - c0 * V);
      for (int i = threadIdx.x; i < cols; i += NT) {
        float xk = 0.f, xq = 0.f;
        for (int r = 0; r < RG; ++r) {
          xk += red[r * W + i];
          xq += red[(RG + r) * W + i];
        }
        const float u = beta * (sv[c0 * V + i] - g * rk * xk);
        su[c0 * V + i] = u;
        so[c0 * V + i] = g * rq * xq + kq * u;
      }
      __syncthreads();
      if (c < units) {
        float u[V];
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = su[c * V + e] * rk;
        const bool store = !resident || t == info.len - 1;
        if constexpr (R > 0) {
#pragma unroll
          for (int i = 0; i < R; ++i) {
            const int r = rg + i * RG;
            if (r >= dk) continue;
            const float x = sk[r];
            float* sp = S + static_cast<int64_t>(r) * dv + c * V;
#pragma unroll
            for (int e = 0; e < V; ++e) s[i][e] = g * s[i][e] + x * u[e];
            if (store) {
              if constexpr (V == 4) *reinterpret_cast<float4*>(sp) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
              else *sp = s[i][0];
            }
          }
        } else {
          for (int r = rg; r < dk; r += RG) {
            float* sp = S + static_cast<int64_t>(r) * dv + c * V;
#pragma unroll
            for (int e = 0; e < V; ++e) sp[e] = g * (zero ? 0.f : sp[e]) + sk[r] * u[e];
          }
        }
      }
    }
    float ss = 0.f;
    for (int i = lane; i < dv; i += 32) ss += so[i] * so[i];
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(dv) + a.eps);
    T* op = static_cast<T*>(a.out) + (tok * a.H + head) * dv;
    if (threadIdx.x < dv) op[threadIdx.x] = from_float<T>(so[threadIdx.x] * inv * my_norm * silu_for<T>(to_float<T>(my_gate)));
    for (int i = threadIdx.x + NT; i < dv; i += NT) op[i] = from_float<T>(so[i] * inv * a.norm_w[i] * silu_for<T>(to_float<T>(gp[i])));
    if (!CONV) __syncthreads();
  }
}

template <typename T, bool CONV, int V, int R>
int launch_serial(const DeltaArgs& a, int threads, int CL, cudaStream_t s) {
  const size_t smem = (2 * static_cast<size_t>(a.dk) + 3 * static_cast<size_t>(a.dv) + 2 * static_cast<size_t>(threads) * V) *
                      sizeof(float);
  auto kern = delta_serial_kernel<T, CONV, V, R>;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem)) != cudaSuccess)
    return B200_ERR_LAUNCH;
  kern<<<dim3(a.H, a.n), threads, smem, s>>>(a, CL);
  return launch_result();
}

template <typename T, bool CONV>
int dispatch_serial(const DeltaArgs& a, cudaStream_t s) {
  const bool vec = a.dv % 4 == 0 && aligned16(a.state);
  int threads = 256, CL = 4;
  const int units = vec ? a.dv / 4 : a.dv;
  while (CL < units && CL < threads) CL *= 2;
  if (!vec) return launch_serial<T, CONV, 1, 0>(a, threads, CL, s);
  int rows = (a.dk + threads / CL - 1) / (threads / CL);
  if (rows > 16) {
    threads = 512;
    rows = (a.dk + threads / CL - 1) / (threads / CL);
  }
  if (rows <= 4) return launch_serial<T, CONV, 4, 4>(a, threads, CL, s);
  if (rows <= 8) return launch_serial<T, CONV, 4, 8>(a, threads, CL, s);
  if (rows <= 16) return launch_serial<T, CONV, 4, 16>(a, threads, CL, s);
  return launch_serial<T, CONV, 4, 0>(a, threads, CL, s);
}

// ---------------------------------------------------------------------------------------------
// One token per sequence, sizes that fill the CTA: dv = 4 CL, dk = R RG, CL * RG threads.  A thread holds R rows x 4
// columns of the state as packed pairs; every load of the state is issued before anything else happens.
// ---------------------------------------------------------------------------------------------
// Three CTAs per SM for the 64 KB states: a few spilled registers cost less than the third state in flight gains (256
// sequences x 32 heads: 244 against 285 us).
template <typename T, int CL, int RG, int R>
__global__ void __launch_bounds__(CL * RG, CL * RG == 256 && R == 16 ? 3 : 1) delta_step_kernel(const DeltaArgs a) {
  constexpr int NT = CL * RG, DK = R * RG, DV = 4 * CL;
  __shared__ float raw[2 * DK + DV];               // q | k | v behind the activation
  __shared__ ulonglong2 kq[DK];                    // {k, k}, {q, q} per row: packed operands
  __shared__ float4 red[2][RG][CL];
  __shared__ float su[DV], so[DV], gates[2];       // write, output; decay and write strength
  const int head = blockIdx.x, seq = blockIdx.y, kh = head / (a.H / a.G);
  const int tid = threadIdx.x, lane = tid & 31, cu = tid % CL, rg = tid / CL;
  SeqInfo info;
  if (!sequence_info(a, seq, &info)) return;
  float* S = a.state + (info.slot * a.H + head) * static_cast<int64_t>(DK * DV) + rg * DV + cu * 4;
  f32x2 s[R][2];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const ulonglong2 x = info.fresh ? make_ulonglong2(0ull, 0ull) : *reinterpret_cast<const ulonglong2*>(S + i * RG * DV);
    s[i][0] = x.x;
    s[i][1] = x.y;
  }
  const int64_t tok = info.tok0, prow = tok * a.proj_stride + head;
  const T my_gate = tid < DV ? static_cast<const T*>(a.gate)[tok * a.proj_stride + head * DV + tid] : from_float<T>(0.f);
  const float my_norm = tid < DV ? a.norm_w[tid] : 0.f;
  const int ring0 = static_cast<int>(info.pos0 % a.taps);
  float* ring = a.conv_ring + info.slot * a.taps * a.conv_width;
  for (int i = tid; i < 2 * DK + DV; i += NT) {
    const bool is_q = i < DK, is_k = !is_q && i < 2 * DK;
    const int at = is_q ? kh * DK + i : is_k ? kh * DK + i - DK : head * DV + i - 2 * DK;
    const int col = (is_q ? a.col_q : is_k ? a.col_k : a.col_v) + at;
    const float x = to_float<T>(static_cast<const T*>(is_q ? a.q : is_k ? a.k : a.v)[tok * a.act_stride + at]);
    float y = a.conv_w[(a.taps - 1) * a.conv_width + col] * x;
    for (int m = 1; m < a.taps; ++m)
      if (m <= info.pos0)
        y += a.conv_w[(a.taps - 1 - m) * a.conv_width + col] * ring[(ring0 >= m ? ring0 - m : ring0 - m + a.taps) * a.conv_width + col];
    ring[ring0 * a.conv_width + col] = x;
    raw[i] = to_float<T>(from_float<T>(silu_for<T>(y)));
  }
  if (tid == NT - 1) {
    gates[0] = expf(log_decay(to_float<T>(static_cast<const T*>(a.a)[prow]) + a.dt_bias[head], a.a_log[head]));
    gates[1] = sigmoid_f(to_float<T>(static_cast<const T*>(a.b)[prow]));
  }
  __syncthreads();
  float qq = 0.f, kk = 0.f, dot = 0.f;             // every warp for itself
#pragma unroll
  for (int i = 0; i < DK / 32; ++i) {
    const float x = raw[i * 32 + lane], y = raw[DK + i * 32 + lane];
    qq += x * x;
    kk += y * y;
    dot += x * y;
  }
  const float rq = rsqrtf(warp_sum(qq) + 1e-6f) * rsqrtf(static_cast<float>(DK)), rk = rsqrtf(warp_sum(kk) + 1e-6f);
  dot = warp_sum(dot) * rq * rk;
  for (int i = tid; i < DK; i += NT) {
    const float k = raw[DK + i] * rk, q = raw[i] * rq;
    kq[i] = make_ulonglong2(pack2(k, k), pack2(q, q));
  }
  __syncthreads();
  {
    f32x2 pk[2] = {0ull, 0ull}, pq[2] = {0ull, 0ull};
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const ulonglong2 x = kq[rg + i * RG];
      pk[0] = fma2(s[i][0], x.x, pk[0]);
      pk[1] = fma2(s[i][1], x.x, pk[1]);
      pq[0] = fma2(s[i][0], x.y, pq[0]);
      pq[1] = fma2(s[i][1], x.y, pq[1]);
    }
    *reinterpret_cast<ulonglong2*>(&red[0][rg][cu]) = make_ulonglong2(pk[0], pk[1]);
    *reinterpret_cast<ulonglong2*>(&red[1][rg][cu]) = make_ulonglong2(pq[0], pq[1]);
  }
  __syncthreads();
  const float g = gates[0], beta = gates[1];
  for (int i = tid; i < DV; i += NT) {
    float xk = 0.f, xq = 0.f;
#pragma unroll
    for (int r = 0; r < RG; ++r) {
      xk += reinterpret_cast<const float*>(&red[0][r][0])[i];
      xq += reinterpret_cast<const float*>(&red[1][r][0])[i];
    }
    const float u = beta * (raw[2 * DK + i] - g * xk);
    su[i] = u;
    so[i] = g * xq + dot * u;
  }
  __syncthreads();
  {
    const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(su + cu * 4);
    const f32x2 g2 = pack2(g, g);
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const f32x2 k2 = kq[rg + i * RG].x;
      *reinterpret_cast<ulonglong2*>(S + i * RG * DV) =
          make_ulonglong2(fma2(g2, s[i][0], mul2(k2, u.x)), fma2(g2, s[i][1], mul2(k2, u.y)));
    }
  }
  if (tid < DV) {                                  // whole warps
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < DV / 32; ++i) ss += so[i * 32 + lane] * so[i * 32 + lane];
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(DV) + a.eps);
    static_cast<T*>(a.out)[(tok * a.H + head) * DV + tid] =
        from_float<T>(so[tid] * inv * my_norm * silu_for<T>(to_float<T>(my_gate)));
  }
}

// B200_ERR_UNSUPPORTED for other sizes
template <typename T>
int launch_step(const DeltaArgs& a, cudaStream_t s) {
  if (!aligned16(a.state)) return B200_ERR_UNSUPPORTED;
  const dim3 grid(a.H, a.n);
  if (a.dk == 128 && a.dv == 128) delta_step_kernel<T, 32, 8, 16><<<grid, 256, 0, s>>>(a);
  else if (a.dk == 64 && a.dv == 128) delta_step_kernel<T, 32, 8, 8><<<grid, 256, 0, s>>>(a);
  else if (a.dk == 128 && a.dv == 64) delta_step_kernel<T, 16, 8, 16><<<grid, 128, 0, s>>>(a);
  else if (a.dk == 64 && a.dv == 64) delta_step_kernel<T, 16, 8, 8><<<grid, 128, 0, s>>>(a);
  else return B200_ERR_UNSUPPORTED;
  return launch_result();
}

bool delta_args_ok(const DeltaArgs& a) {
  return a.n >= 0 && a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.dk > 0 && a.dv > 0 && a.num_slots >= 0;
}
bool delta_pointers_ok(const DeltaArgs& a) {
  return a.q && a.k && a.v && a.b && a.a && a.gate && a.dt_bias && a.a_log && a.norm_w && a.state && a.slots && a.out;
}

}  // namespace
}  // namespace b200

extern "C" int b200_delta_conv(const void* x, int64_t token_stride, const float* weights, int32_t taps, int32_t width,
                               float* ring, int64_t num_slots, const int64_t* state_slots, const int32_t* cu_seqlens_q,
                               const int32_t* cu_seqlens_k, int32_t num_seqs, int64_t total_tokens, void* out,
                               int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (num_seqs < 0 || taps <= 0 || width <= 0 || num_slots < 0 || total_tokens < 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_seqs == 0 || total_tokens == 0) return B200_OK;
  if (!x || !weights || !ring || !state_slots || !cu_seqlens_q || !cu_seqlens_k || !out) return B200_ERR_ARG;
  if (width % 4 || token_stride % 4 || !aligned16(x) || !aligned16(weights) || !aligned16(ring) || !aligned16(out))
    return B200_ERR_ALIGN;
  ConvArgs a{x, token_stride, weights, ring, state_slots, num_slots, cu_seqlens_q, cu_seqlens_k, nullptr, out, width, taps,
             num_seqs, status};
  const dim3 grid(static_cast<unsigned>(total_tokens / kConvTokens + num_seqs),
                  static_cast<unsigned>((width / 4 + kConvThreads - 1) / kConvThreads));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto go = [&](auto kern) { kern<<<grid, kConvThreads, 0, s>>>(a); };
  if (dtype == B200_DTYPE_F32) {
    if (taps == 4) go(delta_conv_kernel<float, 4>);
    else go(delta_conv_kernel<float, 0>);
  } else {
    if (taps == 4) go(delta_conv_kernel<__nv_bfloat16, 4>);
    else if (taps == 3) go(delta_conv_kernel<__nv_bfloat16, 3>);
    else if (taps == 2) go(delta_conv_kernel<__nv_bfloat16, 2>);
    else go(delta_conv_kernel<__nv_bfloat16, 0>);
  }
  return launch_result();
}

extern "C" size_t b200_delta_rule_workspace_bytes(int32_t num_seqs, int64_t total_tokens, int32_t num_heads, int32_t dim_k,
                                                  int32_t dim_v, int32_t dtype) {
  using namespace b200;
  if (num_seqs <= 0 || total_tokens <= 0 || num_heads <= 0 || dtype != B200_DTYPE_BF16 || !delta_chunk_shape(dim_k, dim_v))
    return 0;
  return delta_chunk_workspace(num_seqs, total_tokens, num_heads);
}

extern "C" int b200_delta_rule(const void* q, const void* k, const void* v, int64_t act_stride, const void* b, const void* a_in,
                               const void* gate, int64_t proj_stride, const float* dt_bias, const float* a_log,
                               const float* norm_w, float eps, float* state, int64_t num_slots, const int64_t* state_slots,
                               const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, int32_t num_seqs,
                               int64_t total_tokens, int32_t num_heads, int32_t num_k_heads, int32_t dim_k, int32_t dim_v,
                               void* out, void* workspace, size_t workspace_bytes, int32_t dtype, int32_t* status,
                               void* stream) {
  using namespace b200;
  DeltaArgs a{};
  a.q = q, a.k = k, a.v = v, a.act_stride = act_stride, a.b = b, a.a = a_in, a.gate = gate, a.proj_stride = proj_stride;
  a.dt_bias = dt_bias, a.a_log = a_log, a.norm_w = norm_w, a.eps = eps, a.state = state, a.slots = state_slots;
  a.num_slots = num_slots, a.cu_q = cu_seqlens_q, a.cu_k = cu_seqlens_k, a.out = out, a.n = num_seqs, a.H = num_heads;
  a.G = num_k_heads, a.dk = dim_k, a.dv = dim_v, a.status = status;
  if (!delta_args_ok(a) || total_tokens < 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_seqs == 0 || total_tokens == 0) return B200_OK;
  if (!delta_pointers_ok(a) || !cu_seqlens_q || !cu_seqlens_k) return B200_ERR_ARG;
  if (num_seqs > 65535 || dim_k > 2048 || dim_v > 2048) return B200_ERR_UNSUPPORTED;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_BF16 && workspace && delta_chunk_shape(dim_k, dim_v) && act_stride % 8 == 0 && proj_stride % 4 == 0 &&
      aligned16(q) && aligned16(k) && aligned16(v) && (reinterpret_cast<uintptr_t>(gate) & 7) == 0 && aligned16(out)) {
    if (workspace_bytes < delta_chunk_workspace(num_seqs, total_tokens, num_heads)) return B200_ERR_WORKSPACE;
    return delta_chunk_launch(a, total_tokens, workspace, s);
  }
  return dtype == B200_DTYPE_F32 ? dispatch_serial<float, false>(a, s) : dispatch_serial<__nv_bfloat16, false>(a, s);
}

extern "C" int b200_delta_step(const void* q, const void* k, const void* v, const void* b, const void* a_in, const void* gate,
                               int64_t proj_stride, const float* conv_w, int32_t taps, int32_t conv_width, int32_t col_q,
                               int32_t col_k, int32_t col_v, float* conv_ring, const float* dt_bias, const float* a_log,
                               const float* norm_w, float eps, float* state, int64_t num_slots, const int64_t* state_slots,
                               const int64_t* context_lens, int32_t num_seqs, int32_t num_heads, int32_t num_k_heads,
                               int32_t dim_k, int32_t dim_v, void* out, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  DeltaArgs a{};
  a.q = q, a.k = k, a.v = v, a.act_stride = proj_stride, a.b = b, a.a = a_in, a.gate = gate, a.proj_stride = proj_stride;
  a.dt_bias = dt_bias, a.a_log = a_log, a.norm_w = norm_w, a.eps = eps, a.state = state, a.slots = state_slots;
  a.num_slots = num_slots, a.ctx_lens = context_lens, a.out = out, a.n = num_seqs, a.H = num_heads, a.G = num_k_heads;
  a.dk = dim_k, a.dv = dim_v, a.conv_w = conv_w, a.conv_ring = conv_ring, a.taps = taps, a.conv_width = conv_width;
  a.col_q = col_q, a.col_k = col_k, a.col_v = col_v, a.status = status;
  if (!delta_args_ok(a) || taps <= 0 || conv_width <= 0 || col_q < 0 || col_k < 0 || col_v < 0 ||
      col_q + num_k_heads * dim_k > conv_width || col_k + num_k_heads * dim_k > conv_width ||
      col_v + num_heads * dim_v > conv_width)
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_seqs == 0) return B200_OK;
  if (!delta_pointers_ok(a) || !conv_w || !conv_ring || !context_lens) return B200_ERR_ARG;
  if (num_seqs > 65535 || dim_k > 2048 || dim_v > 2048) return B200_ERR_UNSUPPORTED;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int rc = dtype == B200_DTYPE_F32 ? launch_step<float>(a, s) : launch_step<__nv_bfloat16>(a, s);
  if (rc != B200_ERR_UNSUPPORTED) return rc;
  return dtype == B200_DTYPE_F32 ? dispatch_serial<float, true>(a, s) : dispatch_serial<__nv_bfloat16, true>(a, s);
}
