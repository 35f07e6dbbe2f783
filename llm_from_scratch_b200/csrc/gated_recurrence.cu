// Linear attention with a data-dependent forget gate that also decides what is written (HGRN2):
//
//   q = silu(q_proj), f = lower + (1 - lower) sigmoid(f_proj + f_bias)      per head and key channel
//   S <- diag(f) S + (1 - f) v^T,   o = S^T q,   out = rms(o) * norm_w      per head
//
// The projections arrive in the activation dtype; everything behind them is fp32.  The state S [dk, dv] of
// every (slot, head) lives in a fp32 pool and is carried from call to call; a sequence whose first token of
// the call is at position 0 starts from zero whatever its slot holds, so slots need no clearing when they
// change hands.
//
// recurrence_step_kernel   one CTA per (sequence, head), tokens in order: decode, and short portions.
#include "common.cuh"

namespace b200 {
namespace {

struct RecArgs {
  const void* q;
  const void* f;
  const void* v;
  int64_t stride;            // elements between tokens, the same for q / f / v (views of one projection)
  const float* f_bias;       // [H, dk]
  const float* lower;        // [H, dk]
  const float* norm_w;       // [dv]
  float eps;
  float* state;              // [slots, H, dk, dv]
  const int64_t* slots;      // [n], < 0: skip the sequence
  int64_t num_slots;
  const int32_t* cu_q;       // [n + 1], or null: one token per sequence
  const int32_t* cu_k;       // [n + 1] with cu_q
  const int64_t* ctx_lens;   // [n] without cu_q: context length including the new token
  void* out;                 // [T, H, dv]
  int H, dk, dv;
  int32_t* status;
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// forget gate and write gate of one channel; 1 - f is formed from sigmoid(-z) so that it keeps its relative
// accuracy when the gate is almost closed
__device__ __forceinline__ void gates(float z, float lower, float* f, float* k) {
  const float open = 1.f - lower;
  *f = lower + open * sigmoid_f(z);
  *k = open * sigmoid_f(-z);
}

// The sequence's token range, first position and state slot; false = nothing to do.
struct SeqInfo {
  int64_t tok0;
  int len;
  bool fresh;
  int64_t slot;
};
__device__ __forceinline__ bool sequence_info(const RecArgs& a, int s, SeqInfo* r) {
  if (a.cu_q != nullptr) {
    r->tok0 = a.cu_q[s];
    r->len = a.cu_q[s + 1] - a.cu_q[s];
    r->fresh = (a.cu_k[s + 1] - a.cu_k[s]) <= r->len;
  } else {
    const int64_t n = a.ctx_lens[s];
    r->tok0 = s;
    r->len = n > 0 ? 1 : 0;
    r->fresh = n <= 1;
  }
  r->slot = a.slots[s];
  if (r->slot >= a.num_slots) {
    if (threadIdx.x == 0) report(a.status, B200_ERR_BOUNDS);
    return false;
  }
  return r->len > 0 && r->slot >= 0;
}

constexpr int kStepThreads = 256;

// Threads are RG row groups x CL column units of V columns; a unit walks the key channels rg, rg + RG, ...
template <typename T, int V>
__global__ void __launch_bounds__(kStepThreads) recurrence_step_kernel(const RecArgs a, int CL) {
  extern __shared__ float sm[];
  const int dk = a.dk, dv = a.dv, head = blockIdx.x;
  float* sf = sm;              // [dk] forget gate
  float* sk = sf + dk;         // [dk] write gate
  float* sq = sk + dk;         // [dk]
  float* so = sq + dk;         // [dv]
  float* red = so + dv;        // [256 * V]
  float* scratch = red + kStepThreads * V;   // [8]
  SeqInfo info;
  if (!sequence_info(a, blockIdx.y, &info)) return;
  const int RG = kStepThreads / CL, cu = threadIdx.x % CL, rg = threadIdx.x / CL;
  const int units = (dv + V - 1) / V;
  float* S = a.state + (info.slot * a.H + head) * static_cast<int64_t>(dk) * dv;
  for (int t = 0; t < info.len; ++t) {
    const int64_t row = (info.tok0 + t) * a.stride;
    const T* qp = static_cast<const T*>(a.q) + row + head * dk;
    const T* fp = static_cast<const T*>(a.f) + row + head * dk;
    const T* vp = static_cast<const T*>(a.v) + row + head * dv;
    const bool zero = info.fresh && t == 0;
    for (int i = threadIdx.x; i < dk; i += kStepThreads) {
      const float qv = to_float<T>(qp[i]);
      sq[i] = qv * sigmoid_f(qv);
      gates(to_float<T>(fp[i]) + a.f_bias[head * dk + i], a.lower[head * dk + i], &sf[i], &sk[i]);
    }
    __syncthreads();
    for (int c0 = 0; c0 < units; c0 += CL) {
      const int c = c0 + cu;
      float acc[V];
#pragma unroll
      for (int k = 0; k < V; ++k) acc[k] = 0.f;
      if (c < units) {
        float vv[V];
#pragma unroll
        for (int k = 0; k < V; ++k) vv[k] = to_float<T>(vp[c * V + k]);
#pragma unroll 8
        for (int r = rg; r < dk; r += RG) {
          float* sp = S + static_cast<int64_t>(r) * dv + c * V;
          const float f = sf[r], kk = sk[r], q = sq[r];
          if constexpr (V == 4) {
            float4 x = zero ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(sp);
            x.x = f * x.x + kk * vv[0];
            x.y = f * x.y + kk * vv[1];
            x.z = f * x.z + kk * vv[2];
            x.w = f * x.w + kk * vv[3];
            acc[0] += q * x.x;
            acc[1] += q * x.y;
            acc[2] += q * x.z;
            acc[3] += q * x.w;
            *reinterpret_cast<float4*>(sp) = x;
          } else {
            const float x = f * (zero ? 0.f : *sp) + kk * vv[0];
            acc[0] += q * x;
            *sp = x;
          }
        }
      }
#pragma unroll
      for (int k = 0; k < V; ++k) red[threadIdx.x * V + k] = acc[k];
      __syncthreads();
      const int cols = min(CL * V, dv - c0 * V);
      for (int i = threadIdx.x; i < cols; i += kStepThreads) {
        float o = 0.f;
        for (int g = 0; g < RG; ++g) o += red[(g * CL) * V + i];
        so[c0 * V + i] = o;
      }
      __syncthreads();
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < dv; i += kStepThreads) ss += so[i] * so[i];
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kStepThreads / 32; ++w) tot += scratch[w];
    const float inv = rsqrtf(tot / static_cast<float>(dv) + a.eps);
    T* op = static_cast<T*>(a.out) + (info.tok0 + t) * a.H * dv + head * dv;
    for (int i = threadIdx.x; i < dv; i += kStepThreads) op[i] = from_float<T>(so[i] * inv * a.norm_w[i]);
    __syncthreads();
  }
}

template <typename T>
int launch_step(const RecArgs& a, int n, bool vec, cudaStream_t s) {
  const int V = vec ? 4 : 1;
  const int units = (a.dv + V - 1) / V;
  int CL = 8;
  while (CL < units && CL < kStepThreads) CL *= 2;
  const size_t smem = (3 * static_cast<size_t>(a.dk) + a.dv + kStepThreads * V + 8) * sizeof(float);
  auto kern = vec ? recurrence_step_kernel<T, 4> : recurrence_step_kernel<T, 1>;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem)) != cudaSuccess)
    return B200_ERR_LAUNCH;
  kern<<<dim3(a.H, n), kStepThreads, smem, s>>>(a, CL);
  return launch_result();
}

}  // namespace
}  // namespace b200

extern "C" size_t b200_gated_recurrence_workspace_bytes(int32_t num_seqs, int64_t total_tokens, int32_t max_seqlen_q,
                                                        int32_t num_heads, int32_t dim_k, int32_t dim_v) {
  return 0;
}

extern "C" int b200_gated_recurrence(const void* q, const void* f, const void* v, int64_t token_stride,
                                     const float* f_bias, const float* lower, const float* norm_w, float eps,
                                     float* state, int64_t num_slots, const int64_t* state_slots,
                                     const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                     const int64_t* context_lens, int32_t num_seqs, int64_t total_tokens,
                                     int32_t max_seqlen_q, int32_t num_heads, int32_t dim_k, int32_t dim_v, void* out,
                                     void* workspace, size_t workspace_bytes, int32_t dtype, int32_t* status,
                                     void* stream) {
  using namespace b200;
  if (num_seqs < 0 || num_heads <= 0 || dim_k <= 0 || dim_v <= 0 || num_slots < 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_seqs == 0) return B200_OK;
  if (!q || !f || !v || !f_bias || !lower || !norm_w || !state || !state_slots || !out) return B200_ERR_ARG;
  if (cu_seqlens_q ? !cu_seqlens_k : !context_lens) return B200_ERR_ARG;
  if (num_seqs > 65535 || dim_k > 8192 || dim_v > 8192) return B200_ERR_UNSUPPORTED;
  RecArgs a{q, f, v, token_stride, f_bias, lower, norm_w, eps, state, state_slots, num_slots, cu_seqlens_q,
            cu_seqlens_k, context_lens, out, num_heads, dim_k, dim_v, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool vec = dim_v % 4 == 0 && aligned16(state);
  return dtype == B200_DTYPE_F32 ? launch_step<float>(a, num_seqs, vec, s)
                                 : launch_step<__nv_bfloat16>(a, num_seqs, vec, s);
}
