// Causal attention over a paged KV pool whose heads are mixed before the softmax ("talking heads"), with a
// soft cap on the scores, a logarithmic distance bias, an optional sliding window and an output gate:
//
//   s[g, j]  = cap tanh(scale q[g] . k[j] / cap) - r1[g] ln(1 + r2[g] (i - j))          for every head g
//   m[h, j]  = sum_g talk[h, g] s[g, j]
//   out[h]   = softmax over { j : 0 <= i - j < window } of m[h, :]  applied to v,  times sigmoid(gate[h])
//
// Scores, caps, biases, the mix, the softmax and the accumulation are fp32.  Keys and values always come from
// the pool (the step's rows are stored before the call), so prompts, portions of prompts and single decoded
// tokens are one case: row t of a sequence sits at position k_len - q_len + t.
//
// This file: the general kernel, one CTA per query token with all heads, any sizes, fp32 and bf16, and the
// dispatch.  Because the mix couples the heads of a (query, key) pair, a CTA holds the scores of all of them.
#include "common.cuh"
#include "talking_attention.cuh"

namespace b200 {
namespace {

constexpr int kThreads = 256;
constexpr int KT = 32;       // keys per tile

template <typename T>
__global__ void __launch_bounds__(kThreads) talking_simple_kernel(const TalkArgs a) {
  extern __shared__ float sm[];
  const int H = a.H, dk = a.dk, dv = a.dv, tid = threadIdx.x;
  float* sq = sm;                     // [H, dk]
  float* acc = sq + H * dk;           // [H, dv]
  float* sc = acc + H * dv;           // [H, KT] scores per head
  float* sp = sc + H * KT;            // [H, KT] mixed scores, then weights
  float* st = sp + H * KT;            // [H, H]
  float* smax = st + H * H;           // [H]
  float* ssum = smax + H;             // [H]
  float* scor = ssum + H;             // [H]
  __shared__ int64_t krow[KT];        // pool row of every key of the tile, -1 = none
  const int row = blockIdx.x;
  int seq, pos;                       // the row's sequence and position
  if (a.cu_q != nullptr) {
    int lo = 0, hi = a.n;             // largest seq with cu_q[seq] <= row
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (a.cu_q[mid] <= row) lo = mid; else hi = mid;
    }
    seq = lo;
    if (row >= a.cu_q[seq + 1]) return;             // padding row
    const int qlen = a.cu_q[seq + 1] - a.cu_q[seq], klen = a.cu_k[seq + 1] - a.cu_k[seq];
    pos = klen - qlen + (row - a.cu_q[seq]);
  } else {
    seq = row;
    pos = static_cast<int>(a.ctx_lens[seq]) - 1;
  }
  if (pos < 0) return;
  const T* qp = static_cast<const T*>(a.q) + static_cast<int64_t>(row) * a.q_stride;
  for (int i = tid; i < H * dk; i += kThreads) sq[i] = to_float<T>(qp[i]);
  for (int i = tid; i < H * dv; i += kThreads) acc[i] = 0.f;
  for (int i = tid; i < H * H; i += kThreads) st[i] = a.talk[i];
  for (int i = tid; i < H; i += kThreads) {
    smax[i] = -INFINITY;
    ssum[i] = 0.f;
  }
  const int G = H / a.Hkv;
  const int first = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const int warp = tid >> 5, lane = tid & 31;
  for (int j0 = first; j0 <= pos; j0 += KT) {
    const int nk = min(KT, pos + 1 - j0);
    __syncthreads();
    if (tid < KT) {
      int64_t r = -1;
      if (tid < nk) {
        const int j = j0 + tid, blk = j / a.bs;
        const int id = blk < a.bt_stride ? a.bt[static_cast<int64_t>(seq) * a.bt_stride + blk] : -1;
        if (id < 0 || id >= a.num_blocks) report(a.status, B200_ERR_BOUNDS);
        else r = static_cast<int64_t>(id) * a.bs + j % a.bs;
      }
      krow[tid] = r;
    }
    __syncthreads();
    for (int idx = tid; idx < H * KT; idx += kThreads) {
      const int h = idx / KT, j = idx % KT;
      float s = 0.f;
      if (krow[j] >= 0) {
        const T* kp = static_cast<const T*>(a.kc) + (krow[j] * a.Hkv + h / G) * dk;
        const float* qh = sq + h * dk;
        float dot = 0.f;
        for (int d = 0; d < dk; ++d) dot += qh[d] * to_float<T>(kp[d]);
        s = dot * a.scale;
        if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
        s -= a.r1[h] * log1pf(a.r2[h] * static_cast<float>(pos - j0 - j));
      }
      sc[idx] = s;
    }
    __syncthreads();
    for (int idx = tid; idx < H * KT; idx += kThreads) {
      const int h = idx / KT, j = idx % KT;
      float m = 0.f;
      for (int g = 0; g < H; ++g) m += st[h * H + g] * sc[g * KT + j];
      sp[idx] = krow[j] >= 0 ? m : -INFINITY;
    }
    __syncthreads();
    for (int h = warp; h < H; h += kThreads / 32) {      // KT == warp width: one key per lane
      const float m = sp[h * KT + lane];
      const float mn = fmaxf(smax[h], warp_max(m));
      const float sub = mn == -INFINITY ? 0.f : mn;
      const float p = expf(m - sub);
      const float cor = expf(smax[h] - sub);
      const float tot = warp_sum(p);
      __syncwarp();
      sp[h * KT + lane] = p;
      if (lane == 0) {
        smax[h] = mn;
        ssum[h] = ssum[h] * cor + tot;
        scor[h] = cor;
      }
    }
    __syncthreads();
    for (int idx = tid; idx < H * dv; idx += kThreads) {
      const int h = idx / dv, d = idx % dv;
      float o = acc[idx] * scor[h];
      for (int j = 0; j < nk; ++j)
        if (krow[j] >= 0)
          o += sp[h * KT + j] * to_float<T>(static_cast<const T*>(a.vc)[(krow[j] * a.Hkv + h / G) * dv + d]);
      acc[idx] = o;
    }
  }
  __syncthreads();
  T* op = static_cast<T*>(a.out) + static_cast<int64_t>(row) * H * dv;
  const T* gp = a.gate ? static_cast<const T*>(a.gate) + static_cast<int64_t>(row) * a.gate_stride : nullptr;
  for (int idx = tid; idx < H * dv; idx += kThreads) {
    const float l = ssum[idx / dv];
    float o = l > 0.f ? acc[idx] / l : 0.f;
    if (gp) o /= 1.f + expf(-to_float<T>(gp[idx]));
    op[idx] = from_float<T>(o);
  }
}

template <typename T>
int launch_simple(const TalkArgs& a, cudaStream_t s) {
  const size_t smem = (static_cast<size_t>(a.H) * (a.dk + a.dv + 2 * KT + a.H + 3)) * sizeof(float);
  if (smem > 220 * 1024) return B200_ERR_UNSUPPORTED;
  auto kern = talking_simple_kernel<T>;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem)) != cudaSuccess)
    return B200_ERR_LAUNCH;
  kern<<<static_cast<unsigned>(a.rows), kThreads, smem, s>>>(a);
  return launch_result();
}

}  // namespace
}  // namespace b200

extern "C" size_t b200_talking_attention_workspace_bytes(int32_t num_seqs, int32_t num_heads, int32_t dim_v,
                                                         int32_t window, int32_t decode, int32_t dtype) {
  using namespace b200;
  if (!decode || dtype != B200_DTYPE_BF16 || num_seqs <= 0 || num_heads <= 0 || dim_v <= 0) return 0;
  return talking_decode_workspace_bytes(num_seqs, num_heads, dim_v, window);
}

extern "C" int b200_talking_attention(const void* q, int64_t q_stride, const void* gate, int64_t gate_stride,
                                      const void* k_cache, const void* v_cache, void* out,
                                      const int32_t* block_tables, int64_t bt_stride, int32_t block_size,
                                      int64_t num_blocks, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                      const int64_t* context_lens, int32_t num_seqs, int64_t rows, int32_t max_seqlen_q,
                                      int32_t num_heads, int32_t num_kv_heads, int32_t dim_k, int32_t dim_v,
                                      float scale, float softcap, const float* r1, const float* r2, const float* talk,
                                      const float* consts_host, const float* bias_table, int32_t bias_len,
                                      int32_t window, const int32_t* plan, int32_t plan_tile_rows,
                                      int32_t plan_capacity, void* workspace, size_t workspace_bytes, int32_t dtype,
                                      int32_t* status, void* stream) {
  using namespace b200;
  if (num_seqs < 0 || rows < 0 || num_heads <= 0 || num_kv_heads <= 0 || num_heads % num_kv_heads || dim_k <= 0 ||
      dim_v <= 0 || block_size <= 0 || bt_stride <= 0 || num_blocks <= 0)
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_seqs == 0 || rows == 0) return B200_OK;
  if (!q || !k_cache || !v_cache || !out || !block_tables || !r1 || !r2 || !talk) return B200_ERR_ARG;
  if (cu_seqlens_q ? !cu_seqlens_k : (!context_lens || rows > num_seqs)) return B200_ERR_ARG;
  if (rows > 2147483647LL) return B200_ERR_TOO_LARGE;
  TalkArgs a{};
  a.q = q;
  a.q_stride = q_stride;
  a.gate = gate;
  a.gate_stride = gate_stride;
  a.kc = k_cache;
  a.vc = v_cache;
  a.out = out;
  a.bt = block_tables;
  a.bt_stride = bt_stride;
  a.bs = block_size;
  a.bs_log2 = -1;
  for (int i = 0; i < 31; ++i)
    if (block_size == 1 << i) a.bs_log2 = i;
  a.num_blocks = num_blocks;
  a.cu_q = cu_seqlens_q;
  a.cu_k = cu_seqlens_k;
  a.ctx_lens = context_lens;
  a.n = num_seqs;
  a.rows = rows;
  a.H = num_heads;
  a.Hkv = num_kv_heads;
  a.dk = dim_k;
  a.dv = dim_v;
  a.scale = scale;
  a.cap = softcap;
  a.r1 = r1;
  a.r2 = r2;
  a.talk = talk;
  a.window = window;
  a.max_q = max_seqlen_q;
  a.plan = cu_seqlens_q && plan_tile_rows == kTalkTileRows && plan_capacity > 0 ? plan : nullptr;
  a.plan_capacity = plan_capacity;
  a.talk_host = consts_host;
  a.r1_host = consts_host ? consts_host + static_cast<size_t>(num_heads) * num_heads : nullptr;
  a.r2_host = consts_host ? a.r1_host + num_heads : nullptr;
  a.bias_table = bias_table;
  a.bias_len = bias_table ? bias_len : 0;
  a.workspace = workspace;
  a.workspace_bytes = workspace_bytes;
  a.status = status;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_F32) return launch_simple<float>(a, s);
  const int rc = a.cu_q ? talking_prefill_mma_launch(a, s) : talking_decode_mma_launch(a, s);
  return rc != B200_ERR_UNSUPPORTED ? rc : launch_simple<__nv_bfloat16>(a, s);
}
