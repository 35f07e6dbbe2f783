// Ragged (varlen) causal prefill attention over cu_seqlens-packed sequences.
//
// Generic path: one warp per (sequence, query token, query head); a lane owns the head-dim
// elements lane, lane+32, ...; keys are visited in order with an fp32 online softmax.  Keys and
// values come either from the packed k/v tensors of the step or, when a cached prefix exists,
// from the paged pool through block_tables (bottom-right aligned causal mask).  The packed keys may come in two parts, the
// second shared by all heads, and a query may see only the last `window` keys.  SIGM: the weights are sigmoid(scale q.k +
// bias[head]), summed as they are over the keys of the query's chunk of positions, and rows leave through a gate.
#include "sequences.cuh"

namespace b200 {
namespace {

struct PrefillArgs {
  const void* q;
  const void* k;
  const void* v;
  void* out;
  int64_t q_stride, k_stride, v_stride;  // token strides, elements
  const int32_t* cu_q;
  const int32_t* cu_k;
  int num_seqs, Hq, Hkv, Dqk, Dv;
  float scale_log2;
  const void* kc;
  const void* vc;
  const int32_t* bt;
  int64_t bt_stride;
  int bs;
  int64_t num_blocks;
  const float* sink;  // [Hq] or null
  const void* k_tail; // [Tk, tail] or null (packed keys): the last `tail` columns of every head's key
  int64_t k_tail_stride;
  int tail;
  int window;         // 0: none
  int32_t* status;
  const float* bias;  // SIGM: [Hq]
  int chunk;          // SIGM: positions per chunk, counted from the first key
  const void* gate;   // SIGM: [tokens, Hq] or null
  int64_t gate_stride;
};

constexpr int kWarps = 4;
constexpr int kMaxPerLane = 8;    // head dims <= 256
constexpr int kWidePerLane = 32;  // head dims <= 1024

template <typename T, int kMaxPerLane, bool SIGM>
__global__ void __launch_bounds__(kWarps * 32) prefill_simple_kernel(const PrefillArgs a) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int s = blockIdx.z, head = blockIdx.y;
  const int qi = blockIdx.x * kWarps + warp;
  const int q0 = a.cu_q[s], q_len = a.cu_q[s + 1] - q0;
  const int k0 = a.cu_k[s], k_len = a.cu_k[s + 1] - k0;
  if (qi >= q_len) return;
  const int G = a.Hq / a.Hkv, kvh = head / G;
  const int nkeys = k_len - q_len + qi + 1;  // causal, bottom-right aligned
  const T* qp = static_cast<const T*>(a.q) + static_cast<int64_t>(q0 + qi) * a.q_stride +
                static_cast<int64_t>(head) * a.Dqk;
  float qv[kMaxPerLane], acc[kMaxPerLane];
#pragma unroll
  for (int i = 0; i < kMaxPerLane; ++i) {
    const int d = lane + 32 * i;
    qv[i] = d < a.Dqk ? to_float<T>(qp[d]) : 0.f;
    acc[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int Dh = a.Dqk - a.tail;
  const int first = SIGM ? (nkeys - 1) / a.chunk * a.chunk : a.window > 0 ? max(nkeys - a.window, 0) : 0;
  for (int j = first; j < nkeys; ++j) {
    const T* kp;
    const T* kt = nullptr;
    const T* vp;
    if (a.bt == nullptr) {
      kp = static_cast<const T*>(a.k) + static_cast<int64_t>(k0 + j) * a.k_stride + static_cast<int64_t>(kvh) * Dh;
      if (a.tail > 0) kt = static_cast<const T*>(a.k_tail) + static_cast<int64_t>(k0 + j) * a.k_tail_stride;
      vp = static_cast<const T*>(a.v) + static_cast<int64_t>(k0 + j) * a.v_stride +
           static_cast<int64_t>(kvh) * a.Dv;
    } else {
      const int blk = j / a.bs;
      if (blk >= a.bt_stride) {
        report(a.status, B200_ERR_BOUNDS);
        break;
      }
      const int id = a.bt[static_cast<int64_t>(s) * a.bt_stride + blk];
      if (static_cast<uint64_t>(static_cast<int64_t>(id)) >= static_cast<uint64_t>(a.num_blocks)) {
        report(a.status, B200_ERR_BOUNDS);
        continue;
      }
      const int64_t row = (static_cast<int64_t>(id) * a.bs + j % a.bs) * a.Hkv + kvh;
      kp = static_cast<const T*>(a.kc) + row * a.Dqk;
      vp = static_cast<const T*>(a.vc) + row * a.Dv;
    }
    float dot = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i) {
      const int d = lane + 32 * i;
      if (d < Dh) dot += qv[i] * to_float<T>(kp[d]);
      else if (d < a.Dqk) dot += qv[i] * to_float<T>(kt[d - Dh]);
    }
    dot = warp_sum(dot);
    if constexpr (SIGM) {
      const float p = sigmoid_f(dot * a.scale_log2 + a.bias[head]);
#pragma unroll
      for (int i = 0; i < kMaxPerLane; ++i) {
        const int d = lane + 32 * i;
        if (d < a.Dv) acc[i] += p * to_float<T>(vp[d]);
      }
      continue;
    }
    dot *= a.scale_log2;
    const float mn = fmaxf(m, dot);
    const float al = exp2f(m - mn), pw = exp2f(dot - mn);
    l = l * al + pw;
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i) {
      const int d = lane + 32 * i;
      if (d < a.Dv) acc[i] = acc[i] * al + pw * to_float<T>(vp[d]);
    }
    m = mn;
  }
  T* op = static_cast<T*>(a.out) + (static_cast<int64_t>(q0 + qi) * a.Hq + head) * a.Dv;
  if (a.sink != nullptr && nkeys > 0) l += exp2f(a.sink[head] * 1.4426950408889634f - m);
  float inv = l > 0.f ? 1.f / l : 0.f;
  if constexpr (SIGM)
    inv = a.gate ? sigmoid_f(to_float<T>(static_cast<const T*>(a.gate)[static_cast<int64_t>(q0 + qi) * a.gate_stride + head])) : 1.f;
#pragma unroll
  for (int i = 0; i < kMaxPerLane; ++i) {
    const int d = lane + 32 * i;
    if (d < a.Dv) op[d] = from_float<T>(acc[i] * inv);
  }
}

}  // namespace

// fast bf16 tensor-core path, defined in prefill_mma.cu; returns B200_ERR_UNSUPPORTED when the
// shape is outside what it implements
int prefill_mma_launch(const void* q, const void* k, const void* v, void* out, int64_t q_stride,
                       int64_t k_stride, int64_t v_stride, const int32_t* cu_q,
                       const int32_t* cu_k, int num_seqs, int max_seqlen_q, int Hq, int Hkv,
                       int Dqk, int Dv, float scale, const void* kc, const void* vc,
                       const int32_t* bt, int64_t bt_stride, int bs, int64_t num_blocks,
                       const int32_t* plan, int plan_tile_rows, int plan_capacity, int32_t* status,
                       cudaStream_t s, const void* k_tail, int64_t k_tail_stride, int tail, const float* sink);

// tcgen05 path for packed keys/values (prefill_umma2.cu): head dims 128/128 and 192/128, 256 query rows of one head per CTA
int prefill_umma2_tile_rows(int Hq, int Hkv, int Dqk, int Dv);
int prefill_umma4_tile_rows(int Hq, int Hkv, int Dqk, int Dv);
int prefill_umma4_launch(const void* q, const void* k, const void* v, void* out, int64_t q_stride, int64_t k_stride,
                         int64_t v_stride, int64_t total_q, int64_t total_k, const int32_t* cu_q,
                         const int32_t* cu_k, int num_seqs, int max_seqlen_q, int Hq, int Hkv, int Dqk, int Dv,
                         float scale, const int32_t* plan, int plan_tile_rows, int plan_capacity, int32_t* status,
                         cudaStream_t s, const float* sink);
int prefill_umma2_launch(const void* q, const void* k, const void* v, void* out, int64_t q_stride, int64_t k_stride,
                         int64_t v_stride, int64_t total_q, int64_t total_k, const int32_t* cu_q,
                         const int32_t* cu_k, int num_seqs, int max_seqlen_q, int Hq, int Hkv, int Dqk, int Dv,
                         float scale, const int32_t* plan, int plan_tile_rows, int plan_capacity, int32_t* status,
                         cudaStream_t s, const void* k_tail, int64_t k_tail_stride, int tail, const float* sink,
                         int window);

// mma.sync path for head sizes below the compiled ones, keys in two parts, a sliding window (prefill_mma.cu); packed keys
bool prefill_mma_general_shape(int Dqk, int Dv, int tail);
int prefill_mma_general_launch(const void* q, const void* k, const void* v, void* out, int64_t q_stride, int64_t k_stride,
                               int64_t v_stride, const int32_t* cu_q, const int32_t* cu_k, int num_seqs, int max_seqlen_q,
                               int Hq, int Hkv, int Dqk, int Dv, float scale, const int32_t* plan, int plan_tile_rows,
                               int plan_capacity, int32_t* status, cudaStream_t s, const void* k_tail, int64_t k_tail_stride,
                               int tail, const float* sink, int window);

// sigmoid weights inside chunks: tcgen05 at head sizes 128 and 64 (prefill_umma2.cu), mma.sync at the general ones (prefill_mma.cu)
int prefill_umma2_sigmoid_tile_rows(int Hq, int Hkv, int Dqk, int Dv);
int prefill_umma2_sigmoid_launch(const void* q, const void* k, const void* v, void* out, int64_t q_stride, int64_t k_stride,
                                 int64_t v_stride, int64_t total_q, int64_t total_k, const int32_t* cu_q, const int32_t* cu_k,
                                 int num_seqs, int max_seqlen_q, int Hq, int Hkv, int Dqk, int Dv, float scale, const float* bias,
                                 int chunk, const void* gate, int64_t gate_stride, const int32_t* plan, int plan_tile_rows,
                                 int plan_capacity, int32_t* status, cudaStream_t s);
int prefill_mma_sigmoid_launch(const void* q, const void* k, const void* v, void* out, int64_t q_stride, int64_t k_stride,
                               int64_t v_stride, const int32_t* cu_q, const int32_t* cu_k, int num_seqs, int max_seqlen_q,
                               int Hq, int Hkv, int Dqk, int Dv, float scale, const float* bias, int chunk, const void* gate,
                               int64_t gate_stride, const int32_t* plan, int plan_tile_rows, int plan_capacity, int32_t* status,
                               cudaStream_t s);

// tcgen05 path for a paged prefix (prefill_umma.cu): head_dim 128, even group size, two heads per CTA
int prefill_umma_launch(const void* q, const void* k, const void* v, void* out, int64_t q_stride,
                        int64_t k_stride, int64_t v_stride, int64_t total_q, int64_t total_k,
                        const int32_t* cu_q, const int32_t* cu_k,
                        int num_seqs, int max_seqlen_q, int Hq, int Hkv, int Dqk, int Dv, float scale,
                        const void* kc, const void* vc, const int32_t* bt, int64_t bt_stride, int bs,
                        int64_t num_blocks, const int32_t* plan, int plan_tile_rows, int plan_capacity,
                        int32_t* status, cudaStream_t s, const float* sink);

}  // namespace b200

extern "C" int32_t b200_prefill_tile_rows(int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                                          int32_t head_dim_v, int32_t dtype) {
  if (dtype != B200_DTYPE_BF16 || num_kv_heads <= 0 || num_q_heads % num_kv_heads != 0) return 0;
  // packed keys: the row-pair tcgen05 kernel serves 128/128 and 192/128 (the two-head kernel, 128 rows per
  // tile, only takes over for a paged prefix and then ignores a 256-row tile list)
  if (const int r = b200::prefill_umma2_tile_rows(num_q_heads, num_kv_heads, head_dim_qk, head_dim_v)) return r;
  // head_dim 64 with query heads in groups of four per KV head: the four-heads-per-CTA tcgen05 kernel, 128 rows
  if (const int r = b200::prefill_umma4_tile_rows(num_q_heads, num_kv_heads, head_dim_qk, head_dim_v)) return r;
  const bool mma = (head_dim_qk == head_dim_v && (head_dim_qk == 32 || head_dim_qk == 64 || head_dim_qk == 128)) ||
                   (head_dim_qk == 192 && head_dim_v == 128);
  return mma ? 64 : 0;
}

namespace b200 {
namespace {
template <bool SIGM = false>
int simple_launch(const PrefillArgs& a, int max_seqlen_q, int32_t dtype, cudaStream_t s) {
  const int widest = a.Dqk > a.Dv ? a.Dqk : a.Dv;
  if (widest > kWidePerLane * 32 || a.num_seqs > 65535 || a.Hq > 65535) return B200_ERR_UNSUPPORTED;
  const dim3 grid((max_seqlen_q + kWarps - 1) / kWarps, a.Hq, a.num_seqs);
  const bool wide = widest > kMaxPerLane * 32;
  if (dtype == B200_DTYPE_F32) {
    if (wide) prefill_simple_kernel<float, kWidePerLane, SIGM><<<grid, kWarps * 32, 0, s>>>(a);
    else prefill_simple_kernel<float, kMaxPerLane, SIGM><<<grid, kWarps * 32, 0, s>>>(a);
  } else {
    if (wide) prefill_simple_kernel<__nv_bfloat16, kWidePerLane, SIGM><<<grid, kWarps * 32, 0, s>>>(a);
    else prefill_simple_kernel<__nv_bfloat16, kMaxPerLane, SIGM><<<grid, kWarps * 32, 0, s>>>(a);
  }
  return launch_result();
}
}  // namespace
}  // namespace b200

static int prefill_attention(const void* q, const void* k, const void* v, void* out,
                                   int64_t q_token_stride, int64_t k_token_stride,
                                   int64_t v_token_stride, int64_t total_q_tokens,
                                   int64_t total_k_tokens, const int32_t* cu_seqlens_q,
                                   const int32_t* cu_seqlens_k, int32_t num_seqs,
                                   int32_t max_seqlen_q, int32_t max_seqlen_k,
                                   int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                                   int32_t head_dim_v, float scale, const void* k_cache,
                                   const void* v_cache, const int32_t* block_tables,
                                   int64_t bt_stride, int32_t block_size, int64_t num_blocks,
                                   const int64_t* slot_mapping, const int32_t* plan, int32_t plan_tile_rows,
                                   int32_t plan_capacity, const float* sink, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (num_seqs < 0 || max_seqlen_q < 0 || max_seqlen_k < 0 || num_q_heads <= 0 ||
      num_kv_heads <= 0 || head_dim_qk <= 0 || head_dim_v <= 0)
    return B200_ERR_ARG;
  if (num_q_heads % num_kv_heads != 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (total_q_tokens < 0 || total_k_tokens < 0) return B200_ERR_ARG;
  if (num_seqs == 0 || max_seqlen_q == 0 || total_q_tokens == 0) return B200_OK;
  if (!q || !out || !cu_seqlens_q || !cu_seqlens_k) return B200_ERR_ARG;
  if (block_tables == nullptr) {
    if (!k || !v) return B200_ERR_ARG;
  } else {
    if (!k_cache || !v_cache || block_size <= 0 || bt_stride <= 0 || num_blocks <= 0)
      return B200_ERR_ARG;
  }
  cudaStream_t s = static_cast<cudaStream_t>(stream);

  if (slot_mapping != nullptr) {
    // the step's store_kvcache scatter rides in this call: the new tokens' rows go into the pool first (its
    // own launch, ahead of the attention grid in the stream), so a paged prefix read sees them
    if (!k || !v || !k_cache || !v_cache || block_size <= 0 || num_blocks <= 0) return B200_ERR_ARG;
    if (head_dim_qk != head_dim_v) return B200_ERR_UNSUPPORTED;
    const int64_t rows = block_tables == nullptr && total_k_tokens < total_q_tokens ? total_k_tokens : total_q_tokens;
    if (rows > 2147483647LL) return B200_ERR_TOO_LARGE;
    const int rc = b200_store_kvcache(k, v, k_token_stride, v_token_stride, const_cast<void*>(k_cache),
                                      const_cast<void*>(v_cache), slot_mapping, static_cast<int32_t>(rows),
                                      num_kv_heads, head_dim_qk, num_blocks * block_size, dtype, status, stream);
    if (rc != B200_OK) return rc;
  }

  if (dtype == B200_DTYPE_BF16) {
    if (block_tables == nullptr) {
      // packed keys: 256 query rows of one head per CTA (measured 967 against 865 TFLOP/s for the two-head
      // kernel on 262,144 ragged tokens at head_dim 128)
      const int rc2 = prefill_umma2_launch(q, k, v, out, q_token_stride, k_token_stride, v_token_stride,
                                           total_q_tokens, total_k_tokens, cu_seqlens_q, cu_seqlens_k, num_seqs,
                                           max_seqlen_q, num_q_heads, num_kv_heads, head_dim_qk, head_dim_v, scale,
                                           plan, plan_tile_rows, plan_capacity, status, s, nullptr, 0, 0, sink, 0);
      if (rc2 != B200_ERR_UNSUPPORTED) return rc2;
      // head_dim 64, four query heads of a KV head per CTA
      const int rc4 = prefill_umma4_launch(q, k, v, out, q_token_stride, k_token_stride, v_token_stride,
                                           total_q_tokens, total_k_tokens, cu_seqlens_q, cu_seqlens_k, num_seqs,
                                           max_seqlen_q, num_q_heads, num_kv_heads, head_dim_qk, head_dim_v, scale,
                                           plan, plan_tile_rows, plan_capacity, status, s, sink);
      if (rc4 != B200_ERR_UNSUPPORTED) return rc4;
    }
    const int rcu = prefill_umma_launch(q, k, v, out, q_token_stride, k_token_stride, v_token_stride,
                                        total_q_tokens, total_k_tokens, cu_seqlens_q, cu_seqlens_k, num_seqs, max_seqlen_q, num_q_heads,
                                        num_kv_heads, head_dim_qk, head_dim_v, scale, k_cache, v_cache,
                                        block_tables, bt_stride, block_size, num_blocks, plan, plan_tile_rows,
                                        plan_capacity, status, s, sink);
    if (rcu != B200_ERR_UNSUPPORTED) return rcu;
    const int rc = prefill_mma_launch(q, k, v, out, q_token_stride, k_token_stride,
                                      v_token_stride, cu_seqlens_q, cu_seqlens_k, num_seqs,
                                      max_seqlen_q, num_q_heads, num_kv_heads, head_dim_qk,
                                      head_dim_v, scale, k_cache, v_cache, block_tables, bt_stride,
                                      block_size, num_blocks, plan, plan_tile_rows, plan_capacity, status, s,
                                      nullptr, 0, 0, sink);
    if (rc != B200_ERR_UNSUPPORTED) return rc;
  }

  PrefillArgs a{};
  a.q = q;
  a.k = k;
  a.v = v;
  a.out = out;
  a.q_stride = q_token_stride;
  a.k_stride = k_token_stride;
  a.v_stride = v_token_stride;
  a.cu_q = cu_seqlens_q;
  a.cu_k = cu_seqlens_k;
  a.num_seqs = num_seqs;
  a.Hq = num_q_heads;
  a.Hkv = num_kv_heads;
  a.Dqk = head_dim_qk;
  a.Dv = head_dim_v;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.kc = k_cache;
  a.vc = v_cache;
  a.bt = block_tables;
  a.bt_stride = bt_stride;
  a.bs = block_size;
  a.num_blocks = num_blocks;
  a.sink = sink;
  a.status = status;
  return simple_launch(a, max_seqlen_q, dtype, s);
}

extern "C" int b200_prefill_varlen(const void* q, const void* k, const void* v, void* out,
                                   int64_t q_token_stride, int64_t k_token_stride,
                                   int64_t v_token_stride, int64_t total_q_tokens,
                                   int64_t total_k_tokens, const int32_t* cu_seqlens_q,
                                   const int32_t* cu_seqlens_k, int32_t num_seqs,
                                   int32_t max_seqlen_q, int32_t max_seqlen_k,
                                   int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                                   int32_t head_dim_v, float scale, const void* k_cache,
                                   const void* v_cache, const int32_t* block_tables,
                                   int64_t bt_stride, int32_t block_size, int64_t num_blocks,
                                   const int64_t* slot_mapping, const int32_t* plan, int32_t plan_tile_rows,
                                   int32_t plan_capacity, int32_t dtype, int32_t* status, void* stream) {
  return prefill_attention(q, k, v, out, q_token_stride, k_token_stride, v_token_stride, total_q_tokens,
                           total_k_tokens, cu_seqlens_q, cu_seqlens_k, num_seqs, max_seqlen_q, max_seqlen_k,
                           num_q_heads, num_kv_heads, head_dim_qk, head_dim_v, scale, k_cache, v_cache, block_tables,
                           bt_stride, block_size, num_blocks, slot_mapping, plan, plan_tile_rows, plan_capacity,
                           nullptr, dtype, status, stream);
}

extern "C" int b200_prefill_varlen_sink(const void* q, const void* k, const void* v, void* out,
                                   int64_t q_token_stride, int64_t k_token_stride,
                                   int64_t v_token_stride, int64_t total_q_tokens,
                                   int64_t total_k_tokens, const int32_t* cu_seqlens_q,
                                   const int32_t* cu_seqlens_k, int32_t num_seqs,
                                   int32_t max_seqlen_q, int32_t max_seqlen_k,
                                   int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                                   int32_t head_dim_v, float scale, const void* k_cache,
                                   const void* v_cache, const int32_t* block_tables,
                                   int64_t bt_stride, int32_t block_size, int64_t num_blocks,
                                   const int64_t* slot_mapping, const int32_t* plan, int32_t plan_tile_rows,
                                   int32_t plan_capacity, const float* sink, int32_t dtype, int32_t* status, void* stream) {
  return prefill_attention(q, k, v, out, q_token_stride, k_token_stride, v_token_stride, total_q_tokens,
                           total_k_tokens, cu_seqlens_q, cu_seqlens_k, num_seqs, max_seqlen_q, max_seqlen_k,
                           num_q_heads, num_kv_heads, head_dim_qk, head_dim_v, scale, k_cache, v_cache, block_tables,
                           bt_stride, block_size, num_blocks, slot_mapping, plan, plan_tile_rows, plan_capacity,
                           sink, dtype, status, stream);
}

extern "C" int b200_prefill_varlen_shared_tail(const void* q, const void* k_head, const void* k_tail, const void* v,
                                               void* out, int64_t q_token_stride, int64_t k_head_token_stride,
                                               int64_t k_tail_token_stride, int64_t v_token_stride,
                                               int64_t total_q_tokens, int64_t total_k_tokens,
                                               const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                               int32_t num_seqs, int32_t max_seqlen_q, int32_t num_heads,
                                               int32_t head_dim_qk, int32_t tail_dim, int32_t head_dim_v,
                                               float scale, const int32_t* plan, int32_t plan_tile_rows,
                                               int32_t plan_capacity, int32_t dtype, int32_t* status,
                                               void* stream) {
  using namespace b200;
  if (num_seqs < 0 || max_seqlen_q < 0 || num_heads <= 0 || head_dim_qk <= 0 || head_dim_v <= 0 ||
      tail_dim <= 0 || tail_dim >= head_dim_qk)
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_seqs == 0 || max_seqlen_q == 0) return B200_OK;
  if (!q || !k_head || !k_tail || !v || !out || !cu_seqlens_q || !cu_seqlens_k) return B200_ERR_ARG;
  if (total_q_tokens <= 0 || total_k_tokens <= 0) return B200_ERR_ARG;
  const int rc2 = prefill_umma2_launch(q, k_head, v, out, q_token_stride, k_head_token_stride, v_token_stride,
                                       total_q_tokens, total_k_tokens, cu_seqlens_q, cu_seqlens_k, num_seqs,
                                       max_seqlen_q, num_heads, num_heads, head_dim_qk, head_dim_v, scale, plan,
                                       plan_tile_rows, plan_capacity, status, static_cast<cudaStream_t>(stream),
                                       k_tail, k_tail_token_stride, tail_dim, nullptr, 0);
  if (rc2 != B200_ERR_UNSUPPORTED) return rc2;
  return prefill_mma_launch(q, k_head, v, out, q_token_stride, k_head_token_stride, v_token_stride, cu_seqlens_q,
                            cu_seqlens_k, num_seqs, max_seqlen_q, num_heads, num_heads, head_dim_qk, head_dim_v,
                            scale, nullptr, nullptr, nullptr, 0, 0, 0, plan, plan_tile_rows, plan_capacity, status,
                            static_cast<cudaStream_t>(stream), k_tail, k_tail_token_stride, tail_dim, nullptr);
}

extern "C" int32_t b200_prefill_window_tile_rows(int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                                                 int32_t tail_dim, int32_t head_dim_v, int32_t dtype) {
  if (dtype != B200_DTYPE_BF16 || num_kv_heads <= 0 || num_q_heads % num_kv_heads != 0) return 0;
  if (tail_dim == 0 || (tail_dim == 64 && head_dim_qk == 192))
    if (const int r = b200::prefill_umma2_tile_rows(num_q_heads, num_kv_heads, head_dim_qk, head_dim_v)) return r;
  return b200::prefill_mma_general_shape(head_dim_qk, head_dim_v, tail_dim) ? 64 : 0;
}

extern "C" int b200_prefill_varlen_window(const void* q, const void* k_head, const void* k_tail, const void* v, void* out,
                                          int64_t q_token_stride, int64_t k_head_token_stride, int64_t k_tail_token_stride,
                                          int64_t v_token_stride, int64_t total_q_tokens, int64_t total_k_tokens,
                                          const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, int32_t num_seqs,
                                          int32_t max_seqlen_q, int32_t num_q_heads, int32_t num_kv_heads,
                                          int32_t head_dim_qk, int32_t tail_dim, int32_t head_dim_v, float scale,
                                          int32_t window, const float* sink, const int32_t* plan, int32_t plan_tile_rows,
                                          int32_t plan_capacity, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (num_seqs < 0 || max_seqlen_q < 0 || num_q_heads <= 0 || num_kv_heads <= 0 || num_q_heads % num_kv_heads || head_dim_qk <= 0 ||
      head_dim_v <= 0 || tail_dim < 0 || tail_dim >= head_dim_qk || window < 0)
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_seqs == 0 || max_seqlen_q == 0) return B200_OK;
  if (!q || !k_head || (tail_dim > 0 && !k_tail) || !v || !out || !cu_seqlens_q || !cu_seqlens_k) return B200_ERR_ARG;
  if (total_q_tokens <= 0 || total_k_tokens <= 0) return B200_ERR_ARG;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_BF16) {
    const int rc2 = prefill_umma2_launch(q, k_head, v, out, q_token_stride, k_head_token_stride, v_token_stride, total_q_tokens,
                                         total_k_tokens, cu_seqlens_q, cu_seqlens_k, num_seqs, max_seqlen_q, num_q_heads,
                                         num_kv_heads, head_dim_qk, head_dim_v, scale, plan, plan_tile_rows, plan_capacity,
                                         status, s, k_tail, k_tail_token_stride, tail_dim, sink, window);
    if (rc2 != B200_ERR_UNSUPPORTED) return rc2;
    const int rc = prefill_mma_general_launch(q, k_head, v, out, q_token_stride, k_head_token_stride, v_token_stride,
                                              cu_seqlens_q, cu_seqlens_k, num_seqs, max_seqlen_q, num_q_heads, num_kv_heads,
                                              head_dim_qk, head_dim_v, scale, plan, plan_tile_rows, plan_capacity, status, s,
                                              k_tail, k_tail_token_stride, tail_dim, sink, window);
    if (rc != B200_ERR_UNSUPPORTED) return rc;
  }
  PrefillArgs a{};
  a.q = q;
  a.k = k_head;
  a.v = v;
  a.out = out;
  a.q_stride = q_token_stride;
  a.k_stride = k_head_token_stride;
  a.v_stride = v_token_stride;
  a.cu_q = cu_seqlens_q;
  a.cu_k = cu_seqlens_k;
  a.num_seqs = num_seqs;
  a.Hq = num_q_heads;
  a.Hkv = num_kv_heads;
  a.Dqk = head_dim_qk;
  a.Dv = head_dim_v;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.sink = sink;
  a.k_tail = k_tail;
  a.k_tail_stride = k_tail_token_stride;
  a.tail = tail_dim;
  a.window = window;
  a.status = status;
  return simple_launch(a, max_seqlen_q, dtype, s);
}

extern "C" int32_t b200_sigmoid_attention_tile_rows(int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                                                    int32_t head_dim_v, int32_t dtype) {
  if (dtype != B200_DTYPE_BF16 || num_kv_heads <= 0 || num_q_heads % num_kv_heads != 0) return 0;
  if (const int r = b200::prefill_umma2_sigmoid_tile_rows(num_q_heads, num_kv_heads, head_dim_qk, head_dim_v)) return r;
  return b200::prefill_mma_general_shape(head_dim_qk, head_dim_v, 0) ? 64 : 0;
}

extern "C" int b200_sigmoid_attention(const void* q, const void* k, const void* v, void* out, int64_t q_token_stride,
                                      int64_t k_token_stride, int64_t v_token_stride, int64_t total_q_tokens,
                                      int64_t total_k_tokens, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                      int32_t num_seqs, int32_t max_seqlen_q, int32_t num_q_heads, int32_t num_kv_heads,
                                      int32_t head_dim_qk, int32_t head_dim_v, float scale, const float* bias, int32_t chunk,
                                      const void* gate, int64_t gate_token_stride, const int32_t* plan, int32_t plan_tile_rows,
                                      int32_t plan_capacity, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (num_seqs < 0 || max_seqlen_q < 0 || num_q_heads <= 0 || num_kv_heads <= 0 || num_q_heads % num_kv_heads || head_dim_qk <= 0 ||
      head_dim_v <= 0 || chunk < 0)
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_seqs == 0 || max_seqlen_q == 0) return B200_OK;
  if (!q || !k || !v || !out || !cu_seqlens_q || !cu_seqlens_k || !bias) return B200_ERR_ARG;
  if (total_q_tokens <= 0 || total_k_tokens <= 0) return B200_ERR_ARG;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_BF16) {
    const int rc2 = prefill_umma2_sigmoid_launch(q, k, v, out, q_token_stride, k_token_stride, v_token_stride, total_q_tokens,
                                                 total_k_tokens, cu_seqlens_q, cu_seqlens_k, num_seqs, max_seqlen_q, num_q_heads,
                                                 num_kv_heads, head_dim_qk, head_dim_v, scale, bias, chunk, gate,
                                                 gate_token_stride, plan, plan_tile_rows, plan_capacity, status, s);
    if (rc2 != B200_ERR_UNSUPPORTED) return rc2;
    const int rc = prefill_mma_sigmoid_launch(q, k, v, out, q_token_stride, k_token_stride, v_token_stride, cu_seqlens_q,
                                              cu_seqlens_k, num_seqs, max_seqlen_q, num_q_heads, num_kv_heads, head_dim_qk,
                                              head_dim_v, scale, bias, chunk, gate, gate_token_stride, plan, plan_tile_rows,
                                              plan_capacity, status, s);
    if (rc != B200_ERR_UNSUPPORTED) return rc;
  }
  PrefillArgs a{};
  a.q = q;
  a.k = k;
  a.v = v;
  a.out = out;
  a.q_stride = q_token_stride;
  a.k_stride = k_token_stride;
  a.v_stride = v_token_stride;
  a.cu_q = cu_seqlens_q;
  a.cu_k = cu_seqlens_k;
  a.num_seqs = num_seqs;
  a.Hq = num_q_heads;
  a.Hkv = num_kv_heads;
  a.Dqk = head_dim_qk;
  a.Dv = head_dim_v;
  a.scale_log2 = scale;       // the sigmoid takes natural exponents
  a.bias = bias;
  a.chunk = chunk > 0 ? chunk : 2147483647;
  a.gate = gate;
  a.gate_stride = gate_token_stride;
  a.status = status;
  return simple_launch<true>(a, max_seqlen_q, dtype, s);
}
