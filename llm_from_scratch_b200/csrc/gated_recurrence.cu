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
// recurrence_step_kernel   one CTA per (sequence, head), tokens in order: decode, and sizes the scan does not take.
//
// recurrence_scan_kernel   prompts and portions, cut into segments of seg_len tokens that run in parallel.  A segment
//                          maps its entry state to D * S + P (D: product of its forget gates, P: its own writes), so
//   pass 1 (scan, LOCAL)   P and D of every segment but the last of its sequence, from the zero state
//   pass 2 (chain)         the entry state of every segment, segment after segment
//   pass 3 (scan)          the outputs from the entry states; the last segment leaves the state in the pool
//                          A sequence of one segment needs pass 3 only.  A thread keeps R key channels x C value
//                          columns of the state in registers and walks the tokens; q / f / k / v of 16 tokens at a
//                          time sit in shared memory as fp32, the RG threads of a column reduce their part of o by
//                          shuffles, and 16 tokens of outputs are normed together.
#include "sequences.cuh"

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

// forget gate and write gate of one channel
__device__ __forceinline__ void gates(float z, float lower, float* f, float* k) {
  const float open = 1.f - lower;
  float s, n;
  sigmoids(z, &s, &n);
  *f = lower + open * s;
  *k = open * n;
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
      sq[i] = silu_f(qv);
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
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(smem)) != cudaSuccess)
    return B200_ERR_LAUNCH;
  kern<<<dim3(a.H, n), kStepThreads, smem, s>>>(a, CL);
  return launch_result();
}

// ---------------------------------------------------------------------------------------------
// Segmented scan
// ---------------------------------------------------------------------------------------------
constexpr int kBlockTokens = 16;     // tokens staged at a time

struct ScanArgs {
  float* seg_state;          // [segments, H, dk, dv]  pass 1: P, after pass 2: entry state
  float* seg_decay;          // [segments, H, dk]      pass 1: D
  int n, seg_len;
  bool async;                // 16-byte copies are possible
};

// RG: threads that share a column group
template <typename T, int R, int C, int RG, bool LOCAL>
__global__ void __launch_bounds__(512, 1) recurrence_scan_kernel(const RecArgs a, const ScanArgs sc) {
  constexpr int DK = R * RG, P = R / 2;
  extern __shared__ __align__(16) float sm[];
  const int dk = a.dk, dv = a.dv, head = blockIdx.y, number = blockIdx.x;
  int seq, index;
  if (!find_segment(a.cu_q, sc.n, sc.seg_len, number, &seq, &index)) return;
  SeqInfo info;
  if (!sequence_info(a, seq, &info)) return;
  const int segments = (info.len + sc.seg_len - 1) / sc.seg_len;
  const bool last = index == segments - 1;
  if (LOCAL && last) return;                       // its own map is never needed
  const int tok_lo = index * sc.seg_len, ntok = min(sc.seg_len, info.len - tok_lo);

  float* sf = sm;                                  // [kBlockTokens, DK]
  float* sk = sf + kBlockTokens * DK;
  float* sq = sk + kBlockTokens * DK;              // outputs only
  float* sv = sq + (LOCAL ? 0 : kBlockTokens * DK);
  float* so = sv + 2 * kBlockTokens * dv;          // [kBlockTokens, dv], outputs only
  // rows of the projection as they are, two blocks: [2][kBlockTokens][f | (q) | v]
  T* raw = reinterpret_cast<T*>(so + (LOCAL ? 0 : kBlockTokens * dv));
  const int at_q = dk, at_v = LOCAL ? dk : 2 * dk, raw_row = at_v + dv;
  const int tid = threadIdx.x, threads = blockDim.x, rg = tid & (RG - 1), c0 = (tid / RG) * C;
  const bool cols = c0 < dv;                       // dv is a multiple of 4: a float4 is in or out as a whole

  // pair p of this thread: rows row(p), row(p) + 1
  auto row = [&](int p) { return (p >> 1) * (4 * RG) + rg * 4 + (p & 1) * 2; };
  f32x2 S[P][C], D[P];
  const int64_t head_state = static_cast<int64_t>(dk) * dv;
  float* pool = a.state + (info.slot * a.H + head) * head_state;
  float* mine = sc.seg_state + (static_cast<int64_t>(number) * a.H + head) * head_state;
  const float* from = LOCAL ? nullptr : segments > 1 ? mine : info.fresh ? nullptr : pool;
#pragma unroll
  for (int p = 0; p < P; ++p) {
    D[p] = pack2(1.f, 1.f);
#pragma unroll
    for (int c = 0; c < C; c += 4) {
      float4 x0 = make_float4(0.f, 0.f, 0.f, 0.f), x1 = x0;
      if (from != nullptr && c0 + c < dv) {
        if (row(p) < dk) x0 = *reinterpret_cast<const float4*>(from + static_cast<int64_t>(row(p)) * dv + c0 + c);
        if (row(p) + 1 < dk) x1 = *reinterpret_cast<const float4*>(from + static_cast<int64_t>(row(p) + 1) * dv + c0 + c);
      }
      S[p][c] = pack2(x0.x, x1.x);
      S[p][c + 1] = pack2(x0.y, x1.y);
      S[p][c + 2] = pack2(x0.z, x1.z);
      S[p][c + 3] = pack2(x0.w, x1.w);
    }
  }

  auto fetch = [&](int b) {                        // block b of the segment -> raw
    const int nb = min(kBlockTokens, ntok - b);
    T* dst = raw + ((b / kBlockTokens) & 1) * kBlockTokens * raw_row;
    const int64_t tok = info.tok0 + tok_lo + b;
    constexpr int E = 16 / sizeof(T);
    const int w = sc.async ? E : 1, ck = dk / w, cv = dv / w, per = (LOCAL ? ck : 2 * ck) + cv;
    for (int i = tid; i < nb * per; i += threads) {
      const int t = i / per, c = i - t * per;
      const int64_t off = (tok + t) * a.stride;
      const T* src;
      int to;
      if (c < ck) {
        src = static_cast<const T*>(a.f) + off + head * dk + c * w;
        to = c * w;
      } else if (!LOCAL && c < 2 * ck) {
        src = static_cast<const T*>(a.q) + off + head * dk + (c - ck) * w;
        to = at_q + (c - ck) * w;
      } else {
        const int cc = c - (LOCAL ? ck : 2 * ck);
        src = static_cast<const T*>(a.v) + off + head * dv + cc * w;
        to = at_v + cc * w;
      }
      if (sc.async) cp_async16(smem_u32(dst + t * raw_row + to), src, 16);
      else dst[t * raw_row + to] = *src;
    }
    cp_async_commit();
  };
  fetch(0);
  for (int b = 0; b < ntok; b += kBlockTokens) {
    const int nb = min(kBlockTokens, ntok - b);
    const int64_t tok = info.tok0 + tok_lo + b;
    cp_async_wait<0>();
    __syncthreads();
    const T* rp = raw + ((b / kBlockTokens) & 1) * kBlockTokens * raw_row;
    if (b + kBlockTokens < ntok) fetch(b + kBlockTokens);
    for (int i = tid; i < nb * DK; i += threads) {
      const int t = i / DK, d = i % DK;
      float f = 1.f, k = 0.f, q = 0.f;
      if (d < dk) {
        gates(to_float<T>(rp[t * raw_row + d]) + __ldg(a.f_bias + head * dk + d), __ldg(a.lower + head * dk + d), &f, &k);
        if (!LOCAL) q = silu_f(to_float<T>(rp[t * raw_row + at_q + d]));
      }
      sf[i] = f;
      sk[i] = k;
      if (!LOCAL) sq[i] = q;
    }
    for (int i = tid; i < nb * dv; i += threads) {
      const int t = i / dv, d = i - t * dv;
      const float x = to_float<T>(rp[t * raw_row + at_v + d]);
      *reinterpret_cast<float2*>(sv + 2 * i) = make_float2(x, x);       // both halves of a packed operand
    }
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < nb; ++t) {
      f32x2 f[P], k[P], q[P], v[C];
#pragma unroll
      for (int i = 0; i < P; i += 2) {
        const int at = t * DK + (i >> 1) * (4 * RG) + rg * 4;
        const ulonglong2 fx = *reinterpret_cast<const ulonglong2*>(sf + at), kx = *reinterpret_cast<const ulonglong2*>(sk + at);
        f[i] = fx.x, f[i + 1] = fx.y, k[i] = kx.x, k[i + 1] = kx.y;
        if (!LOCAL) {
          const ulonglong2 qx = *reinterpret_cast<const ulonglong2*>(sq + at);
          q[i] = qx.x, q[i + 1] = qx.y;
        }
      }
#pragma unroll
      for (int c = 0; c < C; c += 2) {
        // columns past the last one (dv not a multiple of C) repeat column 0: never stored
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(sv + 2 * (t * dv + (c0 + c < dv ? c0 + c : 0)));
        v[c] = x.x;
        v[c + 1] = x.y;
      }
      float o[C];
#pragma unroll
      for (int c = 0; c < C; ++c) {
        f32x2 acc = 0;
#pragma unroll
        for (int p = 0; p < P; ++p) {
          S[p][c] = fma2(f[p], S[p][c], mul2(k[p], v[c]));
          if (!LOCAL) acc = fma2(q[p], S[p][c], acc);
        }
        const float2 h = unpack2(acc);
        o[c] = h.x + h.y;
      }
      if constexpr (LOCAL) {
#pragma unroll
        for (int p = 0; p < P; ++p) D[p] = mul2(D[p], f[p]);
      } else {
        // sum over the row groups; every step a lane keeps half of the columns it still has
        int col = 0;
#pragma unroll
        for (int half = C / 2, step = RG / 2; half >= 1; half >>= 1, step >>= 1) {
          const bool up = rg & step;
#pragma unroll
          for (int c = 0; c < half; ++c) {
            const float send = up ? o[c] : o[c + half], keep = up ? o[c + half] : o[c];
            o[c] = keep + __shfl_xor_sync(0xffffffffu, send, step);
          }
          if (up) col += half;
        }
        constexpr int kLeft = RG / C;        // lanes that still share one column
#pragma unroll
        for (int step = kLeft / 2; step >= 1; step >>= 1) o[0] += __shfl_xor_sync(0xffffffffu, o[0], step);
        if (cols && (rg & (kLeft - 1)) == 0) so[t * dv + c0 + col] = o[0];
      }
    }
    if constexpr (!LOCAL) {
      __syncthreads();
      const int lane = tid & 31;
      for (int t = tid >> 5; t < nb; t += threads >> 5) {
        float ss = 0.f;
        for (int d = lane; d < dv; d += 32) ss += so[t * dv + d] * so[t * dv + d];
        const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(dv) + a.eps);
        T* op = static_cast<T*>(a.out) + ((tok + t) * a.H + head) * dv;
        for (int d = lane; d < dv; d += 32) op[d] = from_float<T>(so[t * dv + d] * inv * a.norm_w[d]);
      }
    }
  }
  if (LOCAL && tid < RG) {
    float* dec = sc.seg_decay + (static_cast<int64_t>(number) * a.H + head) * dk;
#pragma unroll
    for (int p = 0; p < P; ++p) {
      const float2 x = unpack2(D[p]);
      if (row(p) < dk) dec[row(p)] = x.x;
      if (row(p) + 1 < dk) dec[row(p) + 1] = x.y;
    }
  }
  float* to = LOCAL ? mine : last ? pool : nullptr;
  if (to != nullptr) {
#pragma unroll
    for (int p = 0; p < P; ++p)
#pragma unroll
      for (int c = 0; c < C; c += 4) {
        if (c0 + c >= dv) continue;
        const float2 x0 = unpack2(S[p][c]), x1 = unpack2(S[p][c + 1]), x2 = unpack2(S[p][c + 2]), x3 = unpack2(S[p][c + 3]);
        float* at = to + static_cast<int64_t>(row(p)) * dv + c0 + c;
        if (row(p) < dk) *reinterpret_cast<float4*>(at) = make_float4(x0.x, x1.x, x2.x, x3.x);
        if (row(p) + 1 < dk) *reinterpret_cast<float4*>(at + dv) = make_float4(x0.y, x1.y, x2.y, x3.y);
      }
  }
}

// Entry states: one thread carries four consecutive state elements of one (sequence, head) through its segments.
__global__ void __launch_bounds__(256) recurrence_chain_kernel(const RecArgs a, const ScanArgs sc) {
  __shared__ int s_first;
  const int seq = blockIdx.z, head = blockIdx.y;
  SeqInfo info;
  if (!sequence_info(a, seq, &info)) return;
  const int segments = (info.len + sc.seg_len - 1) / sc.seg_len;
  if (segments <= 1) return;
  if (threadIdx.x < 32) {
    const int first = first_segment(a.cu_q, sc.seg_len, seq);
    if (threadIdx.x == 0) s_first = first;
  }
  __syncthreads();
  const int64_t per_head = static_cast<int64_t>(a.dk) * a.dv;
  const int64_t e = (static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x) * 4;
  if (e >= per_head) return;
  const int r = static_cast<int>(e / a.dv);
  float4 S = info.fresh ? make_float4(0.f, 0.f, 0.f, 0.f)
                        : *reinterpret_cast<const float4*>(a.state + (info.slot * a.H + head) * per_head + e);
  float* st = sc.seg_state + (static_cast<int64_t>(s_first) * a.H + head) * per_head + e;
  const float* dec = sc.seg_decay + (static_cast<int64_t>(s_first) * a.H + head) * a.dk + r;
  const int64_t st_step = a.H * per_head, dec_step = static_cast<int64_t>(a.H) * a.dk;
  constexpr int U = 8;                               // loads in flight
  for (int i = 0; i < segments - 1; i += U) {
    float4 p[U];
    float d[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i + u < segments - 1) {
        p[u] = *reinterpret_cast<const float4*>(st + u * st_step);
        d[u] = dec[u * dec_step];
      }
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i + u < segments - 1) {
        *reinterpret_cast<float4*>(st) = S;
        S.x = fmaf(d[u], S.x, p[u].x);
        S.y = fmaf(d[u], S.y, p[u].y);
        S.z = fmaf(d[u], S.z, p[u].z);
        S.w = fmaf(d[u], S.w, p[u].w);
        st += st_step;
        dec += dec_step;
      }
  }
  *reinterpret_cast<float4*>(st) = S;
}

// sizes the scan takes: columns of all threads of a CTA, rows in registers
inline bool scan_shape(int dk, int dv) { return dv % 4 == 0 && ((dk <= 128 && dv <= 256) || (dk <= 256 && dv <= 128)); }

inline int scan_seg_len(int64_t tokens, int H) {
  // long enough to amortise the passes over the states, short enough for two waves of CTAs
  const int64_t want = tokens * H / 600;
  return want >= 128 ? 128 : want >= 64 ? 64 : 32;
}

template <typename T, int R, int C, int RG>
int launch_scan(const RecArgs& a, const ScanArgs& sc, int64_t segments, bool chained, cudaStream_t s) {
  const int groups = (a.dv + C - 1) / C, threads = (groups * RG + 31) / 32 * 32;
  auto local = recurrence_scan_kernel<T, R, C, RG, true>;
  auto full = recurrence_scan_kernel<T, R, C, RG, false>;
  const size_t one = size_t(kBlockTokens) * R * RG * sizeof(float), v = size_t(kBlockTokens) * a.dv * sizeof(float);
  const size_t smem_local = 2 * one + 2 * v + 2 * kBlockTokens * size_t(a.dk + a.dv) * sizeof(T);
  const size_t smem_full = 3 * one + 3 * v + 2 * kBlockTokens * size_t(2 * a.dk + a.dv) * sizeof(T);
  if (smem_full > 40 * 1024 &&
      (cudaFuncSetAttribute(local, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem_local)) != cudaSuccess ||
       cudaFuncSetAttribute(full, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem_full)) != cudaSuccess))
    return B200_ERR_LAUNCH;
  const dim3 grid(static_cast<unsigned>(segments), a.H);
  if (chained) {
    local<<<grid, threads, smem_local, s>>>(a, sc);
    const int64_t units = static_cast<int64_t>(a.dk) * a.dv / 4;
    recurrence_chain_kernel<<<dim3(static_cast<unsigned>((units + 255) / 256), a.H, sc.n), 256, 0, s>>>(a, sc);
  }
  full<<<grid, threads, smem_full, s>>>(a, sc);
  return launch_result();
}

template <typename T>
int dispatch_scan(const RecArgs& a, const ScanArgs& sc, int64_t segments, bool chained, cudaStream_t s) {
  if (a.dk <= 64) return launch_scan<T, 8, 4, 8>(a, sc, segments, chained, s);
  if (a.dk <= 128) return launch_scan<T, 8, 8, 16>(a, sc, segments, chained, s);
  return launch_scan<T, 16, 4, 16>(a, sc, segments, chained, s);
}

}  // namespace
}  // namespace b200

extern "C" size_t b200_gated_recurrence_workspace_bytes(int32_t num_seqs, int64_t total_tokens, int32_t max_seqlen_q,
                                                        int32_t num_heads, int32_t dim_k, int32_t dim_v) {
  using namespace b200;
  if (num_seqs <= 0 || total_tokens <= 0 || max_seqlen_q <= 1 || num_heads <= 0 || !scan_shape(dim_k, dim_v)) return 0;
  const int seg = scan_seg_len(total_tokens, num_heads);
  if (max_seqlen_q <= seg) return 0;                      // every sequence is one segment
  const size_t segments = static_cast<size_t>(total_tokens / seg + num_seqs);
  return segments * num_heads * (static_cast<size_t>(dim_k) * dim_v + dim_k) * sizeof(float);
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
  if (cu_seqlens_q && vec && max_seqlen_q > 1 && scan_shape(dim_k, dim_v)) {
    ScanArgs sc{};
    sc.n = num_seqs;
    sc.seg_len = scan_seg_len(total_tokens, num_heads);
    const int64_t es = dtype == B200_DTYPE_F32 ? 4 : 2;
    sc.async = dim_k * es % 16 == 0 && dim_v * es % 16 == 0 && token_stride * es % 16 == 0 && aligned16(q) &&
               aligned16(f) && aligned16(v);
    const int64_t segments = total_tokens / sc.seg_len + num_seqs;
    const bool chained = max_seqlen_q > sc.seg_len;
    if (chained) {
      if (!workspace || workspace_bytes < b200_gated_recurrence_workspace_bytes(num_seqs, total_tokens, max_seqlen_q,
                                                                               num_heads, dim_k, dim_v))
        return B200_ERR_WORKSPACE;
      sc.seg_state = static_cast<float*>(workspace);
      sc.seg_decay = sc.seg_state + static_cast<size_t>(segments) * num_heads * dim_k * dim_v;
    }
    return dtype == B200_DTYPE_F32 ? dispatch_scan<float>(a, sc, segments, chained, s)
                                   : dispatch_scan<__nv_bfloat16>(a, sc, segments, chained, s);
  }
  return dtype == B200_DTYPE_F32 ? launch_step<float>(a, num_seqs, vec, s)
                                 : launch_step<__nv_bfloat16>(a, num_seqs, vec, s);
}
