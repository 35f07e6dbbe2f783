// Linear maps of rows grouped by expert for every size and both dtypes (fp32 arithmetic): what the tensor-core grouped GEMMs do
// not take.  out[r] = X[r] . W_e^T with W [E, n_out, k], or with `glu` the clamped gated unit of the two halves of
// W [E, 2 n_out, k] = [gate | up], or max(., 0)^2 of the plain map.  Expert e owns rows [offsets[e-1], offsets[e]).
#include "common.cuh"

namespace b200 {
namespace {

constexpr int TM = 64, TN = 64, TK = 16;

struct GlArgs {
  const void* x;             // [R, k]
  const void* w;
  void* out;                 // [R, n_out]
  const int32_t* offsets;    // [E]
  int num_experts, n_out, k;
  int64_t rows;
  float limit, slope;
};

// One CTA per 64 rows of an expert and 64 output columns; 4 x 4 results per thread
template <typename T, int ACT>
__global__ void __launch_bounds__(256) grouped_linear_kernel(const GlArgs a) {
  constexpr bool GLU = ACT == B200_EXPERT_CLAMPED_GLU;
  constexpr int P = GLU ? 2 : 1;
  __shared__ float sx[TK][TM + 4], sw[P][TK][TN + 4];
  // the row tile: experts in order, ceil(rows / 64) tiles each
  int left = blockIdx.y, e = 0, row0 = 0, rows = 0;
  for (; e < a.num_experts; ++e) {
    row0 = e ? a.offsets[e - 1] : 0;
    rows = max(a.offsets[e] - row0, 0);
    const int tiles = (rows + TM - 1) / TM;
    if (left < tiles) break;
    left -= tiles;
  }
  if (e == a.num_experts) return;
  row0 += left * TM;
  rows = min(rows - left * TM, TM);
  if (row0 < 0 || row0 + static_cast<int64_t>(rows) > a.rows) return;      // offsets outside the rows
  const int n0 = blockIdx.x * TN, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* x = static_cast<const T*>(a.x) + static_cast<int64_t>(row0) * a.k;
  const T* w = static_cast<const T*>(a.w) + static_cast<int64_t>(e) * P * a.n_out * a.k;
  float acc[P][4][4] = {};
  for (int k0 = 0; k0 < a.k; k0 += TK) {
    for (int i = threadIdx.x; i < TM * TK; i += 256) {
      const int r = i / TK, c = i % TK;
      sx[c][r] = r < rows && k0 + c < a.k ? to_float<T>(x[static_cast<int64_t>(r) * a.k + k0 + c]) : 0.f;
    }
#pragma unroll
    for (int p = 0; p < P; ++p)
      for (int i = threadIdx.x; i < TN * TK; i += 256) {
        const int r = i / TK, c = i % TK;
        sw[p][c][r] = n0 + r < a.n_out && k0 + c < a.k
                          ? to_float<T>(w[(static_cast<int64_t>(p) * a.n_out + n0 + r) * a.k + k0 + c]) : 0.f;
      }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < TK; ++c) {
      float xv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) xv[i] = sx[c][ty * 4 + i];
#pragma unroll
      for (int p = 0; p < P; ++p)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float wv = sw[p][c][tx * 4 + j];
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[p][i][j] = fmaf(xv[i], wv, acc[p][i][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= rows) continue;
    T* o = static_cast<T*>(a.out) + (static_cast<int64_t>(row0) + r) * a.n_out;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= a.n_out) continue;
      if constexpr (GLU) o[n] = from_float<T>(clamped_glu_f(acc[0][i][j], acc[P - 1][i][j], a.limit, a.slope));
      else o[n] = from_float<T>(ACT == B200_EXPERT_SQUARED_RELU ? squared_relu_f(acc[0][i][j]) : acc[0][i][j]);
    }
  }
}

template <typename T>
void launch(const GlArgs& a, dim3 grid, int act, cudaStream_t s) {
  if (act == B200_EXPERT_CLAMPED_GLU) grouped_linear_kernel<T, B200_EXPERT_CLAMPED_GLU><<<grid, 256, 0, s>>>(a);
  else if (act == B200_EXPERT_SQUARED_RELU) grouped_linear_kernel<T, B200_EXPERT_SQUARED_RELU><<<grid, 256, 0, s>>>(a);
  else grouped_linear_kernel<T, B200_EXPERT_LINEAR><<<grid, 256, 0, s>>>(a);
}

}  // namespace

int grouped_linear_any_launch(const void* x, const void* w, void* out, const int32_t* expert_offsets, int64_t num_rows,
                              int num_experts, int n_out, int k_dim, int act, float limit, float slope, int32_t dtype,
                              cudaStream_t s) {
  const int64_t row_tiles = (num_rows + TM - 1) / TM + num_experts;      // at most this many
  const int col_tiles = (n_out + TN - 1) / TN;
  if (row_tiles > 65535) return B200_ERR_TOO_LARGE;
  GlArgs a{x, w, out, expert_offsets, num_experts, n_out, k_dim, num_rows, limit, slope};
  const dim3 grid(col_tiles, static_cast<unsigned>(row_tiles));
  if (dtype == B200_DTYPE_F32) launch<float>(a, grid, act, s);
  else launch<__nv_bfloat16>(a, grid, act, s);
  return launch_result();
}

}  // namespace b200
