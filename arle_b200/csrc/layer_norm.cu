// Layer norm (with a weight, without a bias): (x - mean) / sqrt(mean((x - mean)^2) + eps) * weight, statistics and arithmetic
// float32, in two places, and the short causal convolution that a block may put before its mixer.
//
//  * layernorm: the norm on a sublayer's input or at the model's ends, with the sum of a pending branch output in front of
//    it (the layer-norm twin of rmsnorm).
//  * branch_layernorm_add: the norm on a sublayer's OUTPUT, resid += LN(branch) * weight, with the rounded residual that the
//    next sublayer reads written in the same pass.  In a step of decoded tokens only it can also run the NEXT block's input
//    convolution on the new residual: a row has one token there, so all it needs besides is the request's own history.
//  * input_conv: out[t, c] = x[t, c] + sum_j w[j, c] * x[t - (taps - 1) + j, c] over the tokens of t's row, zeros before a
//    request's first token.  `w` comes transposed ([taps][C]) and with one added to its last row, so that the kernel forms
//    one sum.  The request's last taps - 1 inputs live in its state slot at conv_off + j * C + c, oldest first; x is the
//    float32 residual, so what the state keeps is unrounded.  A step of decoded tokens only updates the state in the same
//    launch (one thread owns a channel of a request); otherwise a second launch does it after every reader has finished.
//
// A thread meets the same numbers in all loops over a row, so the row in shared memory needs no barrier of its own.
#include "common.cuh"
using namespace arle;

// mean and 1 / standard deviation of the row in xs (this thread's numbers only are read; sum: this thread's part of the row's sum)
template <int VEC>
__device__ __forceinline__ void row_moments(const float* xs, float sum, int hidden, float eps, float* red, float& mean, float& inv) {
  mean = block_sum(sum, red) / (float)hidden;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < hidden; c += blockDim.x * VEC) {
    float x[VEC];
    load_vec<float, VEC>(xs + c, x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const float d = x[i] - mean;
      ss += d * d;
    }
  }
  inv = 1.0f / sqrtf(block_sum(ss, red) / (float)hidden + eps);
}

// For output row i (source row r = rows[i], or i): x = resid[r] (+ delta[r]); resid[r] = x when write_resid; out[i] = LN(x) * weight.
template <typename TA, int VEC>
__global__ void layernorm_kernel(float* __restrict__ resid, const TA* __restrict__ delta, const int* __restrict__ rows,
                                 const float* __restrict__ weight, TA* out, int hidden, float eps, int write_resid) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float xs[];
  __shared__ float red[33];
  const int i_out = blockIdx.x;
  const int r = rows ? rows[i_out] : i_out;
  float* xr = resid + (size_t)r * hidden;
  float sum = 0.f;
  for (int c = threadIdx.x * VEC; c < hidden; c += blockDim.x * VEC) {
    float x[VEC];
    load_vec<float, VEC>(xr + c, x);
    if (delta) {
      float d[VEC];
      load_vec<TA, VEC>(delta + (size_t)r * hidden + c, d);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] += d[i];
      if (write_resid) store_vec<float, VEC>(xr + c, x);
    }
    store_vec<float, VEC>(xs + c, x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) sum += x[i];
  }
  float mean, inv;
  row_moments<VEC>(xs, sum, hidden, eps, red, mean, inv);
  for (int c = threadIdx.x * VEC; c < hidden; c += blockDim.x * VEC) {
    float x[VEC], w[VEC];
    load_vec<float, VEC>(xs + c, x);
    load_vec<float, VEC>(weight + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = (x[i] - mean) * inv * w[i];
    store_vec<TA, VEC>(out + (size_t)i_out * hidden + c, x);
  }
}

// CONV: the next block's input convolution on the new residual, for steps in which every row has one token (row = token).
template <typename TA, int VEC, bool CONV>
__global__ void branch_layernorm_add_kernel(float* __restrict__ resid, const TA* __restrict__ branch, int branch_stride,
                                            const float* __restrict__ weight, TA* __restrict__ copy, int hidden, float eps,
                                            const float* __restrict__ conv_w, int taps, float* __restrict__ state, long slot_stride,
                                            const int* __restrict__ state_slots, TA* __restrict__ conv_out) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float xs[];
  __shared__ float red[33];
  const int t = blockIdx.x;
  float* xr = resid + (size_t)t * hidden;
  const TA* br = branch + (size_t)t * branch_stride;
  float sum = 0.f;
  for (int c = threadIdx.x * VEC; c < hidden; c += blockDim.x * VEC) {
    float x[VEC];
    load_vec<TA, VEC>(br + c, x);
    store_vec<float, VEC>(xs + c, x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) sum += x[i];
  }
  float mean, inv;
  row_moments<VEC>(xs, sum, hidden, eps, red, mean, inv);
  float* st = CONV ? state + (size_t)state_slots[t] * slot_stride : nullptr;
  for (int c = threadIdx.x * VEC; c < hidden; c += blockDim.x * VEC) {
    float x[VEC], b[VEC], w[VEC];
    load_vec<float, VEC>(xr + c, x);
    load_vec<float, VEC>(xs + c, b);
    load_vec<float, VEC>(weight + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] += (b[i] - mean) * inv * w[i];
    store_vec<float, VEC>(xr + c, x);
    if (copy) store_vec<TA, VEC>(copy + (size_t)t * hidden + c, x);
    if (CONV) {
      float acc[VEC], h[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) acc[i] = 0.f;
      for (int j = 0; j < taps - 1; ++j) {
        load_vec<float, VEC>(st + (size_t)j * hidden + c, h);
        load_vec<float, VEC>(conv_w + (size_t)j * hidden + c, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc[i] = fmaf(w[i], h[i], acc[i]);
        if (j > 0) store_vec<float, VEC>(st + (size_t)(j - 1) * hidden + c, h);
      }
      load_vec<float, VEC>(conv_w + (size_t)(taps - 1) * hidden + c, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) acc[i] = fmaf(w[i], x[i], acc[i]);
      if (taps > 1) store_vec<float, VEC>(st + (size_t)(taps - 2) * hidden + c, x);
      store_vec<TA, VEC>(conv_out + (size_t)t * hidden + c, acc);
    }
  }
}

constexpr int kConvTokens = 8;        // consecutive tokens of the step a block takes

// TAPS: the number of taps when it is known to the compiler (the weights then live in registers), 0: any number.
// SINGLE: every row has one token; the state is brought up to date by the thread that read it.
template <typename TO, int VEC, int TAPS, bool SINGLE>
__global__ void __launch_bounds__(128) input_conv_kernel(const float* __restrict__ x, const float* __restrict__ w, float* __restrict__ state,
                                                         long slot_stride, const int* __restrict__ q_indptr,
                                                         const int* __restrict__ row_of_token, const int* __restrict__ state_slots,
                                                         TO* __restrict__ out, int num_tokens, int C, int taps_arg) {
  pdl_launch_dependents();
  pdl_wait();
  const int taps = TAPS > 0 ? TAPS : taps_arg;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= C) return;
  constexpr int NW = TAPS > 0 ? TAPS : 1;
  float wr[NW][VEC];
  if (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < NW; ++j) load_vec<float, VEC>(w + (size_t)j * C + c, wr[j]);
  }
  const int t0 = blockIdx.x * (SINGLE ? 1 : kConvTokens), t1 = min(num_tokens, t0 + (SINGLE ? 1 : kConvTokens));
#pragma unroll
  for (int t = t0; t < t1; ++t) {
    const int r = row_of_token[t];
    const int beg = q_indptr[r];
    float* st = state ? state + (size_t)state_slots[r] * slot_stride + c : nullptr;
    float acc[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc[i] = 0.f;
#pragma unroll
    for (int j = 0; j < taps; ++j) {
      const int src = t - beg - (taps - 1) + j;             // index among this step's tokens of the row; below zero: in the state
      float v[VEC], wj[VEC];
      if (src >= 0) load_vec<float, VEC>(x + (size_t)(beg + src) * C + c, v);
      else load_vec<float, VEC>(st + (size_t)(src + taps - 1) * C, v);
      if (TAPS == 0) load_vec<float, VEC>(w + (size_t)j * C + c, wj);
#pragma unroll
      for (int i = 0; i < VEC; ++i) acc[i] = fmaf(TAPS > 0 ? wr[TAPS > 0 ? j : 0][i] : wj[i], v[i], acc[i]);
      if (SINGLE && j > 0) store_vec<float, VEC>(st + (size_t)(j - 1) * C, v);
    }
    store_vec<TO, VEC>(out + (size_t)t * C + c, acc);
  }
}

__global__ void input_conv_state_kernel(const float* __restrict__ x, float* __restrict__ state, long slot_stride,
                                        const int* __restrict__ q_indptr, const int* __restrict__ state_slots, int C, int taps) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int beg = q_indptr[r], n = q_indptr[r + 1] - beg;
  if (n <= 0) return;
  float* st = state + (size_t)state_slots[r] * slot_stride + c;
  for (int j = 0; j < taps - 1; ++j) {                 // ascending: place j is written after place j + n was read
    const int src = n + j - (taps - 1);
    st[(size_t)j * C] = src >= 0 ? x[(size_t)(beg + src) * C + c] : st[(size_t)(src + taps - 1) * C];
  }
}

namespace {

// Threads a row: with few rows (a decode step) as many as the row has accesses, so that every loop over it is one round.
int row_threads(int hidden, int per, int rows) {
  if (rows <= 296) {
    const int n = ((hidden + per - 1) / per + 31) / 32 * 32;
    return n < 64 ? 64 : (n > 1024 ? 1024 : n);
  }
  return hidden >= 2048 * per ? 512 : (hidden >= 512 * per ? 256 : 128);
}

template <typename TA>
int launch_layernorm(float* resid, const void* delta, const int* rows, const float* weight, void* out, int n_out, int hidden, float eps,
                     int write_resid, cudaStream_t s) {
  const size_t smem = (size_t)hidden * sizeof(float);
  const bool vec = hidden % 4 == 0 && vec_aligned<4>(resid, sizeof(float)) && vec_aligned<4>(weight, sizeof(float)) &&
                   vec_aligned<4>(delta, sizeof(TA)) && vec_aligned<4>(out, sizeof(TA));
  auto kernel = vec ? layernorm_kernel<TA, 4> : layernorm_kernel<TA, 1>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  launch_kernel(kernel, dim3(n_out), dim3(row_threads(hidden, vec ? 4 : 1, n_out)), smem, s, 1, resid, (const TA*)delta, rows, weight, (TA*)out, hidden,
                eps, write_resid);
  return launch_status();
}

template <typename TA>
int launch_branch_layernorm(float* resid, const void* branch, int branch_stride, const float* weight, void* copy, int num_tokens, int hidden,
                            float eps, const float* conv_w, int taps, float* state, long slot_stride, const int* state_slots, void* conv_out,
                            cudaStream_t s) {
  const size_t smem = (size_t)hidden * sizeof(float);
  const bool vec = hidden % 4 == 0 && branch_stride % 4 == 0 && slot_stride % 4 == 0 && vec_aligned<4>(resid, sizeof(float)) &&
                   vec_aligned<4>(weight, sizeof(float)) && vec_aligned<4>(branch, sizeof(TA)) && vec_aligned<4>(copy, sizeof(TA)) &&
                   vec_aligned<4>(conv_w, sizeof(float)) && vec_aligned<4>(state, sizeof(float)) && vec_aligned<4>(conv_out, sizeof(TA));
  auto kernel = conv_w ? (vec ? branch_layernorm_add_kernel<TA, 4, true> : branch_layernorm_add_kernel<TA, 1, true>)
                       : (vec ? branch_layernorm_add_kernel<TA, 4, false> : branch_layernorm_add_kernel<TA, 1, false>);
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  launch_kernel(kernel, dim3(num_tokens), dim3(row_threads(hidden, vec ? 4 : 1, num_tokens)), smem, s, 1, resid, (const TA*)branch, branch_stride, weight,
                (TA*)copy, hidden, eps, conv_w, taps, state, slot_stride, state_slots, (TA*)conv_out);
  return launch_status();
}

template <typename TO, int VEC, bool SINGLE>
int launch_input_conv(const float* x, const float* w, float* state, long slot_stride, const int* q_indptr, const int* row_of_token,
                      const int* state_slots, void* out, int num_tokens, int R, int C, int taps, cudaStream_t s) {
  const int per = 128 * VEC;
  dim3 grid(SINGLE ? num_tokens : (num_tokens + kConvTokens - 1) / kConvTokens, (C + per - 1) / per);
  if (grid.y > 65535) return ARLE_E_UNSUPPORTED;
  auto kernel = taps == 2 ? input_conv_kernel<TO, VEC, 2, SINGLE>
              : taps == 3 ? input_conv_kernel<TO, VEC, 3, SINGLE>
              : taps == 4 ? input_conv_kernel<TO, VEC, 4, SINGLE> : input_conv_kernel<TO, VEC, 0, SINGLE>;
  launch_kernel(kernel, grid, dim3(128), 0, s, 1, x, w, state, slot_stride, q_indptr, row_of_token, state_slots, (TO*)out, num_tokens, C, taps);
  if (!SINGLE && taps > 1)
    launch_kernel(input_conv_state_kernel, dim3(R, (C + 127) / 128), dim3(128), 0, s, 1, x, state, slot_stride, q_indptr, state_slots, C, taps);
  return launch_status();
}

}  // namespace

// resid float32 [*, hidden] contiguous; delta [*, hidden] and out [n_out, hidden] contiguous in the activation type (out may be
// resid itself in float32); weight float32 [hidden].
ARLE_API int arle_layernorm(float* resid, const void* delta, const int* rows, const float* weight, void* out, int dtype, int n_out, int hidden,
                            float eps, int write_resid, cudaStream_t s) {
  if (n_out <= 0) return 0;
  if (hidden <= 0 || !weight || !out) return ARLE_E_BADARG;
  if ((size_t)hidden * sizeof(float) > 160 * 1024) return ARLE_E_UNSUPPORTED;
  if (dtype == 0) return launch_layernorm<float>(resid, delta, rows, weight, out, n_out, hidden, eps, write_resid, s);
  if (dtype == 1) return launch_layernorm<__nv_bfloat16>(resid, delta, rows, weight, out, n_out, hidden, eps, write_resid, s);
  return ARLE_E_BADARG;
}

// resid float32 [T, hidden] contiguous; branch [T, hidden] in the activation type (row stride given); copy [T, hidden] contiguous or
// null.  conv_w float32 [taps, hidden] (null: no convolution): then token t is row t of the step, its history is at
// state[state_slots[t] * slot_stride + j * hidden + c], and conv_out [T, hidden] gets the convolved residual.
ARLE_API int arle_branch_layernorm_add(float* resid, const void* branch, int branch_stride, const float* weight, void* copy, int dtype,
                                       int num_tokens, int hidden, float eps, const float* conv_w, int taps, float* state, long slot_stride,
                                       const int* state_slots, void* conv_out, cudaStream_t s) {
  if (num_tokens <= 0) return 0;
  if (hidden <= 0 || !branch || !weight) return ARLE_E_BADARG;
  if (conv_w && (taps < 1 || !conv_out || !state_slots || (taps > 1 && (!state || slot_stride < (long)hidden * (taps - 1))))) return ARLE_E_BADARG;
  if ((size_t)hidden * sizeof(float) > 160 * 1024) return ARLE_E_UNSUPPORTED;
  if (dtype == 0)
    return launch_branch_layernorm<float>(resid, branch, branch_stride, weight, copy, num_tokens, hidden, eps, conv_w, taps, state, slot_stride,
                                          state_slots, conv_out, s);
  if (dtype == 1)
    return launch_branch_layernorm<__nv_bfloat16>(resid, branch, branch_stride, weight, copy, num_tokens, hidden, eps, conv_w, taps, state,
                                                  slot_stride, state_slots, conv_out, s);
  return ARLE_E_BADARG;
}

// x float32 [T, C] contiguous, w float32 [taps, C], out [T, C] contiguous (out_dtype 0 float32, 1 bfloat16).  single: every row of the
// step has exactly one token.
ARLE_API int arle_input_conv(const float* x, const float* w, float* state, long slot_stride, const int* q_indptr, const int* row_of_token,
                             const int* state_slots, void* out, int out_dtype, int num_tokens, int R, int C, int taps, int single,
                             cudaStream_t s) {
  if (num_tokens <= 0) return 0;
  if (C <= 0 || taps <= 0 || R <= 0 || (out_dtype != 0 && out_dtype != 1)) return ARLE_E_BADARG;
  if (taps > 1 && (!state || slot_stride < (long)C * (taps - 1))) return ARLE_E_BADARG;
  if (single && num_tokens != R) return ARLE_E_BADARG;
  const size_t eb = out_dtype == 0 ? sizeof(float) : sizeof(__nv_bfloat16);
  const bool vec = C % 4 == 0 && slot_stride % 4 == 0 && vec_aligned<4>(x, sizeof(float)) && vec_aligned<4>(w, sizeof(float)) &&
                   vec_aligned<4>(state, sizeof(float)) && vec_aligned<4>(out, eb);
#define ARLE_ICONV(TO, V, S) \
  return launch_input_conv<TO, V, S>(x, w, state, slot_stride, q_indptr, row_of_token, state_slots, out, num_tokens, R, C, taps, s)
  if (out_dtype == 0) {
    if (vec && single) ARLE_ICONV(float, 4, true);
    if (vec) ARLE_ICONV(float, 4, false);
    if (single) ARLE_ICONV(float, 1, true);
    ARLE_ICONV(float, 1, false);
  }
  if (vec && single) ARLE_ICONV(__nv_bfloat16, 4, true);
  if (vec) ARLE_ICONV(__nv_bfloat16, 4, false);
  if (single) ARLE_ICONV(__nv_bfloat16, 1, true);
  ARLE_ICONV(__nv_bfloat16, 1, false);
#undef ARLE_ICONV
}
