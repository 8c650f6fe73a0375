// Token shift: several mixes of the current and the previous token's row, each with a weight of its own per channel,
//
//     out[s][t, c] = h[t, c] + (h[t - 1, c] - h[t, c]) * mu[s, c]        s = 0 .. S - 1
//
// in float32, rounded once.  Before a row's first token of the step stands the last row of the request's step before, kept
// float32 in its state slot (zero for a new request), which is left holding this step's last row.  One pass reads h and
// writes all S mixes.  A step of decoded tokens only updates the state in the same launch (a thread owns a channel of a
// request); otherwise a second launch does it after every reader has finished.
#include "common.cuh"
using namespace arle;

constexpr int kShiftTokens = 8;       // consecutive tokens of the step a block takes

template <typename T, int VEC, bool SINGLE>
__global__ void __launch_bounds__(128) token_shift_kernel(const T* __restrict__ h, int h_stride, const float* __restrict__ mu, int S,
                                                          float* __restrict__ state, long slot_stride, const int* __restrict__ q_indptr,
                                                          const int* __restrict__ row_of_token, const int* __restrict__ state_slots,
                                                          T* __restrict__ out, size_t mix_stride, int num_tokens, int C) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= C) return;
  const int t0 = blockIdx.x * (SINGLE ? 1 : kShiftTokens), t1 = min(num_tokens, t0 + (SINGLE ? 1 : kShiftTokens));
  float before[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) before[i] = 0.f;
  for (int t = t0; t < t1; ++t) {
    const int r = row_of_token[t];
    float cur[VEC];
    load_vec<T, VEC>(h + (size_t)t * h_stride + c, cur);
    float* st = state + (size_t)state_slots[r] * slot_stride + c;
    if (t == q_indptr[r]) load_vec<float, VEC>(st, before);
    else if (t == t0) load_vec<T, VEC>(h + (size_t)(t - 1) * h_stride + c, before);
    for (int s = 0; s < S; ++s) {
      float m[VEC], y[VEC];
      load_vec<float, VEC>(mu + (size_t)s * C + c, m);
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = fmaf(before[i] - cur[i], m[i], cur[i]);
      store_vec<T, VEC>(out + (size_t)s * mix_stride + (size_t)t * C + c, y);
    }
    if (SINGLE) store_vec<float, VEC>(st, cur);
#pragma unroll
    for (int i = 0; i < VEC; ++i) before[i] = cur[i];
  }
}

template <typename T>
__global__ void token_shift_state_kernel(const T* __restrict__ h, int h_stride, float* __restrict__ state, long slot_stride,
                                         const int* __restrict__ q_indptr, const int* __restrict__ state_slots, int C) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C || q_indptr[r + 1] <= q_indptr[r]) return;
  state[(size_t)state_slots[r] * slot_stride + c] = to_f32(h[(size_t)(q_indptr[r + 1] - 1) * h_stride + c]);
}

namespace {

template <typename T>
int launch_shift(const void* h, int h_stride, const float* mu, int S, float* state, long slot_stride, const int* q_indptr, const int* row_of_token,
                 const int* state_slots, void* out, size_t mix_stride, int num_tokens, int R, int C, int single, cudaStream_t s) {
  const bool vec = C % 4 == 0 && h_stride % 4 == 0 && slot_stride % 4 == 0 && mix_stride % 4 == 0 && vec_aligned<4>(h, sizeof(T)) &&
                   vec_aligned<4>(mu, sizeof(float)) && vec_aligned<4>(state, sizeof(float)) && vec_aligned<4>(out, sizeof(T));
  const int per = 128 * (vec ? 4 : 1);
  dim3 grid(single ? num_tokens : (num_tokens + kShiftTokens - 1) / kShiftTokens, (C + per - 1) / per);
  if (grid.y > 65535) return ARLE_E_UNSUPPORTED;
  auto kernel = single ? (vec ? token_shift_kernel<T, 4, true> : token_shift_kernel<T, 1, true>)
                       : (vec ? token_shift_kernel<T, 4, false> : token_shift_kernel<T, 1, false>);
  launch_kernel(kernel, grid, dim3(128), 0, s, 1, (const T*)h, h_stride, mu, S, state, slot_stride, q_indptr, row_of_token, state_slots, (T*)out,
                mix_stride, num_tokens, C);
  if (!single)
    launch_kernel(token_shift_state_kernel<T>, dim3(R, (C + 127) / 128), dim3(128), 0, s, 1, (const T*)h, h_stride, state, slot_stride, q_indptr,
                  state_slots, C);
  return launch_status();
}

}  // namespace

// h [T, C] (row stride given) and out [S][T, C] (mix_stride elements from one mix to the next) in the activation type; mu float32
// [S, C]; the request's last row at state[slot * slot_stride + c], float32.  single: every row of the step has exactly one token.
ARLE_API int arle_token_shift(const void* h, int dtype, int h_stride, const float* mu, int S, float* state, long slot_stride,
                              const int* q_indptr, const int* row_of_token, const int* state_slots, void* out, long mix_stride, int num_tokens,
                              int R, int C, int single, cudaStream_t s) {
  if (num_tokens <= 0) return 0;
  if (C <= 0 || S <= 0 || R <= 0 || slot_stride < C || mix_stride < (long)num_tokens * C || (single && num_tokens != R)) return ARLE_E_BADARG;
  if (dtype == 0)
    return launch_shift<float>(h, h_stride, mu, S, state, slot_stride, q_indptr, row_of_token, state_slots, out, (size_t)mix_stride, num_tokens, R,
                               C, single, s);
  if (dtype == 1)
    return launch_shift<__nv_bfloat16>(h, h_stride, mu, S, state, slot_stride, q_indptr, row_of_token, state_slots, out, (size_t)mix_stride,
                                       num_tokens, R, C, single, s);
  return ARLE_E_BADARG;
}
