// Token embedding: residual[t, :] = float32(table[ids[t], :]) * scale (scale 1 for most models), plus float32(pos_table[p, :]) for
// a token at position p in models with a learned position table; out2 (may be null) gets the same rows once more, for models that
// add them to the residual again later.
// A negative id is a placeholder for "the token this request sampled last": it is read
// from last_token[slot_of_token[t]], which the sampling kernels write on the device, so
// that a decode step can be launched before the host has seen the previous step's tokens.
// The residual stream is kept in 32-bit in both engine precisions, so the table
// row is widened here once.  An id outside [0, vocab) writes zeros and raises the
// error flag instead of reading out of bounds (the host checks ids first); so does a position outside the position table.
#include "common.cuh"
using namespace arle;

template <typename T>
__global__ void embedding_kernel(const int* __restrict__ ids, const T* __restrict__ table,
                                 float* __restrict__ out, int hidden, int vocab,
                                 int* __restrict__ err, const int* __restrict__ last_token,
                                 const int* __restrict__ slot_of_token, float scale, const T* __restrict__ pos_table, int num_pos,
                                 const int* __restrict__ positions, float* __restrict__ out2) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 && last_token) id = last_token[slot_of_token[t]];
  float* o = out + (size_t)t * hidden;
  float* o2 = out2 ? out2 + (size_t)t * hidden : nullptr;
  const int p = pos_table ? positions[t] : 0;
  if (id < 0 || id >= vocab || p < 0 || p >= num_pos) {
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
      o[i] = 0.f;
      if (o2) o2[i] = 0.f;
    }
    if (threadIdx.x == 0 && err) atomicExch(err, 1);
    return;
  }
  const T* row = table + (size_t)id * hidden;
  const T* prow = pos_table ? pos_table + (size_t)p * hidden : nullptr;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    float v = to_f32(row[i]) * scale;
    if (prow) v += to_f32(prow[i]);
    o[i] = v;
    if (o2) o2[i] = v;
  }
}

// Eight table elements per thread and step (16-byte loads of bfloat16 rows).
__global__ void embedding_bf16_vec_kernel(const int* __restrict__ ids, const __nv_bfloat16* __restrict__ table,
                                          float* __restrict__ out, int hidden, int vocab, int* __restrict__ err,
                                          const int* __restrict__ last_token, const int* __restrict__ slot_of_token, float scale,
                                          const __nv_bfloat16* __restrict__ pos_table, int num_pos, const int* __restrict__ positions,
                                          float* __restrict__ out2) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 && last_token) id = last_token[slot_of_token[t]];
  const int p = pos_table ? positions[t] : 0;
  const bool bad = id < 0 || id >= vocab || p < 0 || p >= num_pos;
  if (bad && threadIdx.x == 0 && err) atomicExch(err, 1);
  const uint4* row = reinterpret_cast<const uint4*>(table + (size_t)(bad ? 0 : id) * hidden);
  float4* o = reinterpret_cast<float4*>(out + (size_t)t * hidden);
  for (int c = threadIdx.x; c < hidden / 8; c += blockDim.x) {
    uint4 u = make_uint4(0, 0, 0, 0);
    if (!bad) u = row[c];
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
    float4 a = make_float4(__low2float(h[0]) * scale, __high2float(h[0]) * scale, __low2float(h[1]) * scale, __high2float(h[1]) * scale);
    float4 b = make_float4(__low2float(h[2]) * scale, __high2float(h[2]) * scale, __low2float(h[3]) * scale, __high2float(h[3]) * scale);
    if (pos_table) {
      const uint4 w = bad ? make_uint4(0, 0, 0, 0) : reinterpret_cast<const uint4*>(pos_table + (size_t)p * hidden)[c];
      const __nv_bfloat162* g = reinterpret_cast<const __nv_bfloat162*>(&w);
      a.x += __low2float(g[0]), a.y += __high2float(g[0]), a.z += __low2float(g[1]), a.w += __high2float(g[1]);
      b.x += __low2float(g[2]), b.y += __high2float(g[2]), b.z += __low2float(g[3]), b.w += __high2float(g[3]);
    }
    o[2 * c] = a;
    o[2 * c + 1] = b;
    if (out2) {
      float4* o2 = reinterpret_cast<float4*>(out2 + (size_t)t * hidden);
      o2[2 * c] = a;
      o2[2 * c + 1] = b;
    }
  }
}

// pos_table (may be null): [num_pos, hidden] in the table's type, rows chosen by positions.
ARLE_API int arle_embedding(const int* ids, const void* table, int table_dtype, float* out,
                            int num_tokens, int hidden, int vocab, int* err, const int* last_token,
                            const int* slot_of_token, float scale, const void* pos_table, int num_pos, const int* positions,
                            float* out2, cudaStream_t s) {
  if (last_token && !slot_of_token) return ARLE_E_BADARG;
  if (pos_table ? (!positions || num_pos <= 0) : false) return ARLE_E_BADARG;
  if (!pos_table) num_pos = 1;              // position 0 stands for "none"
  if (num_tokens <= 0) return 0;
  if (hidden <= 0 || vocab <= 0) return ARLE_E_BADARG;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == 1 && hidden % 8 == 0 && ((uintptr_t)table & 15) == 0 && ((uintptr_t)out & 15) == 0 && ((uintptr_t)pos_table & 15) == 0 &&
      ((uintptr_t)out2 & 15) == 0) {
    int th = hidden / 8;
    th = th <= 32 ? 32 : (th <= 64 ? 64 : (th <= 128 ? 128 : (th <= 256 ? 256 : 512)));
    launch_kernel(embedding_bf16_vec_kernel, dim3(num_tokens), dim3(th), 0, s, 1, ids, (const __nv_bfloat16*)table, out, hidden, vocab, err, last_token, slot_of_token, scale,
                  (const __nv_bfloat16*)pos_table, num_pos, positions, out2);
    return launch_status();
  }
  if (table_dtype == 0)
    launch_kernel(embedding_kernel<float>, dim3(num_tokens), dim3(threads), 0, s, 1, ids, (const float*)table, out, hidden, vocab, err, last_token, slot_of_token, scale,
                  (const float*)pos_table, num_pos, positions, out2);
  else if (table_dtype == 1)
    launch_kernel(embedding_kernel<__nv_bfloat16>, dim3(num_tokens), dim3(threads), 0, s, 1, ids, (const __nv_bfloat16*)table, out, hidden, vocab, err, last_token, slot_of_token, scale,
                  (const __nv_bfloat16*)pos_table, num_pos, positions, out2);
  else
    return ARLE_E_BADARG;
  return launch_status();
}

// 1: kernels are launched so that the next kernel of the stream may start its set-up
// (barriers, weight prefetch) while the previous one finishes; 0 (default): plain launches.
ARLE_API void arle_set_programmatic_launch(int mode) { arle::pdl_enabled() = mode & 3; }
