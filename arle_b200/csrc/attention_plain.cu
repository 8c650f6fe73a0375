// General paged causal attention: any head size up to 256, any page size, any
// number of heads and groups, float32 or bfloat16 storage, float32 arithmetic
// throughout (scores, softmax, P.V; P is not rounded before P.V).  It serves the
// 32-bit path of the engine and is the yardstick of the tensor-core kernels.
//
// One block per (token, query head).  The query at absolute position p of request
// row r sees keys j in [max(0, p - window + 1), p] (window <= 0: from 0), found
// through the row's block table.  Warp w takes key tiles w, w+4, ... of 32 keys
// counted from the first visible key, keeps an online softmax (m, l, acc), and
// the four partial results are merged at the end.  The order of all sums depends
// on (first key, p) only, so a token's result is the same however the prompt was
// cut into steps and whatever else is in the batch.
//
// Values may have another width than keys (vd; the value cache is [page][kv_head][slot][vd]).  With a sink the
// softmax has one more term in its denominator, exp(sink_logit), that carries no value:
// p_j = exp(s_j) / (exp(sink_logit) + sum exp(s_j)), one sink score per query head.  With a gate, head h's output is
// multiplied by sigmoid(gate[t, h]).
//
// With sigmoid weights (pb: one number per query head, added to the scaled score) there is no softmax: a visible key's weight
// is sigmoid(score + pb[h]) as it is, and the values' weighted sum is the result.  With chunks a query sees only the keys of
// its own chunk of positions (counted from position 0).
#include "common.cuh"
using namespace arle;

constexpr int kAttnWarps = 4;
constexpr int kAttnMaxD = 8;  // head_dim <= 256

template <typename T>
__global__ void paged_attention_plain_kernel(const T* __restrict__ q, int q_row_stride, T* __restrict__ out,
                                             const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                                             const int* __restrict__ positions,
                                             const int* __restrict__ row_of_token,
                                             const int* __restrict__ block_table, int bt_stride, int nq,
                                             int nkv, int hd, int vd, int page_size, float scale, int window,
                                             HeadTail<T> tail, int keep_first, float softcap, int chunk, const float* __restrict__ pb) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float qs[256];
  __shared__ float acc_s[kAttnWarps][256];
  __shared__ float m_s[kAttnWarps], l_s[kAttnWarps];
  const int t = blockIdx.x, h = blockIdx.y;
  const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = h / (nq / nkv);
  const int pos = positions[t];
  const int* bt = block_table + (size_t)row_of_token[t] * bt_stride;
  const int lo = first_visible_key(pos, window, chunk);
  const int ka = min(keep_first, lo);                // kept first keys outside the window
  const int nvis = ka + pos - lo + 1;                // visible keys: index i is key i (i < ka) or key lo + i - ka

  const T* qp = q + (size_t)t * q_row_stride + (size_t)h * hd;
  for (int e = threadIdx.x; e < hd; e += blockDim.x) qs[e] = to_f32(qp[e]) * scale;
  __syncthreads();

  float m = -INFINITY, l = 0.f;
  float acc[kAttnMaxD];
#pragma unroll
  for (int i = 0; i < kAttnMaxD; ++i) acc[i] = 0.f;

  const size_t page_stride = (size_t)nkv * page_size * hd;
  const size_t vpage_stride = (size_t)nkv * page_size * vd;
  for (int i0 = w * 32; i0 < nvis; i0 += kAttnWarps * 32) {
    const int iv = i0 + lane;
    const int j = iv < ka ? iv : lo + iv - ka;
    float sc = -INFINITY;
    if (iv < nvis) {
      const int page = bt[j / page_size];
      const T* kp = k_cache + (size_t)page * page_stride + ((size_t)kvh * page_size + j % page_size) * hd;
      float d = 0.f;
      for (int e = 0; e < hd; ++e) d = fmaf(qs[e], to_f32(kp[e]), d);
      sc = softcap > 0.f ? softcap * tanhf(d / softcap) : d;
    }
    float p;
    if (pb) {
      p = iv < nvis ? 1.0f / (1.0f + expf(-(sc + pb[h]))) : 0.f;
      m = 0.f;                                       // every warp's sums count as they are
    } else {
      const float mt = warp_max(sc);
      const float m_new = fmaxf(m, mt);
      p = iv < nvis ? expf(sc - m_new) : 0.f;
      const float corr = expf(m - m_new);
      l = l * corr + warp_sum(p);
#pragma unroll
      for (int i = 0; i < kAttnMaxD; ++i) acc[i] *= corr;
      m = m_new;
    }
    const int nvalid = min(32, nvis - i0);
    for (int jj = 0; jj < nvalid; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const int jk = i0 + jj < ka ? i0 + jj : lo + i0 + jj - ka;
      const int page = bt[jk / page_size];
      const T* vp = v_cache + (size_t)page * vpage_stride + ((size_t)kvh * page_size + jk % page_size) * vd;
#pragma unroll
      for (int i = 0; i < kAttnMaxD; ++i) {
        const int d = lane + 32 * i;
        if (d < vd) acc[i] = fmaf(pj, to_f32(vp[d]), acc[i]);
      }
    }
  }
  if (lane == 0) {
    m_s[w] = m;
    l_s[w] = l;
  }
#pragma unroll
  for (int i = 0; i < kAttnMaxD; ++i) {
    const int d = lane + 32 * i;
    if (d < vd) acc_s[w][d] = acc[i];
  }
  __syncthreads();
  const bool has_sink = tail.sinks != nullptr;
  const float sink_logit = has_sink ? tail.sinks[h] : 0.f;
  float mm = has_sink ? sink_logit : m_s[0];
  for (int i = has_sink ? 0 : 1; i < kAttnWarps; ++i) mm = fmaxf(mm, m_s[i]);
  float f[kAttnWarps], ll = has_sink ? expf(sink_logit - mm) : 0.f;
  for (int i = 0; i < kAttnWarps; ++i) {
    f[i] = expf(m_s[i] - mm);  // a warp without keys has m = -inf, so f = 0
    ll += l_s[i] * f[i];
  }
  if (pb) ll = 1.f;
  const float gate = tail.gate_of(t, h);
  T* op = out + ((size_t)t * nq + h) * vd;
  for (int d = threadIdx.x; d < vd; d += blockDim.x) {
    float o = 0.f;
    for (int i = 0; i < kAttnWarps; ++i) o += acc_s[i][d] * f[i];
    op[d] = from_f32<T>(o / ll * gate);
  }
}

ARLE_API int arle_paged_attention_plain(const void* q, int q_row_stride, void* out, const void* k_cache,
                                        const void* v_cache, int dtype, const int* positions,
                                        const int* row_of_token, const int* block_table, int bt_stride,
                                        int nq, int nkv, int hd, int vd, int page_size, float scale, int window,
                                        const float* sinks, const void* gate, int gate_stride, int keep_first, float softcap, int chunk, const float* pb,
                                        int num_tokens, cudaStream_t s) {
  if (num_tokens <= 0) return 0;
  if (chunk < 0 || (chunk > 0 && window > 0) || (pb && sinks)) return ARLE_E_BADARG;
  if (vd <= 0 || vd > 256) return ARLE_E_UNSUPPORTED;
  if (hd <= 0 || hd > 256 || nq <= 0 || nkv <= 0 || nq % nkv != 0 || page_size <= 0) return ARLE_E_UNSUPPORTED;
  if (nq > 65535) return ARLE_E_UNSUPPORTED;
  if (keep_first < 0 || softcap < 0.f) return ARLE_E_BADARG;
  dim3 grid(num_tokens, nq);
  if (dtype == 0)
    launch_kernel(paged_attention_plain_kernel<float>, dim3(grid), dim3(kAttnWarps * 32), 0, s, 1, 
        (const float*)q, q_row_stride, (float*)out, (const float*)k_cache, (const float*)v_cache, positions,
        row_of_token, block_table, bt_stride, nq, nkv, hd, vd, page_size, scale, window,
        HeadTail<float>{sinks, (const float*)gate, gate_stride}, keep_first, softcap, chunk, pb);
  else if (dtype == 1)
    launch_kernel(paged_attention_plain_kernel<__nv_bfloat16>, dim3(grid), dim3(kAttnWarps * 32), 0, s, 1, 
        (const __nv_bfloat16*)q, q_row_stride, (__nv_bfloat16*)out, (const __nv_bfloat16*)k_cache,
        (const __nv_bfloat16*)v_cache, positions, row_of_token, block_table, bt_stride, nq, nkv, hd, vd,
        page_size, scale, window, HeadTail<__nv_bfloat16>{sinks, (const __nv_bfloat16*)gate, gate_stride}, keep_first, softcap, chunk, pb);
  else
    return ARLE_E_BADARG;
  return launch_status();
}
