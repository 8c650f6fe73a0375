// Matrix memories with one constant decay per head, over long rows of a step, in chunks of tokens that run side by side:
//
//     S_t = a S_(t-1) + k_t v_t^T,        o_t = S_t^T (q_scale q_t)          (S: dim x vdim, float32; a = decay[h])
//
// With S_0 the memory before a chunk of n tokens (0-based places i, j in the chunk),
//     o_i = sum_(j <= i) a^(i - j) (q_i . k_j) v_j + a^(i + 1) S_0^T q_i,
//     S_n = a^n S_0 + sum_j a^(n - 1 - j) k_j v_j^T,
// so only the carry from chunk to chunk is serial.  Three kernels over the chunks of all long rows of the step:
//  * chunk_own: U_c = sum_j a^(n - 1 - j) k_j v_j^T of every chunk (a block per chunk, head, tile of 64 or 128 columns of v);
//  * chunk_carry: walks a row's chunks in order, S_c = a^n S_(c-1) + U_c element by element; leaves the memory BEFORE every chunk
//    in U_c's place and the row's last memory in its state slot;
//  * chunk_out: scores of the chunk's queries against its own keys with the decay's powers as a mask, times v, plus the read-out
//    of the memory before the chunk.
// Everything is float32 (FFMA) whatever the activation type.  q and k may be rotated (half-split pairs, cosines and sines from the
// step's table) or go through silu (then v too) as they are staged.  The powers are powf(a, n).  A chunk is 64 tokens counted from
// the row's first token of the step, so the order of a token's sums depends on where its portion starts: within rounding.
// chunk_plan lists the chunks of the step once for all layers.  Rows of up to `longest` tokens are left alone (the scan in
// recurrent.cu runs them).
#include "common.cuh"
using namespace arle;

namespace {

constexpr int kC = 64;                  // tokens of a chunk
constexpr int kThreads = 256;
constexpr int kPad = 4;                 // floats behind a row in shared memory: rows fall on different banks, 16-byte aligned

struct Chunk {
  int t0, n, row, index;                // first token, tokens, row of the step, place among the row's chunks
};

// plan: first [R + 1] (a row's first chunk; the total at the end), padded to a multiple of 4, then a Chunk each.
__global__ void __launch_bounds__(kThreads) chunk_plan_kernel(const int* __restrict__ q_indptr, int R, int longest, int* __restrict__ plan) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int sums[kThreads];
  Chunk* list = reinterpret_cast<Chunk*>(plan + ((R + 1 + 3) & ~3));
  int carry = 0;
  for (int base = 0; base < R; base += kThreads) {
    const int r = base + threadIdx.x;
    const int beg = r < R ? q_indptr[r] : 0, len = r < R ? q_indptr[r + 1] - beg : 0;
    const int mine = len > longest ? (len + kC - 1) / kC : 0;
    sums[threadIdx.x] = mine;
    __syncthreads();
    for (int o = 1; o < kThreads; o <<= 1) {
      const int v = threadIdx.x >= o ? sums[threadIdx.x - o] : 0;
      __syncthreads();
      sums[threadIdx.x] += v;
      __syncthreads();
    }
    const int first = carry + sums[threadIdx.x] - mine;
    if (r < R) plan[r] = first;
    for (int c = 0; c < mine; ++c) list[first + c] = Chunk{beg + c * kC, min(kC, len - c * kC), r, c};
    carry += sums[kThreads - 1];
    __syncthreads();
  }
  if (threadIdx.x == 0) plan[R] = carry;
}

struct Stage {                          // how q and k are read
  const float2* angles;                 // [T, rotary_dim / 2] (cos, sin), or null: no rotation
  int rotary_dim, act;                  // act 1: silu
};

__device__ __forceinline__ float silu(float x) { return x / (1.0f + expf(-x)); }

// rows 0 .. n-1 of NS arrays (row strides given, dim numbers), rotated, times scale (and w[row], if given), into dst [kC][DP + kPad];
// zeros past dim and past n.  Four numbers an access; a thread's loads of up to four places are asked for together.
template <typename T, int DP, int NS>
__device__ __forceinline__ void stage_rows_vec(const T* const (&x)[NS], const long (&stride)[NS], int t0, int n, int dim, const Stage& st,
                                               const float (&scale)[NS], const float* w, float* const (&dst)[NS]) {
  constexpr int PITCH = DP + kPad, Q = DP / 4, ITEMS = kC * Q / kThreads, B = ITEMS < 4 ? ITEMS : 4;
  typedef Pack<T, 4> P4;
  const int half = st.rotary_dim >> 1;
#pragma unroll
  for (int b0 = 0; b0 < ITEMS; b0 += B) {
    P4 own[NS][B], other[NS][B];
    float4 ca[B], cb[B];
#pragma unroll
    for (int b = 0; b < B; ++b) {
      const int idx = threadIdx.x + (b0 + b) * kThreads;
      const int tt = idx / Q, e = (idx - tt * Q) * 4;
      const bool in = tt < n && e < dim;
      const bool turns = in && e < st.rotary_dim, first = e < half;
      ca[b] = cb[b] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int m = 0; m < NS; ++m) {
        const T* p = x[m] + (size_t)(t0 + tt) * stride[m] + e;
#pragma unroll
        for (int g = 0; g < 4; ++g) own[m][b].e[g] = other[m][b].e[g] = from_f32<T>(0.f);
        if (in) own[m][b] = *reinterpret_cast<const P4*>(p);
        if (turns) other[m][b] = *reinterpret_cast<const P4*>(first ? p + half : p - half);
      }
      if (turns) {
        const float4* a = reinterpret_cast<const float4*>(st.angles + (size_t)(t0 + tt) * half + (first ? e : e - half));
        ca[b] = a[0];
        cb[b] = a[1];
      }
    }
#pragma unroll
    for (int b = 0; b < B; ++b) {
      const int idx = threadIdx.x + (b0 + b) * kThreads;
      const int tt = idx / Q, e = (idx - tt * Q) * 4;
      const bool turns = tt < n && e < st.rotary_dim;
      const float side = e < half ? -1.f : 1.f;
      const float cs[4] = {ca[b].x, ca[b].z, cb[b].x, cb[b].z}, sn[4] = {ca[b].y, ca[b].w, cb[b].y, cb[b].w};
#pragma unroll
      for (int m = 0; m < NS; ++m) {
        const float f = w ? scale[m] * w[tt] : scale[m];
        float v[4];
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          v[g] = to_f32(own[m][b].e[g]);
          if (turns) v[g] = v[g] * cs[g] + side * (to_f32(other[m][b].e[g]) * sn[g]);
          v[g] = (st.act ? silu(v[g]) : v[g]) * f;
        }
        *reinterpret_cast<float4*>(dst[m] + tt * PITCH + e) = make_float4(v[0], v[1], v[2], v[3]);
      }
    }
  }
}

// The same number by number, for rows that are not on the boundaries the other needs.
template <typename T, int DP>
__device__ __forceinline__ void stage_rows_any(const T* __restrict__ x, long stride, int t0, int n, int dim, const Stage& st, float scale,
                                               const float* w, float* dst) {
  constexpr int PITCH = DP + kPad;
  const int half = st.rotary_dim >> 1;
  for (int idx = threadIdx.x; idx < kC * DP; idx += kThreads) {
    const int tt = idx / DP, e = idx - tt * DP;
    float v = 0.f;
    if (tt < n && e < dim) {
      const T* row = x + (size_t)(t0 + tt) * stride;
      v = to_f32(row[e]);
      if (e < st.rotary_dim) {
        const bool first = e < half;
        const int i = first ? e : e - half;
        const float2 a = st.angles[(size_t)(t0 + tt) * half + i];
        const float o = to_f32(row[first ? e + half : i]);
        v = first ? v * a.x - o * a.y : v * a.x + o * a.y;
      }
      v = (st.act ? silu(v) : v) * (w ? scale * w[tt] : scale);
    }
    dst[tt * PITCH + e] = v;
  }
}

// U[chunk][h][v][d] = sum_j a^(n - 1 - j) k_j[d] v_j[v]
template <typename T, int DP, int VT, bool VEC>
__global__ void __launch_bounds__(kThreads, 2) chunk_own_kernel(const T* __restrict__ k, const T* __restrict__ v, long k_stride, long v_stride,
                                                             const float* __restrict__ decay, const int* __restrict__ plan, int R,
                                                             Stage st, float* __restrict__ own, int H, int dim, int vdim) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int PITCH = DP + kPad;
  constexpr int ND = DP / 16;                           // numbers of d a thread holds: groups of min(4, ND), 64 apart
  constexpr int GD = ND < 4 ? ND : 4;
  constexpr int NV = VT / 16;                           // columns of v a thread holds: groups of four, 64 apart
  extern __shared__ __align__(16) float sm[];
  float* ks = sm;                                       // [kC][PITCH], times the decay's power
  float* vs = ks + kC * PITCH;                          // [kC][VT]
  float* pw = vs + kC * VT;                             // [kC]
  const Chunk ch = reinterpret_cast<const Chunk*>(plan + ((R + 1 + 3) & ~3))[blockIdx.z];
  const int h = blockIdx.y, v0 = blockIdx.x * VT;
  const float a = decay[h];
  if (threadIdx.x < kC) pw[threadIdx.x] = threadIdx.x < ch.n ? powf(a, (float)(ch.n - 1 - threadIdx.x)) : 0.f;
  __syncthreads();
  if constexpr (VEC) {
    constexpr int Q = VT / 4, ITEMS = kC * Q / kThreads;
    Pack<T, 4> x[ITEMS];
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int idx = threadIdx.x + i * kThreads;
      const int tt = idx / Q, c = v0 + (idx - tt * Q) * 4;
#pragma unroll
      for (int g = 0; g < 4; ++g) x[i].e[g] = from_f32<T>(0.f);
      if (tt < ch.n && c < vdim) x[i] = *reinterpret_cast<const Pack<T, 4>*>(v + (size_t)(ch.t0 + tt) * v_stride + (size_t)h * vdim + c);
    }
    const T* const src[1] = {k + (size_t)h * dim};
    const long strides[1] = {k_stride};
    const float one[1] = {1.0f};
    float* const dst[1] = {ks};
    stage_rows_vec<T, DP, 1>(src, strides, ch.t0, ch.n, dim, st, one, pw, dst);
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      float y[4];
#pragma unroll
      for (int g = 0; g < 4; ++g) y[g] = st.act ? silu(to_f32(x[i].e[g])) : to_f32(x[i].e[g]);
      *reinterpret_cast<float4*>(vs + (threadIdx.x + i * kThreads) * 4) = make_float4(y[0], y[1], y[2], y[3]);
    }
  } else {
    stage_rows_any<T, DP>(k + (size_t)h * dim, k_stride, ch.t0, ch.n, dim, st, 1.0f, pw, ks);
    for (int idx = threadIdx.x; idx < kC * VT; idx += kThreads) {
      const int tt = idx / VT, c = v0 + idx - tt * VT;
      const float x = (tt < ch.n && c < vdim) ? to_f32(v[(size_t)(ch.t0 + tt) * v_stride + (size_t)h * vdim + c]) : 0.f;
      vs[idx] = st.act ? silu(x) : x;
    }
  }
  __syncthreads();
  const int td = threadIdx.x & 15, tv = threadIdx.x >> 4;
  float acc[NV][ND];
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int d = 0; d < ND; ++d) acc[i][d] = 0.f;
#pragma unroll 2
  for (int j = 0; j < ch.n; ++j) {
    float vr[NV];
#pragma unroll
    for (int g = 0; g < NV / 4; ++g) {
      const float4 vv = *reinterpret_cast<const float4*>(vs + j * VT + g * 64 + tv * 4);
      vr[4 * g] = vv.x, vr[4 * g + 1] = vv.y, vr[4 * g + 2] = vv.z, vr[4 * g + 3] = vv.w;
    }
#pragma unroll
    for (int g = 0; g < ND / GD; ++g) {
      float kr[GD];
      load_vec<float, GD>(ks + j * PITCH + g * 16 * GD + td * GD, kr);
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int d = 0; d < GD; ++d) acc[i][g * GD + d] = fmaf(vr[i], kr[d], acc[i][g * GD + d]);
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = v0 + (i >> 2) * 64 + tv * 4 + (i & 3);
    if (c >= vdim) break;
    float* o = own + (((size_t)blockIdx.z * H + h) * vdim + c) * dim;
#pragma unroll
    for (int g = 0; g < ND / GD; ++g) {
      const int d0 = g * 16 * GD + td * GD;
      if (VEC && GD == 4) {
        if (d0 < dim) *reinterpret_cast<float4*>(o + d0) = make_float4(acc[i][g * GD], acc[i][g * GD + 1], acc[i][g * GD + GD - 2], acc[i][g * GD + GD - 1]);
      } else {
#pragma unroll
        for (int d = 0; d < GD; ++d)
          if (d0 + d < dim) o[d0 + d] = acc[i][g * GD + d];
      }
    }
  }
}

// A thread walks G numbers of a row's memories through the row's chunks.
template <int G>
__global__ void __launch_bounds__(kThreads) chunk_carry_kernel(float* __restrict__ own, const float* __restrict__ decay, const int* __restrict__ plan,
                                                               int R, float* __restrict__ state, long slot_stride,
                                                               const int* __restrict__ state_slots, long per_head, long total) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.y;
  const int first = plan[r], count = plan[r + 1] - first;
  const long e = ((long)blockIdx.x * kThreads + threadIdx.x) * G;
  if (count == 0 || e >= total) return;
  const Chunk* list = reinterpret_cast<const Chunk*>(plan + ((R + 1 + 3) & ~3));
  const float a = decay[e / per_head];
  const float whole = powf(a, (float)kC), last = powf(a, (float)list[first + count - 1].n);
  float* sp = state + (size_t)state_slots[r] * slot_stride + e;
  float* up = own + (size_t)first * total + e;
  float S[G];
  load_vec<float, G>(sp, S);
  constexpr int B = 8;                                  // chunks asked for together
  for (int c0 = 0; c0 < count; c0 += B) {
    float U[B][G];
#pragma unroll
    for (int b = 0; b < B; ++b)
      if (c0 + b < count) load_vec<float, G>(up + (size_t)(c0 + b) * total, U[b]);
#pragma unroll
    for (int b = 0; b < B; ++b) {
      if (c0 + b < count) {
        store_vec<float, G>(up + (size_t)(c0 + b) * total, S);
        const float p = c0 + b == count - 1 ? last : whole;
#pragma unroll
        for (int g = 0; g < G; ++g) S[g] = fmaf(p, S[g], U[b][g]);
      }
    }
  }
  store_vec<float, G>(sp, S);
}

__device__ __forceinline__ void copy16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

template <typename T, int DP, int VT, bool VEC>
__global__ void __launch_bounds__(kThreads, VT == 128 ? 1 : 2) chunk_out_kernel(
    const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long q_stride, long k_stride, long v_stride,
    const float* __restrict__ decay, const int* __restrict__ plan, int R, Stage st, const float* __restrict__ before,
    float* __restrict__ out, int H, int dim, int vdim, float q_scale) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int PITCH = DP + kPad, AP = kC + kPad;
  constexpr int NC = VT / 16;                           // columns a thread holds, 16 apart
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;                                       // [kC][PITCH]
  float* ks = qs + kC * PITCH;                          // [kC][PITCH]
  float* ms = ks + kC * PITCH;                          // [VT][PITCH] the memory's columns
  float* as = ms + VT * PITCH;                          // [kC][AP] scores with the decay's powers
  float* vt = as + kC * AP;                             // [VT][AP] v transposed
  float* pw = vt + VT * AP;                             // [kC + 1]
  const Chunk ch = reinterpret_cast<const Chunk*>(plan + ((R + 1 + 3) & ~3))[blockIdx.z];
  const int h = blockIdx.y, v0 = blockIdx.x * VT, n = ch.n;
  const float a = decay[h];
  if (threadIdx.x <= kC) pw[threadIdx.x] = powf(a, (float)threadIdx.x);
  // the memory before the chunk: on its way while q, k and v are staged and the scores are formed
  const float* bp = before + (((size_t)blockIdx.z * H + h) * vdim + v0) * dim;
  constexpr int G = VEC ? 4 : 1;
  for (int idx = threadIdx.x; idx < VT * (DP / G); idx += kThreads) {
    const int c = idx / (DP / G), e = (idx - c * (DP / G)) * G;
    float* dst = ms + c * PITCH + e;
    if (v0 + c < vdim && e < dim) {
      if (VEC) copy16(dst, bp + (size_t)c * dim + e);
      else *dst = bp[(size_t)c * dim + e];
    } else {
#pragma unroll
      for (int g = 0; g < G; ++g) dst[g] = 0.f;
    }
  }
  if constexpr (VEC) {
    // v: four columns of four tokens a thread, turned round in registers; eight lanes write a column's tokens side by side
    constexpr int CG = VT / 4, ITEMS = CG * (kC / 4) / kThreads;
    Pack<T, 4> x[ITEMS][4];
#pragma unroll
    for (int it = 0; it < ITEMS; ++it) {
      const int idx = threadIdx.x + it * kThreads;
      const int j0 = ((idx & 7) + idx / (8 * CG) * 8) * 4, c = (idx / 8) % CG * 4;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
#pragma unroll
        for (int g = 0; g < 4; ++g) x[it][i].e[g] = from_f32<T>(0.f);
        if (j0 + i < n && v0 + c < vdim)
          x[it][i] = *reinterpret_cast<const Pack<T, 4>*>(v + (size_t)(ch.t0 + j0 + i) * v_stride + (size_t)h * vdim + v0 + c);
      }
    }
    const T* const src[2] = {q + (size_t)h * dim, k + (size_t)h * dim};
    const long strides[2] = {q_stride, k_stride};
    const float scales[2] = {q_scale, 1.0f};
    float* const dst[2] = {qs, ks};
    stage_rows_vec<T, DP, 2>(src, strides, ch.t0, n, dim, st, scales, nullptr, dst);
#pragma unroll
    for (int it = 0; it < ITEMS; ++it) {
      const int idx = threadIdx.x + it * kThreads;
      const int j0 = ((idx & 7) + idx / (8 * CG) * 8) * 4, c = (idx / 8) % CG * 4;
#pragma unroll
      for (int g = 0; g < 4; ++g) {
        float y[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) y[i] = st.act ? silu(to_f32(x[it][i].e[g])) : to_f32(x[it][i].e[g]);
        *reinterpret_cast<float4*>(vt + (c + g) * AP + j0) = make_float4(y[0], y[1], y[2], y[3]);
      }
    }
  } else {
    stage_rows_any<T, DP>(q + (size_t)h * dim, q_stride, ch.t0, n, dim, st, q_scale, nullptr, qs);
    stage_rows_any<T, DP>(k + (size_t)h * dim, k_stride, ch.t0, n, dim, st, 1.0f, nullptr, ks);
    for (int idx = threadIdx.x; idx < VT * kC; idx += kThreads) {
      const int c = idx & (VT - 1), j = idx / VT;
      const float x = (j < n && v0 + c < vdim) ? to_f32(v[(size_t)(ch.t0 + j) * v_stride + (size_t)h * vdim + v0 + c]) : 0.f;
      vt[c * AP + j] = st.act ? silu(x) : x;
    }
  }
  __syncthreads();
  const int tc = threadIdx.x & 15, ti = threadIdx.x >> 4;
  // acc[i][c] += sum_e x[ti * 4 + i][e] y[tc + 16 c][e]
  auto product = [&](auto& acc, const float* x, const float* y, int xp, int yp, int len) {
    constexpr int N = sizeof(acc[0]) / sizeof(float);
#pragma unroll 2
    for (int e = 0; e < len; e += 4) {
      float4 xr[4], yr[N];
#pragma unroll
      for (int i = 0; i < 4; ++i) xr[i] = *reinterpret_cast<const float4*>(x + (ti * 4 + i) * xp + e);
#pragma unroll
      for (int c = 0; c < N; ++c) yr[c] = *reinterpret_cast<const float4*>(y + (tc + 16 * c) * yp + e);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int c = 0; c < N; ++c) {
          acc[i][c] = fmaf(xr[i].x, yr[c].x, acc[i][c]);
          acc[i][c] = fmaf(xr[i].y, yr[c].y, acc[i][c]);
          acc[i][c] = fmaf(xr[i].z, yr[c].z, acc[i][c]);
          acc[i][c] = fmaf(xr[i].w, yr[c].w, acc[i][c]);
        }
    }
  };
  {
    float sc[4][kC / 16];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int c = 0; c < kC / 16; ++c) sc[i][c] = 0.f;
    product(sc, qs, ks, PITCH, PITCH, DP);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int c = 0; c < kC / 16; ++c) {
        const int row = ti * 4 + i, col = tc + 16 * c;
        as[row * AP + col] = col <= row ? sc[i][c] * pw[row - col] : 0.f;
      }
  }
  if (VEC) asm volatile("cp.async.wait_all;\n" ::: "memory");
  __syncthreads();
  float acc[4][NC];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int c = 0; c < NC; ++c) acc[i][c] = 0.f;
  product(acc, qs, ms, PITCH, PITCH, DP);
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int c = 0; c < NC; ++c) acc[i][c] *= pw[ti * 4 + i + 1];
  product(acc, as, vt, AP, AP, (min(n, ti * 4 + 4) + 3) & ~3);        // scores beyond the query's own place are zero
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (ti * 4 + i >= n) break;
    float* o = out + ((size_t)(ch.t0 + ti * 4 + i) * H + h) * vdim + v0;
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (v0 + tc + 16 * c < vdim) o[tc + 16 * c] = acc[i][c];
  }
}

template <typename T, int DP, int VT, bool VEC>
int launch_as(const void* q, const void* k, const void* v, int q_stride, int k_stride, int v_stride, const float* decay, float* state,
              long slot_stride, const int* state_slots, const int* plan, int chunks, const Stage& st, float* own, float* out, int R, int H,
              int dim, int vdim, float q_scale, cudaStream_t s) {
  const dim3 grid((vdim + VT - 1) / VT, H, chunks);
  const size_t smem1 = (size_t)(kC * (DP + kPad) + kC * VT + kC) * sizeof(float);
  const size_t smem3 = (size_t)((2 * kC + VT) * (DP + kPad) + (kC + VT) * (kC + kPad) + kC + 4) * sizeof(float);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(chunk_own_kernel<T, DP, VT, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(chunk_out_kernel<T, DP, VT, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  launch_kernel(chunk_own_kernel<T, DP, VT, VEC>, grid, dim3(kThreads), smem1, s, 1, (const T*)k, (const T*)v, (long)k_stride, (long)v_stride, decay,
                plan, R, st, own, H, dim, vdim);
  const long total = (long)H * vdim * dim;
  if (dim % 4 == 0 && slot_stride % 4 == 0 && vec_aligned<4>(state, 4) && vec_aligned<4>(own, 4))
    launch_kernel(chunk_carry_kernel<4>, dim3((unsigned)((total / 4 + kThreads - 1) / kThreads), R), dim3(kThreads), 0, s, 1, own, decay, plan, R,
                  state, slot_stride, state_slots, (long)vdim * dim, total);
  else
    launch_kernel(chunk_carry_kernel<1>, dim3((unsigned)((total + kThreads - 1) / kThreads), R), dim3(kThreads), 0, s, 1, own, decay, plan, R,
                  state, slot_stride, state_slots, (long)vdim * dim, total);
  launch_kernel(chunk_out_kernel<T, DP, VT, VEC>, grid, dim3(kThreads), smem3, s, 1, (const T*)q, (const T*)k, (const T*)v, (long)q_stride,
                (long)k_stride, (long)v_stride, decay, plan, R, st, own, out, H, dim, vdim, q_scale);
  return launch_status();
}

}  // namespace

// Ints of a step's plan for this many rows and chunks, and the chunks of a row of this many tokens.
ARLE_API int arle_decay_chunk_plan_ints(int rows, int chunks) { return ((rows + 1 + 3) & ~3) + 4 * chunks; }
ARLE_API int arle_decay_chunk_tokens() { return kC; }

ARLE_API int arle_decay_chunk_plan(const int* q_indptr, int rows, int longest, int* plan, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (longest < 0 || !plan || ((uintptr_t)plan & 15)) return ARLE_E_BADARG;
  launch_kernel(chunk_plan_kernel, dim3(1), dim3(kThreads), 0, s, 1, q_indptr, rows, longest, plan);
  return launch_status();
}

// q, k [T, H*dim], v [T, H*vdim] in the activation type (row strides given); decay float32 [H]; state float32, a slot every
// slot_stride numbers, [H][vdim][dim] at its start; plan: arle_decay_chunk_plan's, with `chunks` chunks in all; angles: float32
// [T, rotary_dim / 2, 2] or null; act 1: silu on q, k and v; own: float32 scratch [chunks, H, vdim, dim]; out float32 [T, H, vdim]
// (rows that have no chunk are not written).  dim at most 128.
ARLE_API int arle_decay_chunks(const void* q, const void* k, const void* v, int dtype, int q_stride, int k_stride, int v_stride,
                               const float* decay, float* state, long slot_stride, const int* state_slots, const int* plan, int chunks,
                               const float* angles, int rotary_dim, int act, float* own, float* out, int R, int H, int dim, int vdim,
                               float q_scale, cudaStream_t s) {
  if (R <= 0 || chunks <= 0) return 0;
  if (!decay || !state || !plan || !own || !out || H <= 0 || dim <= 0 || vdim <= 0 || rotary_dim < 0 || rotary_dim % 2 || rotary_dim > dim ||
      (rotary_dim && (!angles || act)))
    return ARLE_E_BADARG;
  if (dim > 128 || H > 65535 || chunks > 65535 || R > 65535) return ARLE_E_UNSUPPORTED;
  const Stage st{reinterpret_cast<const float2*>(angles), rotary_dim, act};
  const size_t el = dtype == 0 ? 4 : 2;
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && rotary_dim % 8 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && v_stride % 4 == 0 &&
                   vec_aligned<4>(q, el) && vec_aligned<4>(k, el) && vec_aligned<4>(v, el) &&
                   vec_aligned<4>(angles, 4) && vec_aligned<4>(own, 4);
#define ARLE_CHUNKS(TT, D, VT, V) \
  return launch_as<TT, D, VT, V>(q, k, v, q_stride, k_stride, v_stride, decay, state, slot_stride, state_slots, plan, chunks, st, own, out, R, H, \
                                 dim, vdim, q_scale, s)
#define ARLE_CHUNKS_D(TT, V) \
  do { \
    if (dim <= 32) ARLE_CHUNKS(TT, 32, 64, V); \
    if (dim <= 64) ARLE_CHUNKS(TT, 64, 64, V); \
    if (vdim <= 64) ARLE_CHUNKS(TT, 128, 64, V); \
    ARLE_CHUNKS(TT, 128, 128, V); \
  } while (0)
  if (dtype == 0) {
    if (vec) ARLE_CHUNKS_D(float, true);
    ARLE_CHUNKS_D(float, false);
  }
  if (dtype == 1) {
    if (vec) ARLE_CHUNKS_D(__nv_bfloat16, true);
    ARLE_CHUNKS_D(__nv_bfloat16, false);
  }
#undef ARLE_CHUNKS_D
#undef ARLE_CHUNKS
  return ARLE_E_BADARG;
}
