// A layer's input that belongs to the token itself: a part of the token's row of a second embedding table, gated by a
// projection of the residual stream,
//
//   g[t, j] = gelu_tanh(W_gate x_t)_j * table[id_t, offset + j]            j < D
//
// (the projection of g back to the width and its norm are a library product and the norm kernel that reads it).
//
//   qb_token_input_act  : from the gate product's float32 accumulators
//   qb_token_input_gate : steps of few tokens: product, activation and gather in one launch; a block a gate row and up to
//                         TI_TOK tokens, the row read once for all of them, threads stride the width (their sums are added
//                         across lanes, then warps in order)
//
// gelu_tanh(z) = z / 2 (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))).  float32 inside; one rounding at the store.  A token
// id outside the table is recorded and its row becomes zeros.
#include "common.cuh"

constexpr int TI_TOK = 8;
constexpr int TI_WARPS = 4;

template <typename A>
__global__ void token_input_act_kernel(const float* __restrict__ gate, int gate_stride, const A* __restrict__ table,
                                       int table_stride, int offset, const int* __restrict__ ids, A* __restrict__ out,
                                       int T, int D, int V, int* status) {
  const size_t n = (size_t)T * D;
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const int t = (int)(i / D), j = (int)(i % D);
    const int id = ids[t];
    if (id < 0 || id >= V) {
      qb_set_status(status, QB_STATUS_BAD_TOKEN, id, 1);
      out[i] = qb_from_float<A>(0.f);
      continue;
    }
    const float e = qb_to_float<A>(table[(size_t)id * table_stride + offset + j]);
    out[i] = qb_from_float<A>(qb_gelu_tanh(gate[(size_t)t * gate_stride + j]) * e);
  }
}

extern "C" int qb_token_input_act(const float* gate, int gate_stride, const void* table, int table_stride, int offset,
                                  const int* ids, void* out, int dtype, int T, int D, int V, int* status,
                                  cudaStream_t stream) {
  if (T <= 0) return 0;
  if (D <= 0 || offset < 0 || offset + D > table_stride || gate_stride < D) return QB_ERR_BAD_ARG;
  const size_t n = (size_t)T * D;
  const int blocks = (int)((n + 255) / 256 < 4096 ? (n + 255) / 256 : 4096);
  QB_DISPATCH_DTYPE(dtype, A, token_input_act_kernel<A><<<blocks, 256, 0, stream>>>(
      gate, gate_stride, (const A*)table, table_stride, offset, ids, (A*)out, T, D, V, status));
  QB_LAUNCH_CHECK();
  return 0;
}

template <typename A, bool VEC>
__global__ void __launch_bounds__(TI_WARPS * 32)
token_input_gate_kernel(const A* __restrict__ x, const A* __restrict__ w, const A* __restrict__ table, int table_stride,
                        int offset, const int* __restrict__ ids, A* __restrict__ out, int T, int W, int D, int V,
                        int* status) {
  __shared__ float s_sum[TI_WARPS][TI_TOK];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int j = blockIdx.x;
  const int t0 = blockIdx.y * TI_TOK, n = min(TI_TOK, T - t0);
  const A* wrow = w + (size_t)j * W;
  // the table's number is asked for first: its address is a chain of two loads
  int id = -1;
  float e_val = 0.f;
  if ((int)threadIdx.x < n) {
    id = ids[t0 + threadIdx.x];
    if (id >= 0 && id < V) e_val = qb_to_float<A>(table[(size_t)id * table_stride + offset + j]);
  }
  float acc[TI_TOK];
#pragma unroll
  for (int u = 0; u < TI_TOK; ++u) acc[u] = 0.f;
  if (VEC) {
    for (int i = threadIdx.x * 8; i < W; i += TI_WARPS * 256) {
      float wv[8];
      QbVec8<A>::load(wrow + i, wv);
#pragma unroll
      for (int u = 0; u < TI_TOK; ++u) {
        if (u < n) {
          float xv[8];
          QbVec8<A>::load(x + (size_t)(t0 + u) * W + i, xv);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[u] = fmaf(wv[e], xv[e], acc[u]);
        }
      }
    }
  } else {
    for (int i = threadIdx.x; i < W; i += TI_WARPS * 32) {
      const float wv = qb_to_float<A>(wrow[i]);
#pragma unroll
      for (int u = 0; u < TI_TOK; ++u)
        if (u < n) acc[u] = fmaf(wv, qb_to_float<A>(x[(size_t)(t0 + u) * W + i]), acc[u]);
    }
  }
#pragma unroll
  for (int u = 0; u < TI_TOK; ++u) {
    const float s = qb_warp_sum(acc[u]);
    if (lane == 0) s_sum[warp][u] = s;
  }
  __syncthreads();
  if ((int)threadIdx.x < n) {
    float z = 0.f;
#pragma unroll
    for (int q = 0; q < TI_WARPS; ++q) z += s_sum[q][threadIdx.x];
    if (id < 0 || id >= V) qb_set_status(status, QB_STATUS_BAD_TOKEN, id, 1);
    const float v = id < 0 || id >= V ? 0.f : qb_gelu_tanh(z) * e_val;
    out[(size_t)(t0 + threadIdx.x) * D + j] = qb_from_float<A>(v);
  }
}

// x [T, W], w [D, W], table [V, table_stride] and out [T, D] in one dtype
extern "C" int qb_token_input_gate(const void* x, const void* w, const void* table, int table_stride, int offset,
                                   const int* ids, void* out, int dtype, int T, int W, int D, int V, int* status,
                                   cudaStream_t stream) {
  if (T <= 0) return 0;
  if (D <= 0 || W <= 0 || offset < 0 || offset + D > table_stride) return QB_ERR_BAD_ARG;
  const dim3 grid(D, (T + TI_TOK - 1) / TI_TOK);
  const bool vec = W % 8 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0;
  QB_DISPATCH_DTYPE(dtype, A, {
    if (vec) token_input_gate_kernel<A, true><<<grid, TI_WARPS * 32, 0, stream>>>(
        (const A*)x, (const A*)w, (const A*)table, table_stride, offset, ids, (A*)out, T, W, D, V, status);
    else token_input_gate_kernel<A, false><<<grid, TI_WARPS * 32, 0, stream>>>(
        (const A*)x, (const A*)w, (const A*)table, table_stride, offset, ids, (A*)out, T, W, D, V, status);
  });
  QB_LAUNCH_CHECK();
  return 0;
}
