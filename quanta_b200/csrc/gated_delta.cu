// Gated delta rule: a recurrence over time whose state is a matrix S [key channel i, value channel j] per
// (request, head), float32, kept in the request's state slot.  With one decay g and one write strength beta per
// (token, head), unit keys k and scaled unit queries q (shared by the heads of a group) and values v:
//
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q          (in this order)
//
// With a decay per key channel, g is a vector [D] per (token, head) and row i of S is multiplied by g[i].
//
// A first kernel turns the step's projections into what the chain reads: q and k of every (token, group) divided
// by sqrt(sum of squares + unit_eps), q also times q_scale; beta = sigmoid(b); g = exp(-exp(A_log) * softplus(a +
// dt_bias)), one number a head or D of them; all float32.  The recurrence is a chain in time.  A column j of S never meets another column, so
// eight neighbouring lanes own one column (lane p the rows 4 (p + 8 j) .. + 3) in registers for the whole step, and a
// block owns some columns of one (request, head).  Tokens are taken in chunks whose k, q, v, g and beta come into
// shared memory by asynchronous copies while the chunk before is walked.  A column's numbers do not depend on which
// block owns it.  Steps of portions take four tokens at a time (second half of this file): the same sums in another
// order, so the cut of a sequence shows in rounding only.
#include "common.cuh"

constexpr int GD_MAX_THREADS = 512;

// Block (t, y) of a token.  qk: float32 rows [q (G x D) | k (G x D) | ...] (row stride qk_stride); ab: float32 rows whose
// column b_off + h holds the pre-activation of beta (row stride ab_stride); a: float32 rows (row stride a_stride) of the
// decay's pre-activations, `per_head` numbers a head (1, or D for a decay per key channel), dt_bias laid out alike,
// A_log one number a head.  The blocks of a token share its decays; the first one also does the unit vectors and beta.
__global__ void gated_delta_prep_kernel(const float* __restrict__ qk, int qk_stride, const float* __restrict__ a,
                                        int a_stride, const float* __restrict__ ab, int ab_stride, int b_off,
                                        const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                                        float* __restrict__ q_out, float* __restrict__ k_out, float* __restrict__ g_out,
                                        float* __restrict__ beta_out, int T, int H, int G, int D, int per_head,
                                        float q_scale, float unit_eps) {
  const int t = blockIdx.x;
  if (t >= T) return;
  const int n_g = H * per_head;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < n_g; i += blockDim.x * gridDim.y) {
    const float z = a[(size_t)t * a_stride + i] + dt_bias[i];
    const float sp = z > 20.f ? z : log1pf(expf(z));
    g_out[(size_t)t * n_g + i] = expf(-expf(A_log[i / per_head]) * sp);
  }
  if (blockIdx.y != 0) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const float* row = qk + (size_t)t * qk_stride;
  for (int v = warp; v < 2 * G; v += nwarps) {          // v < G: the queries of group v; else the keys of group v - G
    const float* src = row + (size_t)v * D;
    float ss = 0.f;
    for (int i = lane; i < D; i += 32) ss += src[i] * src[i];
    ss = qb_warp_sum(ss);
    const float inv = (v < G ? q_scale : 1.f) / sqrtf(ss + unit_eps);
    float* dst = (v < G ? q_out + ((size_t)t * G + v) * D : k_out + ((size_t)t * G + (v - G)) * D);
    for (int i = lane; i < D; i += 32) dst[i] = src[i] * inv;
  }
  for (int h = threadIdx.x; h < H; h += blockDim.x)
    beta_out[(size_t)t * H + h] = 1.f / (1.f + expf(-ab[(size_t)t * ab_stride + b_off + h]));
}

__device__ __forceinline__ void gd_copy4(float* dst_smem, const float* src) {
  const unsigned d = (unsigned)__cvta_generic_to_shared(dst_smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

__device__ __forceinline__ void gd_copy16(float* dst_smem, const float* src) {
  const unsigned d = (unsigned)__cvta_generic_to_shared(dst_smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}

// GD_LANES neighbouring lanes own a column; RPT rows of it a lane: D <= GD_LANES * RPT; CH: a decay per key channel
template <int RPT, int GD_LANES, bool CH>
__global__ void __launch_bounds__(GD_MAX_THREADS, 1)
gated_delta_kernel(const float* __restrict__ q_in, const float* __restrict__ k_in, const float* __restrict__ v_in,
                   int v_stride, const float* __restrict__ g_in, const float* __restrict__ beta_in,
                   float* __restrict__ state, float* __restrict__ out, const int* __restrict__ req_start,
                   const int* __restrict__ req_slot, int H, int G, int D, int DV, int cols_per_block, int chunk) {
  extern __shared__ __align__(16) float sm[];
  constexpr int DP = GD_LANES * RPT;       // padded key channels
  const int r = blockIdx.x, h = blockIdx.y;
  const int grp = h / (H / G);
  const int col0 = blockIdx.z * cols_per_block;
  const int tid = threadIdx.x;
  const int p = tid % GD_LANES;
  const int jl = tid / GD_LANES;
  const int j = col0 + jl;
  const bool owns = jl < cols_per_block && j < DV;
  // a buffer: k [chunk, DP], q [chunk, DP], with CH g [chunk, DP], v [chunk, cols], g [chunk], beta [chunk]
  constexpr int PLANES = CH ? 3 : 2;
  const size_t plane = (size_t)chunk * DP;
  const size_t buf_floats = PLANES * plane + (size_t)chunk * cols_per_block + 2 * chunk;
  // the padding rows (i >= D) are read as zeros and never written
  for (size_t i = tid; i < 2 * buf_floats; i += blockDim.x) sm[i] = 0.f;

  const int t0 = req_start[r], t1 = req_start[r + 1];
  float* S = state + ((size_t)req_slot[r] * H + h) * D * DV;
  // a lane's rows: groups of four consecutive rows, 4 (p + 8 jj) .. + 3, so that it reads its k and q of a token as
  // 16-byte pieces and the eight lanes of a column read 128 consecutive bytes
  float col[RPT];
#pragma unroll
  for (int ii = 0; ii < RPT; ++ii) {
    const int i = 4 * (p + GD_LANES * (ii >> 2)) + (ii & 3);
    col[ii] = (owns && i < D) ? S[(size_t)i * DV + j] : 0.f;
  }
  __syncthreads();

  const bool wide = D % 4 == 0 && (((uintptr_t)k_in | (uintptr_t)q_in | (CH ? (uintptr_t)g_in : 0)) & 15) == 0;
  auto fetch = [&](int c0, int buf) {
    const int n = min(chunk, t1 - c0);
    float* b = sm + (size_t)buf * buf_floats;
    if (wide) {
      // rows of a multiple of four channels from 16-byte aligned arrays: four channels a copy
      for (int idx = tid; idx < n * (DP / 4); idx += blockDim.x) {
        const int tt = idx / (DP / 4), i = (idx % (DP / 4)) * 4;
        if (i < D) {
          const size_t gsrc = ((size_t)(c0 + tt) * G + grp) * D + i;
          gd_copy16(b + (size_t)tt * DP + i, k_in + gsrc);
          gd_copy16(b + plane + (size_t)tt * DP + i, q_in + gsrc);
          if (CH) gd_copy16(b + 2 * plane + (size_t)tt * DP + i, g_in + ((size_t)(c0 + tt) * H + h) * D + i);
        }
      }
    } else {
      for (int idx = tid; idx < n * DP; idx += blockDim.x) {
        const int tt = idx / DP, i = idx % DP;
        if (i < D) {
          const size_t gsrc = ((size_t)(c0 + tt) * G + grp) * D + i;
          gd_copy4(b + idx, k_in + gsrc);
          gd_copy4(b + plane + idx, q_in + gsrc);
          if (CH) gd_copy4(b + 2 * plane + idx, g_in + ((size_t)(c0 + tt) * H + h) * D + i);
        }
      }
    }
    float* bv = b + PLANES * plane;
    for (int idx = tid; idx < n * cols_per_block; idx += blockDim.x) {
      const int tt = idx / cols_per_block, c = idx % cols_per_block;
      if (col0 + c < DV) gd_copy4(bv + idx, v_in + (size_t)(c0 + tt) * v_stride + (size_t)h * DV + col0 + c);
    }
    float* bg = bv + (size_t)chunk * cols_per_block;
    for (int tt = tid; tt < n; tt += blockDim.x) {
      if (!CH) gd_copy4(bg + tt, g_in + (size_t)(c0 + tt) * H + h);
      gd_copy4(bg + chunk + tt, beta_in + (size_t)(c0 + tt) * H + h);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t0 < t1) fetch(t0, 0);
  int buf = 0;
  for (int c0 = t0; c0 < t1; c0 += chunk, buf ^= 1) {
    const int n = min(chunk, t1 - c0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                        // this chunk has landed, and everyone is done with the other buffer
    if (c0 + chunk < t1) fetch(c0 + chunk, buf ^ 1);
    const float* s_k = sm + (size_t)buf * buf_floats;
    const float* s_q = s_k + plane;
    const float* s_gc = s_q + plane;                       // CH: the decays per channel
    const float* s_v = s_k + PLANES * plane;
    const float* s_g = s_v + (size_t)chunk * cols_per_block;
    const float* s_b = s_g + chunk;
    for (int tt = 0; tt < n; ++tt) {
      const size_t o = (size_t)tt * DP;
      const float g = CH ? 1.f : s_g[tt], beta = s_b[tt];
      // four partial sums a dot product: the chain of dependent additions is a quarter as long
      float d4[4] = {0.f, 0.f, 0.f, 0.f};
      float4 k4[RPT / 4];
#pragma unroll
      for (int jj = 0; jj < RPT / 4; ++jj) {
        k4[jj] = *reinterpret_cast<const float4*>(s_k + o + 4 * (p + GD_LANES * jj));
        if (CH) {
          const float4 g4 = *reinterpret_cast<const float4*>(s_gc + o + 4 * (p + GD_LANES * jj));
          col[4 * jj + 0] *= g4.x; col[4 * jj + 1] *= g4.y; col[4 * jj + 2] *= g4.z; col[4 * jj + 3] *= g4.w;
        } else {
          col[4 * jj + 0] *= g; col[4 * jj + 1] *= g; col[4 * jj + 2] *= g; col[4 * jj + 3] *= g;
        }
        d4[0] += k4[jj].x * col[4 * jj + 0];
        d4[1] += k4[jj].y * col[4 * jj + 1];
        d4[2] += k4[jj].z * col[4 * jj + 2];
        d4[3] += k4[jj].w * col[4 * jj + 3];
      }
      float dot = (d4[0] + d4[1]) + (d4[2] + d4[3]);
      dot += __shfl_xor_sync(0xffffffffu, dot, 1);
      dot += __shfl_xor_sync(0xffffffffu, dot, 2);
      dot += __shfl_xor_sync(0xffffffffu, dot, 4);
      if (GD_LANES == 16) dot += __shfl_xor_sync(0xffffffffu, dot, 8);
      const float vj = owns ? s_v[(size_t)tt * cols_per_block + jl] : 0.f;
      const float u = beta * (vj - dot);
      float a4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int jj = 0; jj < RPT / 4; ++jj) {
        const float4 q4 = *reinterpret_cast<const float4*>(s_q + o + 4 * (p + GD_LANES * jj));
        col[4 * jj + 0] += k4[jj].x * u; col[4 * jj + 1] += k4[jj].y * u;
        col[4 * jj + 2] += k4[jj].z * u; col[4 * jj + 3] += k4[jj].w * u;
        a4[0] += q4.x * col[4 * jj + 0];
        a4[1] += q4.y * col[4 * jj + 1];
        a4[2] += q4.z * col[4 * jj + 2];
        a4[3] += q4.w * col[4 * jj + 3];
      }
      float acc = (a4[0] + a4[1]) + (a4[2] + a4[3]);
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      acc += __shfl_xor_sync(0xffffffffu, acc, 4);
      if (GD_LANES == 16) acc += __shfl_xor_sync(0xffffffffu, acc, 8);
      if (owns && p == 0) out[((size_t)(c0 + tt) * H + h) * DV + j] = acc;
    }
  }
#pragma unroll
  for (int ii = 0; ii < RPT; ++ii) {
    const int i = 4 * (p + GD_LANES * (ii >> 2)) + (ii & 3);
    if (owns && i < D) S[(size_t)i * DV + j] = col[ii];
  }
}

// ---------------------------------------------------------------------------------------------
// The same recurrence for portions, four tokens at a time.  Within a block of tokens 0 .. 3 that starts from the state S,
// with the products of decays G_i = g_0 .. g_i (elementwise, a vector over the key channels):
//
//   u_i = beta_i (v_i - S^T (k_i G_i) - sum_{j < i} A_ij u_j)       A_ij = k_i . (k_j g_(j+1) .. g_i)
//   o_i = S^T (q_i G_i) + sum_{j <= i} B_ij u_j                     B_ij = q_i . (k_j g_(j+1) .. g_i)
//   S  <- G_3 S + sum_j (k_j g_(j+1) .. g_3) u_j^T
//
// which is the recurrence with its terms gathered: the same products in another order, nothing is divided, so decays
// that underflow do no harm.  What does not depend on the state (the vectors k_i G_i, q_i G_i, k_j g_(j+1) .. g_3 and G_3,
// the sixteen numbers A and B, beta) is worked out for all blocks of the step side by side, a warp a (block, head), and
// laid down as one record; the chain then needs eight independent dot products and one chain of sums across lanes for
// four tokens instead of one for each.  Blocks are counted from the first token of a request's portion; a last block
// of fewer tokens is padded with keys, queries and write strengths of zero and decays of one.
constexpr int GB_TOK = 4;
constexpr int GB_STAGES = 4;
constexpr int GB_SCALARS = 20;              // A (above) and B (on and below the diagonal) of a 4 x 4 matrix, four betas

__host__ __device__ constexpr int gb_record(int dp) { return (3 * GB_TOK + 1) * dp + GB_SCALARS; }

// sums of 16 values over the warp's lanes, value i in the lanes 2 i and 2 i + 1
__device__ __forceinline__ float gb_sum16(float (&v)[16]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int n = 8, o = 16; n >= 1; n >>= 1, o >>= 1) {
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float send = (lane & o) ? v[i] : v[i + n], keep = (lane & o) ? v[i + n] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
}

// M: groups of four channels a lane holds, D <= 128 M.  One warp a (block, head); rec [block * H + head][gb_record(dp)].
template <int M>
__global__ void __launch_bounds__(128)
gated_delta_block_prep_kernel(const float* __restrict__ qk, int qk_stride, const float* __restrict__ a, int a_stride,
                              const float* __restrict__ ab, int ab_stride, int b_off, const float* __restrict__ A_log,
                              const float* __restrict__ dt_bias, float* __restrict__ rec,
                              const int* __restrict__ req_start, int R, int H, int G, int D, int dp, int per_channel,
                              float q_scale, float unit_eps) {
  const int lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (h >= H) return;
  // the request and the tokens of block blockIdx.x
  int t0 = -1, n = 0, acc = 0;
  for (int r = 0; r < R; ++r) {
    const int s0 = req_start[r], len = req_start[r + 1] - s0, nb = (len + GB_TOK - 1) / GB_TOK;
    if ((int)blockIdx.x < acc + nb) {
      t0 = s0 + ((int)blockIdx.x - acc) * GB_TOK;
      n = min(GB_TOK, s0 + len - t0);
      break;
    }
    acc += nb;
  }
  if (t0 < 0) return;
  const int grp = h / (H / G);
  float k[GB_TOK][4 * M], q[GB_TOK][4 * M], g[GB_TOK][4 * M];
  float ss[16];
#pragma unroll
  for (int i = 0; i < GB_TOK; ++i) {
    const float* krow = qk + (size_t)(t0 + i) * qk_stride + (size_t)(G + grp) * D;
    const float* qrow = qk + (size_t)(t0 + i) * qk_stride + (size_t)grp * D;
    float sk = 0.f, sq = 0.f, gh = 1.f;
    const float rate = -expf(A_log[h]);
    if (!per_channel && i < n) {
      const float z = a[(size_t)(t0 + i) * a_stride + h] + dt_bias[h];
      gh = expf(rate * (z > 20.f ? z : log1pf(expf(z))));
    }
#pragma unroll
    for (int m = 0; m < M; ++m) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = 4 * (lane + 32 * m) + e;
        const bool in = i < n && d < D;
        const float kv = in ? krow[d] : 0.f, qv = in ? qrow[d] : 0.f;
        float gv = gh;
        if (per_channel) {
          gv = 1.f;
          if (in) {
            const float z = a[(size_t)(t0 + i) * a_stride + (size_t)h * D + d] + dt_bias[(size_t)h * D + d];
            gv = expf(rate * (z > 20.f ? z : log1pf(expf(z))));
          }
        }
        k[i][4 * m + e] = kv; q[i][4 * m + e] = qv; g[i][4 * m + e] = gv;
        sk += kv * kv; sq += qv * qv;
      }
    }
    ss[i] = sk; ss[GB_TOK + i] = sq; ss[8 + i] = 0.f; ss[12 + i] = 0.f;
  }
  const float total = gb_sum16(ss);
#pragma unroll
  for (int i = 0; i < GB_TOK; ++i) {
    const float ik = 1.f / sqrtf(__shfl_sync(0xffffffffu, total, 2 * i) + unit_eps);
    const float iq = q_scale / sqrtf(__shfl_sync(0xffffffffu, total, 2 * (GB_TOK + i)) + unit_eps);
#pragma unroll
    for (int c = 0; c < 4 * M; ++c) { k[i][c] *= ik; q[i][c] *= iq; }
  }
  float* out = rec + ((size_t)blockIdx.x * H + h) * gb_record(dp);
  float cum[4 * M];
#pragma unroll
  for (int c = 0; c < 4 * M; ++c) cum[c] = 1.f;
#pragma unroll
  for (int i = 0; i < GB_TOK; ++i) {
#pragma unroll
    for (int m = 0; m < M; ++m) {
#pragma unroll
      for (int e = 0; e < 4; ++e) cum[4 * m + e] *= g[i][4 * m + e];
      const int d = 4 * (lane + 32 * m);
      if (d < dp) {
        const float4 pk = make_float4(k[i][4 * m] * cum[4 * m], k[i][4 * m + 1] * cum[4 * m + 1],
                                      k[i][4 * m + 2] * cum[4 * m + 2], k[i][4 * m + 3] * cum[4 * m + 3]);
        const float4 pq = make_float4(q[i][4 * m] * cum[4 * m], q[i][4 * m + 1] * cum[4 * m + 1],
                                      q[i][4 * m + 2] * cum[4 * m + 2], q[i][4 * m + 3] * cum[4 * m + 3]);
        *reinterpret_cast<float4*>(out + (size_t)i * dp + d) = pk;
        *reinterpret_cast<float4*>(out + (size_t)(GB_TOK + i) * dp + d) = pq;
        if (i == GB_TOK - 1)
          *reinterpret_cast<float4*>(out + (size_t)3 * GB_TOK * dp + d) =
              make_float4(cum[4 * m], cum[4 * m + 1], cum[4 * m + 2], cum[4 * m + 3]);
      }
    }
  }
  float mat[16];
#pragma unroll
  for (int j = 0; j < GB_TOK; ++j) {
    float cur[4 * M];
#pragma unroll
    for (int c = 0; c < 4 * M; ++c) cur[c] = k[j][c];
#pragma unroll
    for (int i = j; i < GB_TOK; ++i) {
      float sa = 0.f, sb = 0.f;
#pragma unroll
      for (int c = 0; c < 4 * M; ++c) {
        if (i > j) cur[c] *= g[i][c];
        sa += k[i][c] * cur[c];
        sb += q[i][c] * cur[c];
      }
      mat[4 * i + j] = sb;
      if (i > j) mat[4 * j + i] = sa;
    }
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int d = 4 * (lane + 32 * m);
      if (d < dp)
        *reinterpret_cast<float4*>(out + (size_t)(2 * GB_TOK + j) * dp + d) =
            make_float4(cur[4 * m], cur[4 * m + 1], cur[4 * m + 2], cur[4 * m + 3]);
    }
  }
  const float sum = gb_sum16(mat);
  float* sc = out + (size_t)(3 * GB_TOK + 1) * dp;
  if ((lane & 1) == 0) sc[lane >> 1] = sum;
  if (lane < GB_TOK)
    sc[16 + lane] = lane < n ? 1.f / (1.f + expf(-ab[(size_t)(t0 + lane) * ab_stride + b_off + h])) : 0.f;
}

__device__ __forceinline__ uint32_t gb_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ bool gb_try_wait(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
  return ok != 0;
}
// Bounded: false after 0.2 s or GB_SPIN_LIMIT tries.
constexpr uint32_t GB_SPIN_LIMIT = 1u << 22;
__device__ __forceinline__ bool gb_wait(uint32_t bar, uint32_t parity) {
  uint64_t t0 = 0;
  for (uint32_t it = 0; it < GB_SPIN_LIMIT; ++it) {
    if (gb_try_wait(bar, parity)) return true;
    if ((it & 127u) == 127u) {
      uint64_t now;
      asm volatile("mov.u64 %0, %globaltimer;" : "=l"(now));
      if (t0 == 0) t0 = now;
      else if (now - t0 > 200000000ull) break;
    }
  }
  return false;
}

__device__ __forceinline__ float gb_dot(const float4& x, const float* col, float acc) {
  acc = fmaf(x.x, col[0], acc); acc = fmaf(x.y, col[1], acc);
  acc = fmaf(x.z, col[2], acc); return fmaf(x.w, col[3], acc);
}

// A warp owns NC columns (four, or two where that gives every scheduler a second warp); lane p holds the rows
// 4 (p + 32 m) .. + 3 of each, m < M (D <= 128 M), so that a piece of a record is read once for NC columns.  The 8 NC
// partial sums of a block (eight dot products a column) are added across the lanes by halving: lane p ends up with dot
// product p % 8 of column (p / 8) % NC.
template <int M, int NC>
__global__ void __launch_bounds__(GD_MAX_THREADS, 1)
gated_delta_block_kernel(const float* __restrict__ rec, const float* __restrict__ v_in, int v_stride,
                         float* __restrict__ state, float* __restrict__ out, const int* __restrict__ req_start,
                         const int* __restrict__ req_slot, int H, int D, int DV, int cols_per_block, int* status) {
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(8) uint64_t s_full[GB_STAGES];
  static_assert(NC == 2 || NC == 4, "8 NC sums are dealt to 32 lanes");
  constexpr int DP = 128 * M, REC = gb_record(DP), NV = 8 * NC;
  const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * cols_per_block;
  const int tid = threadIdx.x, lane = tid & 31, warp_col = (tid >> 5) * NC;
  const int my_col = warp_col + (lane >> 3) % NC, kind = lane & 7;      // the column and the dot product this lane ends with
  const bool owns = col0 + my_col < DV;
  const int t0 = req_start[r], t1 = req_start[r + 1];
  if (t0 >= t1) return;
  const int n_blocks = (t1 - t0 + GB_TOK - 1) / GB_TOK;
  int first = 0;                              // the request's first block among the step's
  for (int i = 0; i < r; ++i) first += (req_start[i + 1] - req_start[i] + GB_TOK - 1) / GB_TOK;

  float* S = state + ((size_t)req_slot[r] * H + h) * D * DV;
  float col[NC][4 * M];
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int e = 0; e < 4 * M; ++e) {
      const int i = 4 * (lane + 32 * (e >> 2)) + (e & 3), j = col0 + warp_col + c;
      col[c][e] = (i < D && j < DV) ? S[(size_t)i * DV + j] : 0.f;
    }
  // a record arrives as one bulk copy that counts its bytes on the stage's barrier; the values of the lane's column come
  // straight into registers, a block ahead
  if (tid == 0) {
#pragma unroll
    for (int x = 0; x < GB_STAGES; ++x) asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(gb_smem(&s_full[x])));
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  auto fetch = [&](int b) {
    if (tid == 0 && b < n_blocks) {
      const uint32_t bar = gb_smem(&s_full[b % GB_STAGES]);
      asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"((uint32_t)(REC * 4)) : "memory");
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                       gb_smem(sm + (size_t)(b % GB_STAGES) * REC)),
                   "l"(rec + ((size_t)(first + b) * H + h) * REC), "r"((uint32_t)(REC * 4)), "r"(bar)
                   : "memory");
    }
  };
  const float* v_col = v_in + (size_t)h * DV + col0 + my_col;
  float v_next[GB_TOK];
  auto ask_values = [&](int b) {
#pragma unroll
    for (int i = 0; i < GB_TOK; ++i) {
      const int t = t0 + b * GB_TOK + i;
      v_next[i] = owns && t < t1 ? v_col[(size_t)t * v_stride] : 0.f;
    }
  };
#pragma unroll
  for (int b = 0; b < GB_STAGES - 1; ++b) fetch(b);
  ask_values(0);
  for (int b = 0; b < n_blocks; ++b) {
    const bool landed = gb_wait(gb_smem(&s_full[b % GB_STAGES]), (b / GB_STAGES) & 1);
    if (!__syncthreads_and(landed)) {         // also: everyone is done with the block before
      for (int x = b + 1; x < min(n_blocks, b + GB_STAGES - 1); ++x) gb_wait(gb_smem(&s_full[x % GB_STAGES]), (x / GB_STAGES) & 1);
      if (tid == 0) qb_set_status(status, QB_STATUS_WAIT_TIMEOUT, b, 9);
      return;
    }
    fetch(b + GB_STAGES - 1);
    const float v0 = v_next[0], v1 = v_next[1], v2 = v_next[2], v3 = v_next[3];
    ask_values(b + 1);
    const float* st = sm + (size_t)(b % GB_STAGES) * REC;
    const int n = min(GB_TOK, t1 - t0 - b * GB_TOK);
    float part[NV];
#pragma unroll
    for (int x = 0; x < NV; ++x) part[x] = 0.f;
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const float* base = st + 4 * (lane + 32 * m);
#pragma unroll
      for (int i = 0; i < 2 * GB_TOK; ++i) {
        const float4 x = *reinterpret_cast<const float4*>(base + i * DP);
#pragma unroll
        for (int c = 0; c < NC; ++c) part[8 * c + i] = gb_dot(x, col[c] + 4 * m, part[8 * c + i]);
      }
    }
#pragma unroll
    for (int w = NV / 2; w >= 1; w >>= 1) {
#pragma unroll
      for (int x = 0; x < w; ++x) {
        const float send = (lane & w) ? part[x] : part[x + w], keep = (lane & w) ? part[x + w] : part[x];
        part[x] = keep + __shfl_xor_sync(0xffffffffu, send, w);
      }
    }
    float mine = part[0];
    if (NC == 2) mine += __shfl_xor_sync(0xffffffffu, mine, 16);
    const float4* sc = reinterpret_cast<const float4*>(st + (3 * GB_TOK + 1) * DP);
    const float4 m0 = sc[0], m1 = sc[1], m2 = sc[2], m3 = sc[3], be = sc[4];
    // A_ij stands at row j, column i (above the diagonal), B_ij at row i, column j
    const int g8 = lane & 24;
    const float u0 = be.x * (v0 - __shfl_sync(0xffffffffu, mine, g8));
    const float u1 = be.y * (v1 - __shfl_sync(0xffffffffu, mine, g8 + 1) - m0.y * u0);
    const float u2 = be.z * (v2 - __shfl_sync(0xffffffffu, mine, g8 + 2) - m0.z * u0 - m1.z * u1);
    const float u3 = be.w * (v3 - __shfl_sync(0xffffffffu, mine, g8 + 3) - m0.w * u0 - m1.w * u1 - m2.w * u2);
    float u[NC][GB_TOK];
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      u[c][0] = __shfl_sync(0xffffffffu, u0, 8 * c);
      u[c][1] = __shfl_sync(0xffffffffu, u1, 8 * c);
      u[c][2] = __shfl_sync(0xffffffffu, u2, 8 * c);
      u[c][3] = __shfl_sync(0xffffffffu, u3, 8 * c);
    }
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const float* base = st + 4 * (lane + 32 * m);
      const float4 g4 = *reinterpret_cast<const float4*>(base + 3 * GB_TOK * DP);
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        float* s4 = col[c] + 4 * m;
        s4[0] *= g4.x; s4[1] *= g4.y; s4[2] *= g4.z; s4[3] *= g4.w;
      }
#pragma unroll
      for (int i = 0; i < GB_TOK; ++i) {
        const float4 x = *reinterpret_cast<const float4*>(base + (2 * GB_TOK + i) * DP);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float* s4 = col[c] + 4 * m;
          s4[0] = fmaf(x.x, u[c][i], s4[0]); s4[1] = fmaf(x.y, u[c][i], s4[1]);
          s4[2] = fmaf(x.z, u[c][i], s4[2]); s4[3] = fmaf(x.w, u[c][i], s4[3]);
        }
      }
    }
    // the lanes that ended with S^T (q_i G_i) write token i's output
    float o = mine + m0.x * u0;
    if (kind == 5) o = mine + m1.x * u0 + m1.y * u1;
    if (kind == 6) o = mine + m2.x * u0 + m2.y * u1 + m2.z * u2;
    if (kind == 7) o = mine + m3.x * u0 + m3.y * u1 + m3.z * u2 + m3.w * u3;
    if (owns && lane < NV && kind >= GB_TOK && kind - GB_TOK < n)
      out[((size_t)(t0 + b * GB_TOK + kind - GB_TOK) * H + h) * DV + col0 + my_col] = o;
  }
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int e = 0; e < 4 * M; ++e) {
      const int i = 4 * (lane + 32 * (e >> 2)) + (e & 3), j = col0 + warp_col + c;
      if (i < D && j < DV) S[(size_t)i * DV + j] = col[c][e];
    }
}

// whether a step of T tokens in R requests takes the blocks of four tokens (portions of sixteen and more on average)
extern "C" int qb_gated_delta_in_blocks(int T, int R) { return T >= 16 * R ? 1 : 0; }

// floats of scratch memory that qb_gated_delta needs
extern "C" long long qb_gated_delta_scratch(int T, int R, int H, int G, int D, int per_channel) {
  const long long token = (long long)T * (2LL * G * D + (long long)H * (per_channel ? D : 1) + H);
  return qb_gated_delta_in_blocks(T, R) ? ((long long)T / GB_TOK + R) * H * gb_record(D <= 128 ? 128 : 256) : token;
}

// qkv: float32 rows [q (G x D) | k (G x D) | v (H x DV)] after convolution and activation (row stride qkv_stride);
// a: float32 rows of the decay's pre-activations, one a head or (per_channel) D a head; ab: float32 rows with the
// pre-activations of beta (b_off + h); scratch: qb_gated_delta_scratch floats; out: float32 [T, H, DV].
extern "C" int qb_gated_delta(const float* qkv, int qkv_stride, const float* a, int a_stride, const float* ab,
                              int ab_stride, int b_off, int per_channel, const float* A_log, const float* dt_bias,
                              float* state, float* out, float* scratch, const int* req_start, const int* req_slot, int R,
                              int T, int H, int G, int D, int DV, float q_scale, float unit_eps, int* status,
                              cudaStream_t stream) {
  if (R <= 0 || T <= 0) return 0;
  if (D <= 0 || D > 256 || DV <= 0 || DV > 256 || H <= 0 || G <= 0 || H % G) return QB_ERR_UNSUPPORTED;
  const int lanes = 8;
  const int per_lane = (D + lanes - 1) / lanes;
  const int rpt = per_lane <= 4 ? 4 : per_lane <= 8 ? 8 : per_lane <= 16 ? 16 : 32;
  const int dp = rpt * lanes;
  // columns a block: all of them (at most max_cols) unless that leaves most SMs idle; then fewer, down to 16
  // where requests bring portions and down to 4 where every request brings one token; a multiple of 4: whole warps
  const int max_cols = GD_MAX_THREADS / lanes;
  const int min_cols = T > R ? 16 : 4;
  int splits = (DV + max_cols - 1) / max_cols;
  while ((long)R * H * splits < 132 && (DV + 2 * splits - 1) / (2 * splits) >= min_cols) splits *= 2;
  int cols = (DV + splits - 1) / splits;
  cols = (cols + 3) / 4 * 4;
  splits = (DV + cols - 1) / cols;
  const int threads = cols * lanes;
  const dim3 grid(R, H, splits);
  const float* v_in = qkv + (size_t)2 * G * D;
  if (qb_gated_delta_in_blocks(T, R)) {
    const dim3 bgrid(T / GB_TOK + R, (H + 3) / 4);
    const int bdp = D <= 128 ? 128 : 256;
    const size_t bsmem = (size_t)GB_STAGES * gb_record(bdp) * sizeof(float);
    // a second warp a scheduler where four columns a warp leave one or none
    const bool two = (long)R * H * DV <= 4L * 592 && cols <= 32;
#define GB_LAUNCH(M, NC)                                                                                   \
  do {                                                                                                     \
    gated_delta_block_prep_kernel<M><<<bgrid, 128, 0, stream>>>(                                           \
        qkv, qkv_stride, a, a_stride, ab, ab_stride, b_off, A_log, dt_bias, scratch, req_start, R, H, G,   \
        D, bdp, per_channel, q_scale, unit_eps);                                                           \
    QB_LAUNCH_CHECK();                                                                                     \
    auto kern = gated_delta_block_kernel<M, NC>;                                                           \
    if (bsmem + 1024 > 48 * 1024) {   /* the kernel also has some static shared memory */                   \
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bsmem); \
      if (e != cudaSuccess) return (int)e;                                                                 \
    }                                                                                                      \
    kern<<<grid, cols / NC * 32, bsmem, stream>>>(scratch, v_in, qkv_stride, state, out, req_start, req_slot, H,  \
                                           D, DV, cols, status);                                            \
  } while (0)
    if (bdp == 128 && two) GB_LAUNCH(1, 2);
    else if (bdp == 128) GB_LAUNCH(1, 4);
    else if (two) GB_LAUNCH(2, 2);
    else GB_LAUNCH(2, 4);
#undef GB_LAUNCH
    QB_LAUNCH_CHECK();
    return 0;
  }
  const size_t n = (size_t)T * G * D;
  const int per_head = per_channel ? D : 1;
  float *q_s = scratch, *k_s = scratch + n, *g_s = scratch + 2 * n, *b_s = g_s + (size_t)T * H * per_head;
  const dim3 pgrid(T, T >= 512 ? 1 : min(32, (H * per_head + 255) / 256));
  gated_delta_prep_kernel<<<pgrid, 256, 0, stream>>>(qkv, qkv_stride, a, a_stride, ab, ab_stride, b_off, A_log, dt_bias,
                                                     q_s, k_s, g_s, b_s, T, H, G, D, per_head, q_scale, unit_eps);
  QB_LAUNCH_CHECK();
  // eight lanes a column.  Sixteen (half the multiply-adds a lane and token for one more step of the sums) were
  // measured: no faster on a prompt (637 against 631 us for 2,048 tokens, 16 heads of 128 x 128) and slower for single
  // tokens (22 against 14 us for 8 requests), whose state rows then come in shorter pieces
  const int chunk = dp <= 128 ? 16 : 8;
  const size_t smem = (size_t)2 * ((per_channel ? 3 : 2) * chunk * dp + chunk * cols + 2 * chunk) * sizeof(float);
#define GD_LAUNCH_AS(N, L, CH)                                                                              \
  do {                                                                                                     \
    auto kern = gated_delta_kernel<N, L, CH>;                                                                \
    if (smem > 48 * 1024) {                                                                                \
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);  \
      if (e != cudaSuccess) return (int)e;                                                                 \
    }                                                                                                      \
    kern<<<grid, threads, smem, stream>>>(q_s, k_s, v_in, qkv_stride, g_s, b_s, state, out, req_start,     \
                                          req_slot, H, G, D, DV, cols, chunk);                             \
  } while (0)
#define GD_LAUNCH(N, L)                   \
  do {                                    \
    if (per_channel) GD_LAUNCH_AS(N, L, true); \
    else GD_LAUNCH_AS(N, L, false);       \
  } while (0)
  if (rpt == 4) GD_LAUNCH(4, 8);
  else if (rpt == 8) GD_LAUNCH(8, 8);
  else if (rpt == 16) GD_LAUNCH(16, 8);
  else GD_LAUNCH(32, 8);
#undef GD_LAUNCH
#undef GD_LAUNCH_AS
  QB_LAUNCH_CHECK();
  return 0;
}
