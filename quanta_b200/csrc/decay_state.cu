// Linear recurrences over time whose state is a matrix S [key channel i, value channel j] per (request, head) with ONE
// decay a (token, head), float32, kept in the request's state slot:
//
//   S_t = a_t S_(t-1) + w_t k_t v_t^T          o_t = q_scale * S_t^T q_t
//
// and optionally a normaliser n_t = a_t n_(t-1) + w_t k_t with den_t = max(|q_scale * n_t . q_t|, floor_t) + 1e-6.
// Head h reads the queries and keys of group h / (H / G).  Where a_t and w_t come from (DsGates):
//   constant   a_t = decay[h], w_t = 1                                              (linear attention with fixed decays)
//   step       dt = softplus(x_t + bias[h]), a_t = exp(-exp(A_log[h]) dt), w_t = dt  (state-space models)
//   given      a_t = exp(log_decay[t, h]), w_t = weight[t, h]                        (exponential gates, below)
//
// Exponential gates with a running maximum m (memory_gates_kernel): from pre-activations x_i, x_f of a token and head,
//   i = cap tanh((x_i + b_i) / cap), f = logsigmoid(cap tanh((x_f + b_f) / cap)), m_t = max(f + m_(t-1), i),
//   log_decay = f + m_(t-1) - m_t, weight = exp(i - m_t), floor = exp(-m_t).
// m is a scan of the maps m -> max(f + m, i), which compose; it is done in double and rounded once a token, so a cut
// of the sequence changes nothing but that rounding.
//
// Two forms of the recurrence:
//  * ds_chain_kernel, float32 arithmetic on the CUDA cores, token by token: single tokens, short portions, the float32
//    mode and sizes the other form does not take.  A block owns 16 or 32 columns of one (request, head); a thread
//    holds a few rows of four columns in registers, a turn takes four tokens.
//  * ds_chunk_kernel, bfloat16 inputs, chunks of 64 tokens on the tensor cores (mma.sync): with L the cumulated
//    log decays of a chunk,
//      o_t = exp(L_t) S_0^T q_t + sum_{j <= t} exp(L_t - L_j) w_j (q_t . k_j) v_j
//      S   = exp(L_end) S_0 + sum_j k_j (exp(L_end - L_j) w_j v_j)^T
//    A block owns up to 64 columns of one (request, head) and walks its chunks with S in accumulators.  What is not
//    bfloat16 to begin with (S, the weighted scores, the weighted values) enters a product as the sum of two bfloat16
//    parts, 16 bits of mantissa; sums, decays and the state itself are float32.  L is cumulated in double and kept as
//    a float pair, so that differences of two large L keep their low bits.
//    A prompt whose (head, column) blocks do not fill the GPU runs as segments of several chunks in three passes:
//    every segment from a zero state, the segments joined in order, every segment again from its true start.
#include "common.cuh"

constexpr int DS_CONST = 0, DS_STEP = 1;     // kinds of gates; 2: given
constexpr float DS_LOG_FLOOR = -1e4f;      // a smaller log decay is a decay of zero in float32 all the same
constexpr float DS_DEN_EPS = 1e-6f;        // added to the normaliser

struct DsGates {
  int kind;
  const float* decay;        // constant: [H]
  const float* log_decay;    // constant: [H]; given: [T, H]
  const float* step;         // step: rows of step_stride floats, one number a head
  int step_stride;
  const float* step_bias;    // [H]
  const float* A_log;        // [H]
  const float* weight;       // given: [T, H]
};

__device__ __forceinline__ float ds_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// the natural logarithm of the decay and the weight of token t, head h
__device__ __forceinline__ void ds_log_gate(const DsGates& g, int t, int h, int H, float& la, float& w) {
  if (g.kind == DS_CONST) {
    la = g.log_decay[h];
    w = 1.f;
  } else if (g.kind == DS_STEP) {
    w = ds_softplus(g.step[(size_t)t * g.step_stride + h] + g.step_bias[h]);
    la = -expf(g.A_log[h]) * w;
  } else {
    la = g.log_decay[(size_t)t * H + h];
    w = g.weight[(size_t)t * H + h];
  }
}

// ---------------------------------------------------------------------------------------------
// exponential gates
// ---------------------------------------------------------------------------------------------
constexpr int DS_GATE_RUN = 2;        // tokens a thread walks

__device__ __forceinline__ void ds_raw_gates(const float* __restrict__ proj, int stride, int i_off, int f_off, int t,
                                             int h, float bi, float bf, float cap, float& i, float& f) {
  i = cap * tanhf((proj[(size_t)t * stride + i_off + h] + bi) / cap);
  const float z = cap * tanhf((proj[(size_t)t * stride + f_off + h] + bf) / cap);
  f = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

// A block a (request, head); the request's rows in turns of blockDim * DS_GATE_RUN.
__global__ void memory_gates_kernel(const float* __restrict__ proj, int stride, int i_off, int f_off,
                                    const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap,
                                    float* __restrict__ m_state, float* __restrict__ log_decay, float* __restrict__ weight,
                                    float* __restrict__ floor_out, const int* __restrict__ req_start,
                                    const int* __restrict__ req_slot, int H) {
  __shared__ double s_a[32], s_b[32];
  const int r = blockIdx.x, h = blockIdx.y;
  const int t0 = req_start[r], t1 = req_start[r + 1];
  if (t1 <= t0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
  const float bi = i_bias[h], bf = f_bias[h];
  float* m_at = m_state + (size_t)req_slot[r] * H + h;
  double m_in = (double)*m_at;                      // before the turn's first token
  for (int base = t0; base < t1; base += (int)blockDim.x * DS_GATE_RUN) {
    const int first = base + tid * DS_GATE_RUN;
    float iv[DS_GATE_RUN], fv[DS_GATE_RUN];
    double a = 0.0, b = -1e300;                     // the run's map m -> max(a + m, b)
#pragma unroll
    for (int u = 0; u < DS_GATE_RUN; ++u) {
      iv[u] = fv[u] = 0.f;
      if (first + u < t1) {
        ds_raw_gates(proj, stride, i_off, f_off, first + u, h, bi, bf, cap, iv[u], fv[u]);
        a += (double)fv[u];
        b = fmax(b + (double)fv[u], (double)iv[u]);
      }
    }
    // inclusive scan of the maps over the block's threads, earlier maps applied first
    double A = a, B = b;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double pa = __shfl_up_sync(0xffffffffu, A, o), pb = __shfl_up_sync(0xffffffffu, B, o);
      if (lane >= o) {
        B = fmax(A + pb, B);
        A += pa;
      }
    }
    __syncthreads();                                // the turn before has been read
    if (lane == 31) { s_a[warp] = A; s_b[warp] = B; }
    __syncthreads();
    double m = m_in;
    for (int w = 0; w < warp; ++w) m = fmax(s_a[w] + m, s_b[w]);
    const double ea = __shfl_up_sync(0xffffffffu, A, 1), eb = __shfl_up_sync(0xffffffffu, B, 1);
    if (lane > 0) m = fmax(ea + m, eb);
    for (int w = 0; w < n_warps; ++w) m_in = fmax(s_a[w] + m_in, s_b[w]);
#pragma unroll
    for (int u = 0; u < DS_GATE_RUN; ++u) {
      if (first + u < t1) {
        const double before = (double)(float)m;     // as the state of a portion that ends here keeps it
        m = fmax((double)fv[u] + m, (double)iv[u]);
        const float now = (float)m;
        const size_t at = (size_t)(first + u) * H + h;
        log_decay[at] = (float)((double)fv[u] + before - (double)now);
        weight[at] = expf((float)((double)iv[u] - (double)now));
        floor_out[at] = expf(-now);
      }
    }
  }
  if (tid == 0) *m_at = (float)m_in;
}

// The same for a step of single tokens: a thread a (request, head), the same numbers without the scan.
__global__ void memory_gates_single_kernel(const float* __restrict__ proj, int stride, int i_off, int f_off,
                                           const float* __restrict__ i_bias, const float* __restrict__ f_bias, float cap,
                                           float* __restrict__ m_state, float* __restrict__ log_decay,
                                           float* __restrict__ weight, float* __restrict__ floor_out,
                                           const int* __restrict__ req_slot, int R, int H) {
  const int at = blockIdx.x * blockDim.x + threadIdx.x;        // token r of request r
  if (at >= R * H) return;
  const int r = at / H, h = at % H;
  float* m_at = m_state + (size_t)req_slot[r] * H + h;
  float iv, fv;
  ds_raw_gates(proj, stride, i_off, f_off, r, h, i_bias[h], f_bias[h], cap, iv, fv);
  const double before = (double)*m_at, m = fmax((double)fv + before, (double)iv);
  const float now = (float)m;
  log_decay[at] = (float)((double)fv + before - (double)now);
  weight[at] = expf((float)((double)iv - (double)now));
  floor_out[at] = expf(-now);
  *m_at = now;
}

extern "C" int qb_memory_gates(const float* proj, int stride, int i_off, int f_off, const float* i_bias,
                               const float* f_bias, float cap, float* m_state, float* log_decay, float* weight,
                               float* floor_out, const int* req_start, const int* req_slot, int T, int R, int H,
                               cudaStream_t stream) {
  if (T <= 0 || R <= 0) return 0;
  if (H <= 0 || H > 65535 || !(cap > 0.f)) return QB_ERR_BAD_ARG;
  if (T == R) {                                     // every request of a step brings at least one token
    memory_gates_single_kernel<<<(R * H + 63) / 64, 64, 0, stream>>>(proj, stride, i_off, f_off, i_bias, f_bias, cap, m_state,
                                                                     log_decay, weight, floor_out, req_slot, R, H);
    QB_LAUNCH_CHECK();
    return 0;
  }
  int threads = 64;
  while (threads < 1024 && threads * DS_GATE_RUN < T) threads *= 2;
  memory_gates_kernel<<<dim3(R, H), threads, 0, stream>>>(proj, stride, i_off, f_off, i_bias, f_bias, cap, m_state,
                                                         log_decay, weight, floor_out, req_start, req_slot, H);
  QB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------------------------
// token by token, float32
// ---------------------------------------------------------------------------------------------
constexpr int DS_TURN = 4;             // tokens a turn (one where every request brings a single token)
constexpr int DS_CHAIN_THREADS = 256;

struct DsShape {
  int H, G, D, E;
  long long stride;                    // elements between two token rows of q, k and v
};

// VEC columns a thread (4, or 1 where E is no multiple of 4), NR rows a thread, TB tokens a turn; cols: columns a block.
template <typename U, int VEC, int NR, int TB>
__global__ void __launch_bounds__(DS_CHAIN_THREADS, TB == 1 && VEC == 4 && NR <= 4 ? 4 : 1)
ds_chain_kernel(const U* __restrict__ q, const U* __restrict__ k, const U* __restrict__ v, DsShape sh, DsGates gates,
                float* __restrict__ state, float* __restrict__ n_state, const float* __restrict__ floor_in,
                float* __restrict__ den, float* __restrict__ out, const int* __restrict__ req_start,
                const int* __restrict__ req_slot, float q_scale, int silu, int cols, int max_tokens) {
  extern __shared__ __align__(16) float ds_sm[];
  const int D = sh.D, E = sh.E, H = sh.H;
  float* s_k = ds_sm;                          // [TB][D]
  float* s_q = s_k + TB * D;                // [TB][D]
  float* s_v = s_q + TB * D;                // [TB][cols]
  float* s_red = s_v + TB * cols;           // [warps][TB][cols]
  float* s_a = s_red + (DS_CHAIN_THREADS / 32) * TB * cols;   // [TB]
  float* s_w = s_a + TB;                    // [TB]
  const int r = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * cols;
  const int t0 = req_start[r], t1 = req_start[r + 1];
  if (t1 <= t0 || t1 - t0 > max_tokens) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int CQ = cols / VEC, RG = DS_CHAIN_THREADS / CQ;
  const int cq = tid % CQ, rg = tid / CQ;
  const int c0 = e0 + cq * VEC;
  const bool owns = c0 < E;
  const int g = h / (H / sh.G);
  float* S = state + ((size_t)req_slot[r] * H + h) * D * E;
  float s[NR][VEC];
#pragma unroll
  for (int u = 0; u < NR; ++u) {
    const int i = rg + RG * u;
    if (owns && i < D) {
      if constexpr (VEC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(S + (size_t)i * E + c0);
        s[u][0] = x.x; s[u][1] = x.y; s[u][2] = x.z; s[u][3] = x.w;
      } else {
        s[u][0] = S[(size_t)i * E + c0];
      }
    } else {
#pragma unroll
      for (int c = 0; c < VEC; ++c) s[u][c] = 0.f;
    }
  }
  // the normaliser belongs to one warp of the block with the head's first columns
  const bool norms = n_state != nullptr && blockIdx.z == 0 && warp == 0;
  float* N = norms ? n_state + ((size_t)req_slot[r] * H + h) * D : nullptr;
  float nn[8];
#pragma unroll
  for (int u = 0; u < 8; ++u) nn[u] = norms && lane + 32 * u < D ? N[lane + 32 * u] : 0.f;

  auto act = [&](float x) { return silu ? x / (1.f + expf(-x)) : x; };
  for (int tb = t0; tb < t1; tb += TB) {
    const int nt = min(TB, t1 - tb);
    for (int i = tid; i < nt * D; i += DS_CHAIN_THREADS) {
      const int tt = i / D, d = i % D;
      const size_t row = (size_t)(tb + tt) * sh.stride + (size_t)g * D + d;
      s_k[i] = act(qb_to_float<U>(k[row]));
      s_q[i] = act(qb_to_float<U>(q[row]));
    }
    for (int i = tid; i < nt * cols; i += DS_CHAIN_THREADS) {
      const int tt = i / cols, c = i % cols;
      s_v[i] = e0 + c < E ? act(qb_to_float<U>(v[(size_t)(tb + tt) * sh.stride + (size_t)h * E + e0 + c])) : 0.f;
    }
    if (tid < nt) {
      float la, w;
      ds_log_gate(gates, tb + tid, h, H, la, w);
      s_a[tid] = gates.kind == DS_CONST ? gates.decay[h] : expf(la);
      s_w[tid] = w;
    }
    __syncthreads();
    float acc[TB][VEC];
#pragma unroll
    for (int tt = 0; tt < TB; ++tt) {
#pragma unroll
      for (int c = 0; c < VEC; ++c) acc[tt][c] = 0.f;
      if (tt < nt) {
        const float a = s_a[tt], w = s_w[tt];
        float wv[VEC];
#pragma unroll
        for (int c = 0; c < VEC; ++c) wv[c] = w * s_v[tt * cols + cq * VEC + c];
#pragma unroll
        for (int u = 0; u < NR; ++u) {
          const int i = rg + RG * u;
          if (i < D) {
            const float ki = s_k[tt * D + i], qi = s_q[tt * D + i];
#pragma unroll
            for (int c = 0; c < VEC; ++c) {
              s[u][c] = fmaf(a, s[u][c], ki * wv[c]);
              acc[tt][c] = fmaf(qi, s[u][c], acc[tt][c]);
            }
          }
        }
      }
    }
    if (norms) {
      for (int tt = 0; tt < nt; ++tt) {
        const float a = s_a[tt], w = s_w[tt];
        float dot = 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const int i = lane + 32 * u;
          if (i < D) {
            nn[u] = fmaf(a, nn[u], w * s_k[tt * D + i]);
            dot = fmaf(s_q[tt * D + i], nn[u], dot);
          }
        }
        dot = qb_warp_sum(dot);
        if (lane == 0) {
          const size_t at = (size_t)(tb + tt) * H + h;
          den[at] = fmaxf(fabsf(dot * q_scale), floor_in[at]) + DS_DEN_EPS;
        }
      }
    }
    // the row groups' sums: lanes of the same columns, then the warps in order
#pragma unroll
    for (int tt = 0; tt < TB; ++tt) {
#pragma unroll
      for (int c = 0; c < VEC; ++c) {
        if (tt < nt) {
          float x = acc[tt][c];
          for (int o = CQ; o < 32; o <<= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
          if (lane < CQ) s_red[(warp * TB + tt) * cols + cq * VEC + c] = x;
        }
      }
    }
    __syncthreads();
    for (int i = tid; i < nt * cols; i += DS_CHAIN_THREADS) {
      const int tt = i / cols, c = i % cols;
      if (e0 + c < E) {
        float x = 0.f;
#pragma unroll
        for (int w = 0; w < DS_CHAIN_THREADS / 32; ++w) x += s_red[(w * TB + tt) * cols + c];
        out[((size_t)(tb + tt) * H + h) * E + e0 + c] = x * q_scale;
      }
    }
  }
#pragma unroll
  for (int u = 0; u < NR; ++u) {
    const int i = rg + RG * u;
    if (owns && i < D) {
      if constexpr (VEC == 4)
        *reinterpret_cast<float4*>(S + (size_t)i * E + c0) = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
      else
        S[(size_t)i * E + c0] = s[u][0];
    }
  }
#pragma unroll
  for (int u = 0; u < 8; ++u)
    if (norms && lane + 32 * u < D) N[lane + 32 * u] = nn[u];
}

// q, k, v: rows of `stride` elements of in_dtype (the pointers at the first column of each).  state float32
// [slots, H, D, E]; n_state float32 [slots, H, D] with floor_in and den float32 [T, H], or all three null; out float32
// [T, H, E].  silu: q, k and v pass through it as they are read.  Requests that bring more than max_tokens tokens are
// left alone.
extern "C" int qb_decay_chain(const void* q, const void* k, const void* v, int in_dtype, long long stride, int kind,
                              const float* decay, const float* log_decay, const float* step, int step_stride,
                              const float* step_bias, const float* A_log, const float* weight, float* state,
                              float* n_state, const float* floor_in, float* den, float* out, const int* req_start,
                              const int* req_slot, int T, int R, int H, int G, int D, int E, float q_scale, int silu,
                              int max_tokens, cudaStream_t stream) {
  if (T <= 0 || R <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || E <= 0 || kind < 0 || kind > 2) return QB_ERR_BAD_ARG;
  if (D > 256 || H > 65535) return QB_ERR_UNSUPPORTED;
  const bool vec = E % 4 == 0 && ((uintptr_t)state & 15) == 0;
  const int cols = vec && E <= 16 ? 16 : 32;
  const int rg = DS_CHAIN_THREADS / (cols / (vec ? 4 : 1));
  const int nr = (D + rg - 1) / rg;
  const dim3 grid(R, H, (E + cols - 1) / cols);
  const bool single = T == R;                       // every request of a step brings at least one token
  const int turn = single ? 1 : DS_TURN;
  const size_t smem = (size_t)turn * (2 * D + cols + (DS_CHAIN_THREADS / 32) * cols + 2) * sizeof(float);
  const DsShape sh{H, G, D, E, stride};
  const DsGates gates{kind, decay, log_decay, step, step_stride, step_bias, A_log, weight};
#define DS_CHAIN(VEC, NR)                                                                                          \
  if (single) DS_CHAIN_TURN(VEC, NR, 1); else DS_CHAIN_TURN(VEC, NR, DS_TURN)
#define DS_CHAIN_TURN(VEC, NR, TB_)                                                                                \
  ds_chain_kernel<U, VEC, NR, TB_><<<grid, DS_CHAIN_THREADS, smem, stream>>>(                                           \
      (const U*)q, (const U*)k, (const U*)v, sh, gates, state, n_state, floor_in, den, out, req_start, req_slot,   \
      q_scale, silu, cols, max_tokens)
  QB_DISPATCH_DTYPE(in_dtype, U, {
    if (vec) {
      if (nr <= 1) { DS_CHAIN(4, 1); }
      else if (nr <= 2) { DS_CHAIN(4, 2); }
      else if (nr <= 4) { DS_CHAIN(4, 4); }
      else { DS_CHAIN(4, 8); }
    } else {
      if (nr <= 4) { DS_CHAIN(1, 4); }
      else if (nr <= 8) { DS_CHAIN(1, 8); }
      else if (nr <= 16) { DS_CHAIN(1, 16); }
      else { DS_CHAIN(1, 32); }
    }
  });
#undef DS_CHAIN
#undef DS_CHAIN_TURN
  QB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------------------------
// chunks of tokens on the tensor cores
// ---------------------------------------------------------------------------------------------
constexpr int DS_C = 64;                // tokens a chunk
constexpr int DS_CHUNK_THREADS = 256;
constexpr int DS_DIRECT = 0, DS_LOCAL = 1, DS_REPLAY = 2;

__device__ __forceinline__ void ds_ldsm(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ds_ldsm_t(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ds_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ds_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two floats as bfloat16 pairs: their roundings, and the roundings of what is left
__device__ __forceinline__ void ds_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 b = __floats2bfloat162_rn(x - __low2float(a), y - __high2float(a));
  hi = *reinterpret_cast<const uint32_t*>(&a);
  lo = *reinterpret_cast<const uint32_t*>(&b);
}

// The segments of a step: the rows of every request that brings at least min_tokens, in runs of seg_len.  seg[s] = (first
// row, end row, request row, 0); req_seg[r] = (first segment, segments).  One block; R <= 1024.
__global__ void ds_segments_kernel(const int* __restrict__ req_start, int R, int seg_len, int min_tokens, int max_seg,
                                   int4* __restrict__ seg, int2* __restrict__ req_seg, int* __restrict__ n_seg) {
  __shared__ int s_n[1024];
  const int r = threadIdx.x;
  const int t0 = r < R ? req_start[r] : 0, t1 = r < R ? req_start[r + 1] : 0;
  const int n = t1 - t0 >= min_tokens ? (t1 - t0 + seg_len - 1) / seg_len : 0;
  s_n[r] = n;
  __syncthreads();
  for (int o = 1; o < 1024; o <<= 1) {
    const int a = r >= o ? s_n[r - o] : 0;
    __syncthreads();
    s_n[r] += a;
    __syncthreads();
  }
  const int first = s_n[r] - n;
  if (r < R) {
    req_seg[r] = make_int2(first, n);
    for (int c = 0; c < n && first + c < max_seg; ++c)
      seg[first + c] = make_int4(t0 + c * seg_len, min(t1, t0 + (c + 1) * seg_len), r, 0);
  }
  if (r == 1023) n_seg[0] = min(s_n[r], max_seg);
}

// Over a request's segments in order: x <- 2^(log decay) x + (the segment's own contribution), which makes room for the
// value the segment starts from.  A thread a number of S (and, behind them, of n).
__global__ void ds_combine_kernel(float* __restrict__ state, float* __restrict__ n_state, float* __restrict__ seg_state,
                                  float* __restrict__ seg_n, const float* __restrict__ seg_log,
                                  const int2* __restrict__ req_seg, const int* __restrict__ req_slot, int H, int D, int E) {
  const int r = blockIdx.x, h = blockIdx.y;
  const int2 rs = req_seg[r];
  if (rs.y == 0) return;
  const int DE = D * E, total = DE + (n_state != nullptr ? D : 0);
  const size_t own = (size_t)req_slot[r] * H + h;
  for (int idx = blockIdx.z * blockDim.x + threadIdx.x; idx < total; idx += gridDim.z * blockDim.x) {
    const bool is_n = idx >= DE;
    float* at = is_n ? n_state + own * D + (idx - DE) : state + own * DE + idx;
    float* part = is_n ? seg_n + (idx - DE) : seg_state + idx;
    const size_t pitch = is_n ? D : DE;
    float x = *at;
    for (int c0 = 0; c0 < rs.y; c0 += 8) {          // the loads of eight segments are in flight together
      float l[8], p[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        if (c0 + u < rs.y) {
          const size_t sg = (size_t)(rs.x + c0 + u) * H + h;
          l[u] = __ldcg(part + sg * pitch);
          p[u] = exp2f(__ldcg(seg_log + sg));
        }
      }
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        if (c0 + u < rs.y) {
          part[((size_t)(rs.x + c0 + u) * H + h) * pitch] = x;
          x = fmaf(p[u], x, l[u]);
        }
      }
    }
    *at = x;
  }
}

struct DsTrue { static constexpr bool value = true; };
struct DsFalse { static constexpr bool value = false; };

// NM: D <= 64 NM; ET: columns a block; LOCAL: no outputs, from a zero state.  Eight warps: of the outputs a warp takes 16
// tokens and half of the columns (both halves of a token work out its scores); of S it takes MT tiles of 16 channels and
// SN of the NT tiles of 8 columns.
template <int NM, int ET, bool LOCAL>
__global__ void __launch_bounds__(DS_CHUNK_THREADS, NM <= 2 ? 2 : 1)
ds_chunk_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k,
                const __nv_bfloat16* __restrict__ v, DsShape sh, DsGates gates, float* __restrict__ state,
                float* __restrict__ n_state, const float* __restrict__ floor_in, float* __restrict__ den,
                float* __restrict__ out, const int* __restrict__ req_start, const int* __restrict__ req_slot,
                const int4* __restrict__ seg, const int* __restrict__ n_seg, float* __restrict__ seg_state,
                float* __restrict__ seg_n, float* __restrict__ seg_log, int mode, float q_scale, int min_tokens) {
  constexpr int DP = 64 * NM, PK = DP + 8, PV = ET + 8, NT = ET / 8, NO = NT / 2;
  constexpr int MT = NM == 4 ? 2 : 1, SN = NM == 1 ? NT / 2 : NT;
  extern __shared__ __align__(16) unsigned char ds_raw[];
  __nv_bfloat16* Ks0 = reinterpret_cast<__nv_bfloat16*>(ds_raw);       // [2][64][PK]
  __nv_bfloat16* Vs0 = Ks0 + 2 * DS_C * PK;                            // [2][64][PV]
  __nv_bfloat16* Sl = Vs0 + 2 * DS_C * PV;                             // [DP][PV]: the low parts of S, then of the weighted values
  __nv_bfloat16* Sh = Sl + (LOCAL ? DS_C : DP) * PV;                   // [DP][PV]
  __nv_bfloat16* Qs = Sh + (LOCAL ? 0 : DP) * PV;                      // [64][PK]
  // a chunk's gates, two buffers: log2 of the cumulated decay in two parts, weights, weights decayed to the end of their 16
  // tokens, weights decayed to the chunk's end (64 of each), log2 of the chunk's decay
  constexpr int GB = 5 * DS_C + 4;
  float* s_gate = reinterpret_cast<float*>(Qs + (LOCAL ? 0 : DS_C) * PK);
  float* s_rs = s_gate + 2 * GB;                                       // [64] row sums of the weighted scores
  float* s_n = s_rs + DS_C;                                            // [DP] the normaliser
  const int D = sh.D, E = sh.E, H = sh.H;
  const int h = blockIdx.y, e0 = blockIdx.z * ET;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  const int tw = warp & 3, o_tile = (warp >> 2) * NO;                 // token tile and first column tile of the outputs
  const int s_tile = NM == 1 ? (warp >> 2) * SN : 0;                   // first column tile of S
  auto s_chan = [&](int u) { return (NM == 1 ? tw : 8 * u + warp) * 16; };   // first channel of S tile u
  int t0, t1;
  float *S, *N = nullptr;
  const bool norms = n_state != nullptr && blockIdx.z == 0;
  if (mode == DS_DIRECT) {
    const int r = blockIdx.x;
    t0 = req_start[r];
    t1 = req_start[r + 1];
    if (t1 - t0 < min_tokens || t1 <= t0) return;
    const size_t own = (size_t)req_slot[r] * H + h;
    S = state + own * D * E;
    if (norms) N = n_state + own * D;
  } else {
    if ((int)blockIdx.x >= n_seg[0]) return;
    const int4 sg = seg[blockIdx.x];
    t0 = sg.x;
    t1 = sg.y;
    const size_t own = (size_t)blockIdx.x * H + h;
    S = seg_state + own * D * E;
    if (norms) N = seg_n + own * D;
  }
  const int g = h / (H / sh.G);
  const int kd = (D + 15) / 16;
  const int dc = D / 8, ec = min(ET, E - e0) / 8;                      // 16-byte pieces a row

  // what no copy ever writes (channels past D, columns past E, rows past a last chunk's end) is read as zeros
  for (int i = tid; i < (2 * DS_C * (PK + PV)) / 8; i += DS_CHUNK_THREADS) reinterpret_cast<uint4*>(Ks0)[i] = make_uint4(0, 0, 0, 0);
  if (!LOCAL)
    for (int i = tid; i < DS_C * PK / 8; i += DS_CHUNK_THREADS) reinterpret_cast<uint4*>(Qs)[i] = make_uint4(0, 0, 0, 0);
  for (int i = tid; i < DP; i += DS_CHUNK_THREADS) s_n[i] = (norms && !LOCAL && i < D) ? N[i] : 0.f;

  float s[MT][SN][4];
#pragma unroll
  for (int u = 0; u < MT; ++u)
#pragma unroll
    for (int n = 0; n < SN; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int d = s_chan(u) + g8 + 8 * half, e = e0 + (s_tile + n) * 8 + 2 * t4;
        float2 x = make_float2(0.f, 0.f);
        if (!LOCAL && d < D && e < E) x = *reinterpret_cast<const float2*>(S + (size_t)d * E + e);
        s[u][n][2 * half] = x.x;
        s[u][n][2 * half + 1] = x.y;
      }
  __syncthreads();

  // rows of q, k (KEYS) or v of the chunk at c0 by asynchronous copies of 16 bytes; a thread keeps its column
  auto copy = [&](auto keys, __nv_bfloat16* dst, const __nv_bfloat16* src, int pieces, int c0) {
    constexpr bool KEYS = decltype(keys)::value;
    constexpr int SLOTS = KEYS ? DP / 8 : ET / 8, pitch = KEYS ? PK : PV;
    const int c = tid % SLOTS, nt = min(DS_C, t1 - c0);
    if (c < pieces) {
#pragma unroll
      for (int tt = tid / SLOTS; tt < DS_C; tt += DS_CHUNK_THREADS / SLOTS) {
        if (tt < nt) {
          const uint32_t to = (uint32_t)__cvta_generic_to_shared(dst + tt * pitch + c * 8);
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(to), "l"(src + (size_t)(c0 + tt) * sh.stride + c * 8) : "memory");
        }
      }
    }
  };
  constexpr DsTrue of_keys{};
  constexpr DsFalse of_values{};
  const __nv_bfloat16* k_src = k + (size_t)g * D;
  const __nv_bfloat16* q_src = q + (size_t)g * D;
  const __nv_bfloat16* v_src = v + (size_t)h * E + e0;
  copy(of_keys, Ks0, k_src, dc, t0);
  copy(of_values, Vs0, v_src, ec, t0);
  if (!LOCAL) copy(of_keys, Qs, q_src, dc, t0);
  asm volatile("cp.async.commit_group;\n" ::: "memory");

  double seg_total = 0.0;                 // warp 0: log2 of the segment's decay so far
  // warp 0, two tokens a lane: the gates of the chunk at c0, cumulated over the chunk
  auto gates_of = [&](int c0, float* s_hi) {
    const int nt = min(DS_C, t1 - c0);
    float *s_lo = s_hi + DS_C, *s_w = s_lo + DS_C, *s_wl = s_w + DS_C, *s_wt = s_wl + DS_C;
    float la[2] = {0.f, 0.f}, w[2] = {0.f, 0.f};
#pragma unroll
    for (int u = 0; u < 2; ++u)
      if (2 * lane + u < nt) {
        ds_log_gate(gates, c0 + 2 * lane + u, h, H, la[u], w[u]);
        la[u] = fmaxf(la[u], DS_LOG_FLOOR);
      }
    const double LOG2E = 1.4426950408889634;
    const double x0 = (double)la[0] * LOG2E, x1 = x0 + (double)la[1] * LOG2E;
    double sum = x1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double p = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += p;
    }
    const double total = __shfl_sync(0xffffffffu, sum, 31);
    const double tile_end = __shfl_sync(0xffffffffu, sum, lane | 7);   // eight lanes hold 16 tokens
    const double before = sum - x1;
    const double L[2] = {before + x0, sum};
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = 2 * lane + u;
      s_hi[i] = (float)L[u];
      s_lo[i] = (float)(L[u] - (double)(float)L[u]);
      s_w[i] = w[u];
      s_wl[i] = ds_exp2((float)(tile_end - L[u])) * w[u];
      s_wt[i] = ds_exp2((float)(total - L[u])) * w[u];
    }
    if (lane == 0) s_wt[DS_C] = (float)total;
    seg_total += total;
  };
  if (warp == 0) gates_of(t0, s_gate);
  int buf = 0;
  for (int c0 = t0; c0 < t1; c0 += DS_C, buf ^= 1) {
    const int nt = min(DS_C, t1 - c0);
    const bool more = c0 + DS_C < t1;
    __nv_bfloat16* Ks = Ks0 + buf * DS_C * PK;
    __nv_bfloat16* Vs = Vs0 + buf * DS_C * PV;
    const float *s_hi = s_gate + buf * GB, *s_lo = s_hi + DS_C, *s_w = s_lo + DS_C, *s_wl = s_w + DS_C, *s_wt = s_wl + DS_C;
    if (!LOCAL) {
      // S as it stands before the chunk, in two parts
#pragma unroll
      for (int u = 0; u < MT; ++u)
#pragma unroll
        for (int n = 0; n < SN; ++n)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            uint32_t hi, lo;
            ds_split(s[u][n][2 * half], s[u][n][2 * half + 1], hi, lo);
            const int at = (s_chan(u) + g8 + 8 * half) * PV + (s_tile + n) * 8 + 2 * t4;
            *reinterpret_cast<uint32_t*>(Sh + at) = hi;
            *reinterpret_cast<uint32_t*>(Sl + at) = lo;
          }
    }
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();
    if (more) {
      copy(of_keys, Ks0 + (buf ^ 1) * DS_C * PK, k_src, dc, c0 + DS_C);
      copy(of_values, Vs0 + (buf ^ 1) * DS_C * PV, v_src, ec, c0 + DS_C);
      asm volatile("cp.async.commit_group;\n" ::: "memory");
      if (warp == 0) gates_of(c0 + DS_C, s_gate + (buf ^ 1) * GB);     // its tokens have the fewest keys in this chunk
    }
    if (!LOCAL) {
      const int ra = tw * 16 + g8, rb = ra + 8;                      // this thread's two tokens
      const float hi_a = s_hi[ra], hi_b = s_hi[rb], lo_a = s_lo[ra], lo_b = s_lo[rb];
      float o[NO][4];
#pragma unroll
      for (int n = 0; n < NO; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
      for (int kk = 0; kk < kd; ++kk) {
        uint32_t a[4];
        ds_ldsm(a, Qs + (tw * 16 + lane % 16) * PK + kk * 16 + (lane / 16) * 8);
#pragma unroll
        for (int n = 0; n < NO; n += 2) {
          uint32_t b[4];
          const int at = (kk * 16 + lane % 16) * PV + (o_tile + n) * 8 + (lane / 16) * 8;
          ds_ldsm_t(b, Sh + at);
          ds_mma(o[n], a, b[0], b[1]);
          ds_mma(o[n + 1], a, b[2], b[3]);
          ds_ldsm_t(b, Sl + at);
          ds_mma(o[n], a, b[0], b[1]);
          ds_mma(o[n + 1], a, b[2], b[3]);
        }
      }
      const float el_a = ds_exp2(hi_a + lo_a), el_b = ds_exp2(hi_b + lo_b);
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        o[n][0] *= el_a; o[n][1] *= el_a;
        o[n][2] *= el_b; o[n][3] *= el_b;
      }
      float sum_a = 0.f, sum_b = 0.f;
      for (int kt = 0; kt <= tw && kt * 16 < nt; ++kt) {             // keys of 16 tokens a turn, none after the rows'
        float p[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        for (int kk = 0; kk < kd; ++kk) {
          uint32_t a[4], b[4];
          ds_ldsm(a, Qs + (tw * 16 + lane % 16) * PK + kk * 16 + (lane / 16) * 8);
          ds_ldsm(b, Ks + (kt * 16 + (lane / 16) * 8 + lane % 8) * PK + kk * 16 + ((lane / 8) % 2) * 8);
          ds_mma(p[0], a, b[0], b[1]);
          ds_mma(p[1], a, b[2], b[3]);
        }
        if (kt < tw) {
          // all of these keys come before all of the warp's tokens: decays to the keys' last token, then on to the tokens
          const float he = s_hi[kt * 16 + 15], le = s_lo[kt * 16 + 15];
          const float f_a = ds_exp2((hi_a - he) + (lo_a - le)), f_b = ds_exp2((hi_b - he) + (lo_b - le));
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const float2 w = *reinterpret_cast<const float2*>(s_wl + kt * 16 + n * 8 + 2 * t4);
            p[n][0] *= f_a * w.x; p[n][1] *= f_a * w.y;
            p[n][2] *= f_b * w.x; p[n][3] *= f_b * w.y;
          }
        } else {
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int c = 0; c < 2; ++c) {
              const int j = kt * 16 + n * 8 + 2 * t4 + c;
              const float hj = s_hi[j], lj = s_lo[j], wj = s_w[j];
              p[n][c] = j <= ra ? p[n][c] * (ds_exp2((hi_a - hj) + (lo_a - lj)) * wj) : 0.f;
              p[n][2 + c] = j <= rb ? p[n][2 + c] * (ds_exp2((hi_b - hj) + (lo_b - lj)) * wj) : 0.f;
            }
        }
        if (norms) {
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            sum_a += p[n][0] + p[n][1];
            sum_b += p[n][2] + p[n][3];
          }
        }
        uint32_t ph[4], pl[4];
        ds_split(p[0][0], p[0][1], ph[0], pl[0]);
        ds_split(p[0][2], p[0][3], ph[1], pl[1]);
        ds_split(p[1][0], p[1][1], ph[2], pl[2]);
        ds_split(p[1][2], p[1][3], ph[3], pl[3]);
#pragma unroll
        for (int n = 0; n < NO; n += 2) {
          uint32_t b[4];
          ds_ldsm_t(b, Vs + (kt * 16 + lane % 16) * PV + (o_tile + n) * 8 + (lane / 16) * 8);
          ds_mma(o[n], ph, b[0], b[1]);
          ds_mma(o[n + 1], ph, b[2], b[3]);
          ds_mma(o[n], pl, b[0], b[1]);
          ds_mma(o[n + 1], pl, b[2], b[3]);
        }
      }
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        const int e = e0 + (o_tile + n) * 8 + 2 * t4;
        if (e < E) {
          if (ra < nt) *reinterpret_cast<float2*>(out + ((size_t)(c0 + ra) * H + h) * E + e) = make_float2(o[n][0] * q_scale, o[n][1] * q_scale);
          if (rb < nt) *reinterpret_cast<float2*>(out + ((size_t)(c0 + rb) * H + h) * E + e) = make_float2(o[n][2] * q_scale, o[n][3] * q_scale);
        }
      }
      if (norms && warp < 4) {
        // n . q = the row sum of the weighted scores + the decayed old n . q: two threads a token
        sum_a += __shfl_xor_sync(0xffffffffu, sum_a, 1);
        sum_a += __shfl_xor_sync(0xffffffffu, sum_a, 2);
        sum_b += __shfl_xor_sync(0xffffffffu, sum_b, 1);
        sum_b += __shfl_xor_sync(0xffffffffu, sum_b, 2);
        if (t4 == 0) { s_rs[ra] = sum_a; s_rs[rb] = sum_b; }
        __syncwarp();
        const int row = tid >> 1;                                      // a row of this warp's sixteen
        float dot = 0.f;
        for (int d = tid & 1; d < D; d += 2) dot = fmaf(s_n[d], __bfloat162float(Qs[row * PK + d]), dot);
        dot += __shfl_xor_sync(0xffffffffu, dot, 1);
        if ((tid & 1) == 0 && row < nt) {
          const size_t at = (size_t)(c0 + row) * H + h;
          const float nq = (s_rs[row] + ds_exp2(s_hi[row] + s_lo[row]) * dot) * q_scale;
          den[at] = fmaxf(fabsf(nq), floor_in[at]) + DS_DEN_EPS;
        }
      }
      __syncthreads();                    // Q, the unweighted values, the parts of S and n have been read
      if (more) {
        copy(of_keys, Qs, q_src, dc, c0 + DS_C);
        asm volatile("cp.async.commit_group;\n" ::: "memory");
      }
    }
    // values weighted to the chunk's end, in two parts
    for (int i = tid; i < DS_C * ET / 2; i += DS_CHUNK_THREADS) {
      const int tt = i / (ET / 2), c = (i % (ET / 2)) * 2;
      const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(Vs + tt * PV + c);
      const float w = s_wt[tt];
      uint32_t hi, lo;
      ds_split(__low2float(x) * w, __high2float(x) * w, hi, lo);
      *reinterpret_cast<uint32_t*>(Vs + tt * PV + c) = hi;
      *reinterpret_cast<uint32_t*>(Sl + tt * PV + c) = lo;
    }
    const float keep = ds_exp2(s_wt[DS_C]);
    if (norms) {
      for (int d = tid; d < D; d += DS_CHUNK_THREADS) {
        float x = s_n[d] * keep;
        for (int tt = 0; tt < nt; ++tt) x = fmaf(s_wt[tt], __bfloat162float(Ks[tt * PK + d]), x);
        s_n[d] = x;
      }
    }
    __syncthreads();
#pragma unroll
    for (int u = 0; u < MT; ++u)
#pragma unroll
      for (int n = 0; n < SN; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) s[u][n][c] *= keep;
#pragma unroll
    for (int kt = 0; kt < DS_C / 16; ++kt) {
      if (kt * 16 < nt) {
        uint32_t a[MT][4];
#pragma unroll
        for (int u = 0; u < MT; ++u)
          ds_ldsm_t(a[u], Ks + (kt * 16 + (lane / 16) * 8 + lane % 8) * PK + s_chan(u) + ((lane / 8) % 2) * 8);
#pragma unroll
        for (int n = 0; n < SN; n += 2) {
          uint32_t bh[4], bl[4];
          const int at = (kt * 16 + lane % 16) * PV + (s_tile + n) * 8 + (lane / 16) * 8;
          ds_ldsm_t(bh, Vs + at);
          ds_ldsm_t(bl, Sl + at);
#pragma unroll
          for (int u = 0; u < MT; ++u) {
            if (s_chan(u) < D) {
              ds_mma(s[u][n], a[u], bh[0], bh[1]);
              ds_mma(s[u][n + 1], a[u], bh[2], bh[3]);
              ds_mma(s[u][n], a[u], bl[0], bl[1]);
              ds_mma(s[u][n + 1], a[u], bl[2], bl[3]);
            }
          }
        }
      }
    }
    __syncthreads();                      // the chunk's keys and values have been read; their buffer may be filled again
  }
  if (mode != DS_REPLAY) {
#pragma unroll
    for (int u = 0; u < MT; ++u)
#pragma unroll
      for (int n = 0; n < SN; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int d = s_chan(u) + g8 + 8 * half, e = e0 + (s_tile + n) * 8 + 2 * t4;
          if (d < D && e < E) *reinterpret_cast<float2*>(S + (size_t)d * E + e) = make_float2(s[u][n][2 * half], s[u][n][2 * half + 1]);
        }
    if (norms)
      for (int d = tid; d < D; d += DS_CHUNK_THREADS) N[d] = s_n[d];
  }
  if (LOCAL && tid == 0 && blockIdx.z == 0) seg_log[(size_t)blockIdx.x * H + h] = (float)seg_total;
}

// which sizes the chunk form takes (bfloat16 rows of 16-byte pieces)
extern "C" int qb_decay_chunks_supported(int D, int E) { return D > 0 && E > 0 && D <= 256 && D % 8 == 0 && E % 8 == 0 ? 1 : 0; }

static int ds_tile_cols(int D, int E) { return D > 128 || E <= 32 ? 32 : 64; }

// tokens a segment (a multiple of the chunk; 0: the step runs as one pass) for a step of T tokens in R requests
static int ds_segment_tokens(int T, int R, int H, int D, int E) {
  const int et = ds_tile_cols(D, E);
  const long blocks = (long)H * ((E + et - 1) / et);
  const long want = 2l * 148;                       // two blocks an SM
  if (R > 1024 || T < 512 || (long)T < 256l * R || blocks * R >= want * 3 / 4) return 0;
  long seg = (long)T * blocks / want;
  seg = (seg + DS_C - 1) / DS_C * DS_C;
  return (int)(seg < 2 * DS_C ? 2 * DS_C : seg);
}

// floats of scratch of the three-pass form (0: one pass)
extern "C" long long qb_decay_chunks_scratch(int T, int R, int H, int D, int E, int norms) {
  const int len = ds_segment_tokens(T, R, H, D, E);
  if (len == 0) return 0;
  const long long max_seg = T / len + R;
  return 4 * max_seg + ((2ll * R + 3) & ~3ll) + 4 + ((max_seg * H + 3) & ~3ll) + max_seg * H * D * (long long)E +
         (norms ? max_seg * H * D : 0);
}

// As qb_decay_chain with bfloat16 rows, for the requests that bring at least min_tokens tokens.  scratch:
// qb_decay_chunks_scratch floats, 16-byte aligned, or null (one pass).
extern "C" int qb_decay_chunks(const void* q, const void* k, const void* v, long long stride, int kind, const float* decay,
                               const float* log_decay, const float* step, int step_stride, const float* step_bias,
                               const float* A_log, const float* weight, float* state, float* n_state,
                               const float* floor_in, float* den, float* out, float* scratch, const int* req_start,
                               const int* req_slot, int T, int R, int H, int G, int D, int E, float q_scale,
                               int min_tokens, cudaStream_t stream) {
  if (T <= 0 || R <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || kind < 0 || kind > 2) return QB_ERR_BAD_ARG;
  if (!qb_decay_chunks_supported(D, E) || H > 65535 || stride % 8 ||
      (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)scratch) & 15) || (((uintptr_t)state | (uintptr_t)out) & 7))
    return QB_ERR_UNSUPPORTED;
  const int et = ds_tile_cols(D, E);
  const int nm = D <= 64 ? 1 : D <= 128 ? 2 : 4;
  const int zt = (E + et - 1) / et;
  const int seg_len = scratch != nullptr ? ds_segment_tokens(T, R, H, D, E) : 0;
  const int max_seg = seg_len ? T / seg_len + R : 0;
  int4* seg = reinterpret_cast<int4*>(scratch);
  int2* req_seg = seg_len ? reinterpret_cast<int2*>(seg + max_seg) : nullptr;
  int* n_seg = seg_len ? reinterpret_cast<int*>(scratch + 4 * (size_t)max_seg + ((2 * (size_t)R + 3) & ~(size_t)3)) : nullptr;
  float* seg_log = seg_len ? reinterpret_cast<float*>(n_seg + 4) : nullptr;
  float* seg_state = seg_len ? seg_log + (((size_t)max_seg * H + 3) & ~(size_t)3) : nullptr;
  float* seg_n = seg_len && n_state != nullptr ? seg_state + (size_t)max_seg * H * D * E : nullptr;
  const DsShape sh{H, G, D, E, stride};
  const DsGates gates{kind, decay, log_decay, step, step_stride, step_bias, A_log, weight};
#define DS_CHUNK(NM, ET, LOCAL_, MODE_, GX)                                                                              \
  do {                                                                                                                  \
    constexpr int DP = 64 * NM, PK = DP + 8, PV = ET + 8;                                                                \
    const size_t smem = (size_t)(2 * DS_C * (PK + PV) + (LOCAL_ ? DS_C * PV : 2 * DP * PV + DS_C * PK)) * 2 +            \
                        (size_t)(2 * (5 * DS_C + 4) + DS_C + DP) * sizeof(float);                                                     \
    auto kern = ds_chunk_kernel<NM, ET, LOCAL_>;                                                                         \
    if (smem > 48 * 1024) {                                                                                             \
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                \
      if (e != cudaSuccess) return (int)e;                                                                               \
    }                                                                                                                    \
    kern<<<dim3(GX, H, zt), DS_CHUNK_THREADS, smem, stream>>>((const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, \
        sh, gates, state, n_state, floor_in, den, out, req_start, req_slot, seg, n_seg, seg_state, seg_n, seg_log, MODE_, \
        q_scale, min_tokens);                                                                                            \
  } while (0)
#define DS_CHUNK_SIZES(LOCAL_, MODE_, GX)                                  \
  do {                                                                     \
    if (nm == 4) DS_CHUNK(4, 32, LOCAL_, MODE_, GX);                       \
    else if (nm == 2 && et == 64) DS_CHUNK(2, 64, LOCAL_, MODE_, GX);      \
    else if (nm == 2) DS_CHUNK(2, 32, LOCAL_, MODE_, GX);                  \
    else if (et == 64) DS_CHUNK(1, 64, LOCAL_, MODE_, GX);                 \
    else DS_CHUNK(1, 32, LOCAL_, MODE_, GX);                               \
  } while (0)
  if (!seg_len) {
    DS_CHUNK_SIZES(false, DS_DIRECT, R);
  } else {
    ds_segments_kernel<<<1, 1024, 0, stream>>>(req_start, R, seg_len, min_tokens, max_seg, seg, req_seg, n_seg);
    DS_CHUNK_SIZES(true, DS_LOCAL, max_seg);
    int z = (D * E + 255) / 256;
    while ((long)R * H * z > 4096 && z > 1) z = (z + 1) / 2;
    ds_combine_kernel<<<dim3(R, H, z), 256, 0, stream>>>(state, n_state, seg_state, seg_n, seg_log, req_seg, req_slot, H, D, E);
    DS_CHUNK_SIZES(false, DS_REPLAY, max_seg);
  }
#undef DS_CHUNK_SIZES
#undef DS_CHUNK
  QB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------------------------
// float32 columns of wider rows -> contiguous rows of the activation dtype, through silu or as they are
// ---------------------------------------------------------------------------------------------
template <typename O>
__global__ void rows_act_kernel(const float* __restrict__ x, long long stride, O* __restrict__ out, int T, int n, int silu,
                                int vec) {
  if (vec) {
    const int n8 = n / 8;
    const size_t total = (size_t)T * n8;
    for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
      const size_t t = i / n8;
      const int c = (int)(i % n8) * 8;
      float v[8];
      QbVec8<float>::load(x + t * stride + c, v);
      if (silu) {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = v[e] / (1.f + expf(-v[e]));
      }
      QbVec8<O>::store(out + t * n + c, v);
    }
    return;
  }
  const size_t total = (size_t)T * n;
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const float v = x[i / n * stride + i % n];
    out[i] = qb_from_float<O>(silu ? v / (1.f + expf(-v)) : v);
  }
}

extern "C" int qb_rows_act(const float* x, long long stride, void* out, int out_dtype, int T, int n, int silu,
                           cudaStream_t stream) {
  if (T <= 0 || n <= 0) return 0;
  const int vec = n % 8 == 0 && stride % 4 == 0 && (((uintptr_t)x | (uintptr_t)out) & 15) == 0;
  const size_t items = (size_t)T * n / (vec ? 8 : 1);
  const int blocks = (int)((items + 255) / 256 < 8192 ? (items + 255) / 256 : 8192);
  QB_DISPATCH_DTYPE(out_dtype, O, rows_act_kernel<O><<<blocks, 256, 0, stream>>>(x, stride, (O*)out, T, n, silu, vec));
  QB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------------------------
// From the recurrence's results to what the output projection reads, per token:
//   y = o[t, h, :] / den[t, h]  + skip[h] * x[t, h, :]          (den, skip optional)
//   y <- y * silu(gate)                                          (gate_first: the gate before the norm)
//   y <- y / rms over each of `parts` equal parts of the row (eps inside the root) * gain
//   y <- y * sigmoid(gate)                                       (else)
// A group of threads a (token, part): a warp for parts of up to 512 numbers, a block for longer ones.  Parts that move in
// 16-byte pieces and fit (Q pieces a thread) are held in registers, with all loads asked for before the first sum; other
// parts stay in shared memory between the two passes.  Sums in an order that depends on the sizes alone.
// ---------------------------------------------------------------------------------------------
template <typename O, int WARPS, int Q>       // WARPS a part: 1 (four parts a block) or 8; Q 0: shared memory, any sizes
__global__ void __launch_bounds__(WARPS == 1 ? 128 : 256)
decay_out_kernel(const float* __restrict__ o, const float* __restrict__ den, const O* __restrict__ x, long long x_stride,
                 const float* __restrict__ skip, const float* __restrict__ gate, long long gate_stride,
                 const float* __restrict__ gain, O* __restrict__ out, int T, int H, int E, int parts, float eps,
                 int gate_first) {
  extern __shared__ __align__(16) float s_part[];
  __shared__ float s_sum[32];
  const int HE = H * E, n = HE / parts;
  const int group = WARPS == 1 ? threadIdx.x >> 5 : 0, nth = WARPS * 32, me = WARPS == 1 ? threadIdx.x & 31 : threadIdx.x;
  const long long unit = (long long)blockIdx.x * (WARPS == 1 ? 4 : 1) + group;
  if (unit >= (long long)T * parts) return;           // a whole warp (or block) leaves
  const int t = (int)(unit / parts), c0 = (int)(unit % parts) * n;
  const float* orow = o + (size_t)t * HE + c0;
  const float* grow = gate + (size_t)t * gate_stride + c0;
  const float* nrow = gain + c0;
  const O* xrow = skip != nullptr ? x + (size_t)t * x_stride + c0 : nullptr;
  O* to = out + (size_t)t * HE + c0;
  auto root = [&](float ss) {
    if (WARPS == 1) {
      ss = qb_warp_sum(ss);
      __syncwarp();
    } else {
      ss = qb_block_sum(ss, s_sum);
    }
    return 1.f / sqrtf(ss / (float)n + eps);
  };
  if constexpr (Q > 0) {
    float4 y[Q], gv[Q], gn[Q];
    float dn[Q], sk[Q], xv[Q][4];
    struct alignas(4 * sizeof(O)) Four { O v[4]; };
#pragma unroll
    for (int u = 0; u < Q; ++u) {
      const int i = (me + u * nth) * 4;
      dn[u] = 1.f;
      sk[u] = 0.f;
      if (i < n) {
        const int h = (c0 + i) / E;                   // four numbers of one head
        y[u] = *reinterpret_cast<const float4*>(orow + i);
        gv[u] = *reinterpret_cast<const float4*>(grow + i);
        gn[u] = *reinterpret_cast<const float4*>(nrow + i);
        if (den != nullptr) dn[u] = den[(size_t)t * H + h];
        if (skip != nullptr) {
          sk[u] = skip[h];
          const Four f = *reinterpret_cast<const Four*>(xrow + i);
#pragma unroll
          for (int e = 0; e < 4; ++e) xv[u][e] = qb_to_float<O>(f.v[e]);
        }
      } else {
        y[u] = gv[u] = gn[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < Q; ++u) {
      float* yv = &y[u].x;
      float* g = &gv[u].x;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (den != nullptr) yv[e] /= dn[u];
        if (skip != nullptr && (me + u * nth) * 4 < n) yv[e] = fmaf(sk[u], xv[u][e], yv[e]);
        const float sg = 1.f / (1.f + expf(-g[e]));
        if (gate_first) yv[e] *= g[e] * sg;           // silu before the norm
        g[e] = gate_first ? 1.f : sg;                 // what multiplies the normed number
        ss += yv[e] * yv[e];
      }
    }
    const float inv = root(ss);
#pragma unroll
    for (int u = 0; u < Q; ++u) {
      const int i = (me + u * nth) * 4;
      if (i < n) {
        Four four;
#pragma unroll
        for (int e = 0; e < 4; ++e) four.v[e] = qb_from_float<O>((&y[u].x)[e] * inv * (&gn[u].x)[e] * (&gv[u].x)[e]);
        *reinterpret_cast<Four*>(to + i) = four;
      }
    }
  } else {
    float* buf = s_part + group * n;
    float ss = 0.f;
    for (int i = me; i < n; i += nth) {
      const int h = (c0 + i) / E;
      float y = orow[i];
      if (den != nullptr) y = y / den[(size_t)t * H + h];
      if (skip != nullptr) y = fmaf(skip[h], qb_to_float<O>(xrow[i]), y);
      if (gate_first) y *= grow[i] / (1.f + expf(-grow[i]));
      ss += y * y;
      buf[i] = y;
    }
    const float inv = root(ss);
    for (int i = me; i < n; i += nth) {               // every thread finishes the numbers it put there
      float r = buf[i] * inv * nrow[i];
      if (!gate_first) r *= 1.f / (1.f + expf(-grow[i]));
      to[i] = qb_from_float<O>(r);
    }
  }
}

// o float32 [T, H, E]; den float32 [T, H] or null; x (rows of x_stride elements of out_dtype) with skip float32 [H], or
// both null; gate: float32 rows of gate_stride; gain float32 [H * E]; out [T, H * E].
extern "C" int qb_decay_out(const float* o, const float* den, const void* x, long long x_stride, const float* skip,
                            const float* gate, long long gate_stride, const float* gain, void* out, int out_dtype, int T,
                            int H, int E, int parts, float eps, int gate_first, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || E <= 0 || parts <= 0 || ((long long)H * E) % parts || (skip != nullptr) != (x != nullptr)) return QB_ERR_BAD_ARG;
  const int n = H * E / parts;
  const bool warp_form = n <= 512;
  const bool vec = n % 4 == 0 && E % 4 == 0 && gate_stride % 4 == 0 && x_stride % 4 == 0 && n <= 8192 &&
                   (((uintptr_t)o | (uintptr_t)gate | (uintptr_t)gain | (uintptr_t)out | (uintptr_t)x) & 15) == 0;
  const int pieces = (n / 4 + (warp_form ? 32 : 256) - 1) / (warp_form ? 32 : 256);
  const size_t smem = vec ? 0 : (size_t)n * (warp_form ? 4 : 1) * sizeof(float);
  if (smem > 200 * 1024) return QB_ERR_UNSUPPORTED;
  const long long units = (long long)T * parts, blocks = warp_form ? (units + 3) / 4 : units;
  if (blocks > 0x7fffffffll) return QB_ERR_UNSUPPORTED;
#define DS_OUT(WARPS, Q)                                                                                              \
  do {                                                                                                               \
    auto kern = decay_out_kernel<O, WARPS, Q>;                                                                        \
    if (smem > 48 * 1024) {                                                                                           \
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);              \
      if (e != cudaSuccess) return (int)e;                                                                            \
    }                                                                                                                 \
    kern<<<(unsigned)blocks, WARPS == 1 ? 128 : 256, smem, stream>>>(o, den, (const O*)x, x_stride, skip, gate,        \
                                                                     gate_stride, gain, (O*)out, T, H, E, parts, eps, \
                                                                     gate_first);                                     \
  } while (0)
  QB_DISPATCH_DTYPE(out_dtype, O, {
    if (!vec && warp_form) DS_OUT(1, 0);
    else if (!vec) DS_OUT(8, 0);
    else if (warp_form && pieces <= 1) DS_OUT(1, 1);
    else if (warp_form && pieces <= 2) DS_OUT(1, 2);
    else if (warp_form) DS_OUT(1, 4);
    else if (pieces <= 2) DS_OUT(8, 2);
    else if (pieces <= 4) DS_OUT(8, 4);
    else DS_OUT(8, 8);
  });
#undef DS_OUT
  QB_LAUNCH_CHECK();
  return 0;
}
