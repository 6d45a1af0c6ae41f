// Matrix memories with a decay per key channel over a flat batch of segments: the gated delta rule and gated linear
// attention.
//
// Per head a float matrix S [dk, dv], zero for a fresh request, kept in the request's state slot between steps:
//
//   S <- diag(a_t) S;   w = beta_t (v_t - S^T k_t)  (delta form)  or  v_t  (linear form);   S <- S + k_t w^T;   o_t = S^T q_t
//
//   delta   q and k unit vectors per head, x / sqrt(sum(x^2) + unit_eps); a_t = exp(rate[h] * softplus(z_t + bias)) per
//           head and channel (rate = -exp(A_log)); beta = sigmoid of a logit per head
//   linear  q and k as they are; a_t = sigmoid(z_t + bias)^sharp
//   both    q times q_scale; head h reads q/k head h / (H / G); z float rows of their own
//
// q, k and v are columns of the rows `u` in the compute dtype; lengths, decays, betas, state, sums and outputs are float.
// Three ways to run it, picked per launch by the host:
//
//   step    every segment is one token (decode): one pass over the state.
//   walk    token by token, S in registers; any size.
//   chunks  long portions, 16 tokens at a time.  With G_t the log decays summed from the chunk's start up to t (per
//           channel), and of tokens i, j of a chunk A_ij = sum_r k_i k_j e^(G_i - G_j), B_ij = sum_r q_i k_j e^(G_i - G_j),
//             w_i = beta_i (v_i - (k_i e^(G_i))^T S - sum_(j<i) A_ij w_j),   o_i = (q_i e^(G_i))^T S + sum_(j<=i) B_ij w_j
//             S <- e^(G_16) S + sum_j (k_j e^(G_16 - G_j)) w_j^T
//           Everything but the products with S can be worked out for all chunks at once: `prepare` leaves, per chunk and
//           head, the weighted q, k and the solved system; `scan` then takes S through the chunks in order, 16 columns a
//           block.  G is summed in double and kept as two floats, so that G_i - G_j is exact to float however strong a
//           decay lies before it.  Where G stays small A and B are products of rows weighted by e^G and e^(-G); where it
//           does not, every pair is weighted on its own, and no exponent is positive.
#include "common.cuh"

struct MemoryIn {
  const void* u;                 // compute dtype, row pitch u_ld
  long long u_ld;
  int q_off, k_off, v_off;
  const float* z;                // row pitch z_ld
  long long z_ld;
  const float* bias;             // [H*dk]
  const float* rate;             // delta form: [H]
  const void* beta;              // delta form: compute dtype, row pitch b_ld
  long long b_ld;
  float sharp;                   // linear form
  float q_scale, unit_eps;
  int H, G, dk, dv;
};

// log(1 + e^z)
__device__ __forceinline__ float cm_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// the logarithm of a decay
template <bool DELTA>
__device__ __forceinline__ float cm_log_decay(float z, float rate, float sharp) {
  return DELTA ? rate * cm_softplus(z) : -sharp * cm_softplus(-z);
}
__device__ __forceinline__ float cm_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// ---------------------------------------------------------------------------------------------
// The walk.  A block serves one (segment, head, slice of columns of S).  Eight neighbouring threads share a group of one or
// four columns, each holding an eighth of its rows in registers over the whole segment; up to CM_TOKENS tokens' q, k, decays
// and v come into shared memory at a time.
#define CM_TOKENS 16
#define CM_TPC 8               // threads per column group
#define CM_GROUPS 32           // column groups per block
#define CM_THREADS (CM_TPC * CM_GROUPS)

template <bool DELTA, typename T, int DKR, int CPT>
__global__ void __launch_bounds__(CM_THREADS)
channel_walk_kernel(const MemoryIn in, const int* __restrict__ cu_seqlens, const int* __restrict__ seg_start,
                  const int* __restrict__ seg_slot, float* __restrict__ state, float* __restrict__ out, int tokens) {
  pdl_begin();
  extern __shared__ __align__(16) float cm_sh[];
  constexpr int RPT = DKR / CM_TPC;                        // rows of S per thread
  constexpr int COLS = CM_GROUPS * CPT;
  const int dk = in.dk, dv = in.dv, H = in.H;
  const int dkp = (dk + 4 * CM_TPC - 1) / (4 * CM_TPC) * (4 * CM_TPC);
  float* qs = cm_sh;                                       // [tokens][dkp]
  float* ks = qs + tokens * dkp;
  float* as = ks + tokens * dkp;
  float* vs = as + tokens * dkp;                           // [tokens][COLS]
  float* bs = vs + tokens * COLS;                          // [tokens]
  const int b = blockIdx.x, h = blockIdx.y, g = h / (H / in.G);
  const int sub = threadIdx.x & (CM_TPC - 1), group = threadIdx.x / CM_TPC;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col0 = blockIdx.z * COLS, c = col0 + group * CPT;
  const int row0 = cu_seqlens[b], row1 = cu_seqlens[b + 1];
  if (row1 <= row0) return;
  float* slot = state + ((size_t)seg_slot[b] * H + h) * dk * dv;
  const bool fresh = seg_start[b] == 0;
  const bool wide = CPT == 4 && (dv & 3) == 0;             // my four columns as one 16-byte access (all or none exist)

  // registers [i*4 + e][j] hold row 4 CM_TPC i + 4 sub + e, column c + j
  float S[RPT][CPT];
#pragma unroll
  for (int i = 0; i < RPT / 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = 4 * CM_TPC * i + 4 * sub + e;
#pragma unroll
      for (int j = 0; j < CPT; ++j) S[i * 4 + e][j] = 0.f;
      if (!fresh && r < dk) {
        if (wide) {
          if (c < dv) {
            const float4 s4 = *reinterpret_cast<const float4*>(slot + (size_t)r * dv + c);
            S[i * 4 + e][0] = s4.x; S[i * 4 + e][CPT > 1 ? 1 : 0] = s4.y;
            S[i * 4 + e][CPT > 2 ? 2 : 0] = s4.z; S[i * 4 + e][CPT > 3 ? 3 : 0] = s4.w;
          }
        } else {
#pragma unroll
          for (int j = 0; j < CPT; ++j)
            if (c + j < dv) S[i * 4 + e][j] = slot[(size_t)r * dv + c + j];
        }
      }
    }
  const float rate = DELTA ? in.rate[h] : 0.f;
  const T* u = static_cast<const T*>(in.u);
  for (int t0 = row0; t0 < row1; t0 += tokens) {
    const int nt = min(tokens, row1 - t0);
    __syncthreads();                                       // everyone is done with the previous tokens
    for (int i = threadIdx.x; i < nt * dkp; i += CM_THREADS) {
      const int t = i / dkp, r = i - t * dkp;
      float qv = 0.f, kv = 0.f, av = 0.f;
      if (r < dk) {
        const T* row = u + (size_t)(t0 + t) * in.u_ld;
        qv = to_f<T>(row[in.q_off + g * dk + r]);
        kv = to_f<T>(row[in.k_off + g * dk + r]);
        av = expf(cm_log_decay<DELTA>(in.z[(size_t)(t0 + t) * in.z_ld + h * dk + r] + in.bias[h * dk + r], rate, in.sharp));
      }
      qs[i] = DELTA ? qv : qv * in.q_scale;
      ks[i] = kv;
      as[i] = av;
    }
    for (int i = threadIdx.x; i < nt * COLS; i += CM_THREADS) {
      const int t = i / COLS, d = i - t * COLS;
      vs[i] = col0 + d < dv ? to_f<T>(u[(size_t)(t0 + t) * in.u_ld + in.v_off + h * dv + col0 + d]) : 0.f;
    }
    if (DELTA && threadIdx.x < nt) {
      const float z = to_f<T>(static_cast<const T*>(in.beta)[(size_t)(t0 + threadIdx.x) * in.b_ld + h]);
      bs[threadIdx.x] = cm_sigmoid(z);
    }
    __syncthreads();
    for (int t = warp; DELTA && t < nt; t += CM_THREADS / 32) {   // unit lengths, a warp per token
      float sq = 0.f, sk = 0.f;
      for (int r = lane; r < dk; r += 32) {
        sq = fmaf(qs[t * dkp + r], qs[t * dkp + r], sq);
        sk = fmaf(ks[t * dkp + r], ks[t * dkp + r], sk);
      }
      sq = in.q_scale / sqrtf(warp_sum(sq) + in.unit_eps);
      sk = 1.f / sqrtf(warp_sum(sk) + in.unit_eps);
      for (int r = lane; r < dk; r += 32) {
        qs[t * dkp + r] *= sq;
        ks[t * dkp + r] *= sk;
      }
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float *qt = qs + t * dkp, *kt = ks + t * dkp, *at = as + t * dkp;
      float known[CPT], acc[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) known[j] = acc[j] = 0.f;
#pragma unroll
      for (int i = 0; i < RPT / 4; ++i)
        if (4 * CM_TPC * i < dk) {
          const float4 k4 = *reinterpret_cast<const float4*>(kt + 4 * CM_TPC * i + 4 * sub);
          const float4 a4 = *reinterpret_cast<const float4*>(at + 4 * CM_TPC * i + 4 * sub);
          const float kv[4] = {k4.x, k4.y, k4.z, k4.w}, av[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
          for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int j = 0; j < CPT; ++j) {
              S[i * 4 + e][j] *= av[e];
              if (DELTA) known[j] = fmaf(S[i * 4 + e][j], kv[e], known[j]);
            }
        }
#pragma unroll
      for (int w = 1; DELTA && w < CM_TPC; w <<= 1)
#pragma unroll
        for (int j = 0; j < CPT; ++j) known[j] += __shfl_xor_sync(0xffffffffu, known[j], w);
      const float beta = DELTA ? bs[t] : 1.f;
      float write[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) write[j] = DELTA ? beta * (vs[t * COLS + group * CPT + j] - known[j]) : vs[t * COLS + group * CPT + j];
#pragma unroll
      for (int i = 0; i < RPT / 4; ++i)
        if (4 * CM_TPC * i < dk) {
          const float4 k4 = *reinterpret_cast<const float4*>(kt + 4 * CM_TPC * i + 4 * sub);
          const float4 q4 = *reinterpret_cast<const float4*>(qt + 4 * CM_TPC * i + 4 * sub);
          const float kv[4] = {k4.x, k4.y, k4.z, k4.w}, qv[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
          for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int j = 0; j < CPT; ++j) {
              S[i * 4 + e][j] = fmaf(kv[e], write[j], S[i * 4 + e][j]);
              acc[j] = fmaf(S[i * 4 + e][j], qv[e], acc[j]);
            }
        }
#pragma unroll
      for (int w = 1; w < CM_TPC; w <<= 1)
#pragma unroll
        for (int j = 0; j < CPT; ++j) acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], w);
      float* orow = out + ((size_t)(t0 + t) * H + h) * dv + c;
      if (sub < CPT && c + sub < dv) {
        float mine = acc[0];
#pragma unroll
        for (int j = 1; j < CPT; ++j) mine = sub == j ? acc[j] : mine;
        orow[sub] = mine;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < RPT / 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = 4 * CM_TPC * i + 4 * sub + e;
      if (r >= dk) continue;
      if (wide) {
        if (c < dv)
          *reinterpret_cast<float4*>(slot + (size_t)r * dv + c) =
              make_float4(S[i * 4 + e][0], S[i * 4 + e][CPT > 1 ? 1 : 0], S[i * 4 + e][CPT > 2 ? 2 : 0],
                          S[i * 4 + e][CPT > 3 ? 3 : 0]);
      } else {
#pragma unroll
        for (int j = 0; j < CPT; ++j)
          if (c + j < dv) slot[(size_t)r * dv + c + j] = S[i * 4 + e][j];
      }
    }
}


// ---------------------------------------------------------------------------------------------
// The step: one token per segment.  A block serves one (segment, head, slice of up to 128 columns); neighbouring lanes hold
// four columns each of one row of S (`lpr` lanes a row, a power of two), the block's rows are taken in turns.  The state
// is asked for first; the token's q, k and decays come in meanwhile.
#define CS_WARPS 8
#define CS_THREADS (CS_WARPS * 32)

template <bool DELTA, typename T, int RPT>
__global__ void __launch_bounds__(CS_THREADS, 2)
channel_step_kernel(const MemoryIn in, const int* __restrict__ cu_seqlens, const int* __restrict__ seg_start,
                    const int* __restrict__ seg_slot, float* __restrict__ state, float* __restrict__ out, int lpr) {
  pdl_begin();
  __shared__ float qs[256], ks[256], as[256];
  __shared__ __align__(16) float part[CS_WARPS][128];
  __shared__ __align__(16) float whole[128];
  const int dk = in.dk, dv = in.dv, H = in.H;
  const int b = blockIdx.x, h = blockIdx.y, g = h / (H / in.G);
  const int row = cu_seqlens[b];
  if (cu_seqlens[b + 1] <= row) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int rows_at_once = CS_THREADS / lpr;
  const int r0 = threadIdx.x / lpr, cl = threadIdx.x % lpr;
  const int c = blockIdx.z * 128 + 4 * cl;
  const bool live = c < dv;
  float* at = state + ((size_t)seg_slot[b] * H + h) * dk * dv + c;
  const bool fresh = seg_start[b] == 0;
  float4 S[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = r0 + i * rows_at_once;
    S[i] = !fresh && live && r < dk ? *reinterpret_cast<const float4*>(at + (size_t)r * dv) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const T* u = static_cast<const T*>(in.u) + (size_t)row * in.u_ld;
  const float rate = DELTA ? in.rate[h] : 0.f;
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (live) {
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = to_f<T>(u[in.v_off + h * dv + c + e]);
  }
  const float beta = DELTA ? cm_sigmoid(to_f<T>(static_cast<const T*>(in.beta)[(size_t)row * in.b_ld + h])) : 1.f;
  if (threadIdx.x < dk) {
    const int r = threadIdx.x;
    qs[r] = to_f<T>(u[in.q_off + g * dk + r]);
    ks[r] = to_f<T>(u[in.k_off + g * dk + r]);
    as[r] = expf(cm_log_decay<DELTA>(in.z[(size_t)row * in.z_ld + h * dk + r] + in.bias[h * dk + r], rate, in.sharp));
  }
  __syncthreads();
  float sq = in.q_scale, sk = 1.f;
  if (DELTA) {                                             // every warp forms the same two lengths
    float nq = 0.f, nk = 0.f;
    for (int r = lane; r < dk; r += 32) {
      nq = fmaf(qs[r], qs[r], nq);
      nk = fmaf(ks[r], ks[r], nk);
    }
    sq = in.q_scale / sqrtf(warp_sum(nq) + in.unit_eps);
    sk = 1.f / sqrtf(warp_sum(nk) + in.unit_eps);
  }
  // sum a value per column over the block's rows: within the warp, then across the warps, in warp order
  auto over_rows = [&](float4 t) {
    for (int w = lpr; w < 32; w <<= 1) {
      t.x += __shfl_xor_sync(0xffffffffu, t.x, w);
      t.y += __shfl_xor_sync(0xffffffffu, t.y, w);
      t.z += __shfl_xor_sync(0xffffffffu, t.z, w);
      t.w += __shfl_xor_sync(0xffffffffu, t.w, w);
    }
    if (lane < lpr) *reinterpret_cast<float4*>(&part[warp][4 * lane]) = t;
    __syncthreads();
    if (threadIdx.x < 4 * lpr) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < CS_WARPS; ++w) s += part[w][threadIdx.x];
      whole[threadIdx.x] = s;
    }
    __syncthreads();
    return *reinterpret_cast<const float4*>(&whole[4 * cl]);
  };
  float4 known = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = r0 + i * rows_at_once;
    if (r < dk) {
      const float a = as[r];
      S[i].x *= a; S[i].y *= a; S[i].z *= a; S[i].w *= a;
      if (DELTA) {
        const float k = ks[r];
        known.x = fmaf(S[i].x, k, known.x); known.y = fmaf(S[i].y, k, known.y);
        known.z = fmaf(S[i].z, k, known.z); known.w = fmaf(S[i].w, k, known.w);
      }
    }
  }
  float4 w = make_float4(v[0], v[1], v[2], v[3]);
  if (DELTA) {
    known = over_rows(known);
    w = make_float4(beta * (v[0] - sk * known.x), beta * (v[1] - sk * known.y), beta * (v[2] - sk * known.z),
                    beta * (v[3] - sk * known.w));
  }
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = r0 + i * rows_at_once;
    if (r < dk) {
      const float k = DELTA ? sk * ks[r] : ks[r], q = qs[r];
      S[i].x = fmaf(k, w.x, S[i].x); S[i].y = fmaf(k, w.y, S[i].y);
      S[i].z = fmaf(k, w.z, S[i].z); S[i].w = fmaf(k, w.w, S[i].w);
      if (live) *reinterpret_cast<float4*>(at + (size_t)r * dv) = S[i];
      o.x = fmaf(S[i].x, q, o.x); o.y = fmaf(S[i].y, q, o.y);
      o.z = fmaf(S[i].z, q, o.z); o.w = fmaf(S[i].w, q, o.w);
    }
  }
  o = over_rows(o);
  if (r0 == 0 && live)
    *reinterpret_cast<float4*>(out + ((size_t)row * H + h) * dv + c) = make_float4(sq * o.x, sq * o.y, sq * o.z, sq * o.w);
}

// ---------------------------------------------------------------------------------------------
// Chunks.  With B the 16 x 16 matrix of B_ij (j <= i), w = w0 - W S and o = q S + B w = (q - B W) S + B w0: after one product
// with S, [W; q - B W] S, everything of the chunk is there.  What `prepare` leaves for one (chunk, head), DKP rows (dk
// rounded up, zeros behind) and dvp columns (dv rounded up to CC_COLS), floats:
//   A  [MR][DKP + 8]   delta: W, then q - B W, 16 tokens each; linear: the weighted q alone
//   K  [16][DKP + 4]   k_j e^(G_16 - G_j)
//   E  [DKP]           e^(G_16)
//   V  [dvp / 16][2][16][16]   per 16 columns: w0, then B w0
#define CC_Q 16                // tokens per chunk
#define CC_COLS 16             // columns of S per block of `scan`
#define CC_THREADS 256
#ifndef CC_PREPARE_BLOCKS
#define CC_PREPARE_BLOCKS 2    // of `prepare` on an SM, by its registers
#endif
#define CC_WEAK 100.f          // e^(-G) is formed while G stays above -100 powers of two

__host__ __device__ constexpr int cc_rows(bool delta) { return delta ? 2 * CC_Q : CC_Q; }
// floats of a chunk that every block of `scan` reads, and all of them
__host__ __device__ constexpr int cc_shared(bool delta, int dkp) { return cc_rows(delta) * (dkp + 8) + CC_Q * (dkp + 4) + dkp; }
__host__ __device__ __forceinline__ long long cc_floats(bool delta, int dkp, int dvp) {
  return cc_shared(delta, dkp) + (long long)2 * CC_Q * dvp;
}
__device__ __forceinline__ float cc_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// A lane's VL elements of a row of 32 VL: groups of up to four neighbours.
template <int VL>
__device__ __forceinline__ void cc_row(const float* __restrict__ p, int lane, float (&v)[VL]) {
  if constexpr (VL >= 4) {
#pragma unroll
    for (int m = 0; m < VL / 4; ++m) {
      const float4 t = *reinterpret_cast<const float4*>(p + m * 128 + 4 * lane);
      v[4 * m] = t.x; v[4 * m + 1] = t.y; v[4 * m + 2] = t.z; v[4 * m + 3] = t.w;
    }
  } else if constexpr (VL == 2) {
    const float2 t = *reinterpret_cast<const float2*>(p + 2 * lane);
    v[0] = t.x; v[1] = t.y;
  } else {
    v[0] = p[lane];
  }
}
// N (a power of two, at most 32) values a lane, each to be added over the lanes: lane l ends with the sum of value l % N.
template <int N>
__device__ __forceinline__ float cc_transpose_sum(float (&v)[N], int lane) {
#pragma unroll
  for (int o = 16; o >= N; o >>= 1)
#pragma unroll
    for (int t = 0; t < N; ++t) v[t] += __shfl_xor_sync(0xffffffffu, v[t], o);
#pragma unroll
  for (int o = N / 2; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int t = 0; t < o; ++t) {
      const float send = up ? v[t] : v[t + o], keep = up ? v[t + o] : v[t];
      v[t] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return v[0];
}
// x <- (I + m)^-1 x for a strictly lower triangular m
__device__ __forceinline__ void cc_solve(const float (*__restrict__ m)[CC_Q], float (&x)[CC_Q]) {
#pragma unroll
  for (int i = 1; i < CC_Q; ++i)
#pragma unroll
    for (int j = 0; j < i; j += 4) {
      const float4 r = *reinterpret_cast<const float4*>(&m[i][j]);
      x[i] = fmaf(-r.x, x[j], x[i]);
      if (j + 1 < i) x[i] = fmaf(-r.y, x[j + 1], x[i]);
      if (j + 2 < i) x[i] = fmaf(-r.z, x[j + 2], x[i]);
      if (j + 3 < i) x[i] = fmaf(-r.w, x[j + 3], x[i]);
    }
}
// row i of m x for a lower triangular m
__device__ __forceinline__ float cc_apply(const float (*__restrict__ m)[CC_Q], const float (&x)[CC_Q], int i) {
  float s = 0.f;
#pragma unroll
  for (int j = 0; j < CC_Q; j += 4)
    if (j <= i) {
      const float4 r = *reinterpret_cast<const float4*>(&m[i][j]);
      s = fmaf(r.x, x[j], s);
      if (j + 1 <= i) s = fmaf(r.y, x[j + 1], s);
      if (j + 2 <= i) s = fmaf(r.z, x[j + 2], s);
      if (j + 3 <= i) s = fmaf(r.w, x[j + 3], s);
    }
  return s;
}

// pieces: int4 per chunk = segment, first row, rows (up to CC_Q), flags.
template <bool DELTA, typename T, int DKP>
__global__ void __launch_bounds__(CC_THREADS, CC_PREPARE_BLOCKS)
channel_prepare_kernel(const MemoryIn in, const int4* __restrict__ pieces, float* __restrict__ work, int dvp) {
  pdl_begin();
  extern __shared__ __align__(16) float cc_sh[];
  constexpr int VL = DKP / 32, MR = cc_rows(DELTA), AP = DKP + 8, KP = DKP + 4;
  float* qs = cc_sh;                                       // [16][DKP]
  float* ks = qs + CC_Q * DKP;
  float* hi = ks + CC_Q * DKP;                             // G in powers of two: hi + lo
  float* lo = hi + CC_Q * DKP;
  __shared__ __align__(16) float sys[CC_Q][CC_Q];          // beta_i A_ij, j < i
  __shared__ __align__(16) float bm[CC_Q][CC_Q];           // B_ij, j <= i
  __shared__ float bs[CC_Q];
  __shared__ float end_hi[DKP], end_lo[DKP];               // G_16
  const int4 piece = pieces[blockIdx.x];
  const int row0 = piece.y, nt = piece.z;
  const int H = in.H, dk = in.dk, dv = in.dv, h = blockIdx.y, g = h / (H / in.G);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const T* u = static_cast<const T*>(in.u);
  const float rate = DELTA ? in.rate[h] : 0.f;
  float* wa = work + ((size_t)blockIdx.x * H + h) * cc_floats(DELTA, DKP, dvp);
  float *wk = wa + MR * AP, *we = wk + CC_Q * KP, *wv = we + DKP;

  auto values = [&](int c, float (&x)[CC_Q]) {             // column c of v
#pragma unroll
    for (int i = 0; i < CC_Q; ++i)
      x[i] = i < nt && c < dv ? to_f<T>(u[(size_t)(row0 + i) * in.u_ld + in.v_off + h * dv + c]) : 0.f;
  };
  float ahead[CC_Q];                                       // a thread's first column, where that is one of v: on its way
  values((int)threadIdx.x >= DKP ? (int)threadIdx.x - DKP : dv, ahead);

  {
    constexpr int N = CC_Q * DKP / CC_THREADS;             // elements a thread: all loads first, then the arithmetic
    T qv[N], kv[N];
    float zv[N];
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int i = threadIdx.x + n * CC_THREADS, t = i / DKP, r = i % DKP;
      const bool ok = t < nt && r < dk;
      const size_t row = (size_t)(row0 + (ok ? t : 0));
      const int col = ok ? r : 0;
      qv[n] = u[row * in.u_ld + in.q_off + g * dk + col];
      kv[n] = u[row * in.u_ld + in.k_off + g * dk + col];
      zv[n] = in.z[row * in.z_ld + h * dk + col];
    }
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int i = threadIdx.x + n * CC_THREADS, t = i / DKP, r = i % DKP;
      const bool ok = t < nt && r < dk;
      qs[i] = ok ? (DELTA ? to_f<T>(qv[n]) : to_f<T>(qv[n]) * in.q_scale) : 0.f;
      ks[i] = ok ? to_f<T>(kv[n]) : 0.f;
      hi[i] = ok ? cm_log_decay<DELTA>(zv[n] + in.bias[h * dk + r], rate, in.sharp) : 0.f;
    }
  }
  if (threadIdx.x < CC_Q)
    bs[threadIdx.x] = !DELTA ? 1.f : threadIdx.x < nt
        ? cm_sigmoid(to_f<T>(static_cast<const T*>(in.beta)[(size_t)(row0 + threadIdx.x) * in.b_ld + h])) : 0.f;
  __syncthreads();
  if (DELTA)
    for (int t = warp; t < CC_Q; t += CC_THREADS / 32) {   // unit lengths, a warp per token
      float nq = 0.f, nk = 0.f;
#pragma unroll
      for (int e = 0; e < VL; ++e) {
        const float a = qs[t * DKP + lane + 32 * e], b = ks[t * DKP + lane + 32 * e];
        nq = fmaf(a, a, nq);
        nk = fmaf(b, b, nk);
      }
      nq = in.q_scale / sqrtf(warp_sum(nq) + in.unit_eps);
      nk = 1.f / sqrtf(warp_sum(nk) + in.unit_eps);
#pragma unroll
      for (int e = 0; e < VL; ++e) {
        qs[t * DKP + lane + 32 * e] *= nq;
        ks[t * DKP + lane + 32 * e] *= nk;
      }
    }
  bool strong = false;                                     // a decay that e^(-G) could not be formed for
  if (threadIdx.x < DKP) {
    const int r = threadIdx.x;
    double run = 0.0;
#pragma unroll
    for (int t = 0; t < CC_Q; ++t) {
      run += (double)hi[t * DKP + r] * 1.4426950408889634;
      const float top = (float)run;
      hi[t * DKP + r] = top;
      lo[t * DKP + r] = (float)(run - (double)top);
    }
    end_hi[r] = (float)run;
    end_lo[r] = (float)(run - (double)end_hi[r]);
    we[r] = cc_exp2(end_hi[r]);
    strong = end_hi[r] < -CC_WEAK;
  }
  strong = __syncthreads_or(strong);
  // q e^G and k e^G in place of q and k, k e^(-G) in place of G, K
  auto weigh = [&] {
#pragma unroll
    for (int n = 0; n < CC_Q * DKP / CC_THREADS; ++n) {
      const int i = threadIdx.x + n * CC_THREADS, t = i / DKP, r = i % DKP;
      const float top = hi[i], low = lo[i] * 0.6931471805599453f, k = ks[i];
      const float e = cc_exp2(top);
      const float grown = fmaf(e, low, e);
      wk[t * KP + r] = k * cc_exp2((end_hi[r] - top) + (end_lo[r] - lo[i]));
      qs[i] *= grown;
      ks[i] = k * grown;
      if (!strong) {
        const float inv = cc_exp2(-top);
        hi[i] = k * fmaf(inv, -low, inv);
      }
    }
    __syncthreads();
  };
  if (!strong) weigh();

  // A and B, two columns j a warp, so dealt that every warp has equal work under the triangle: as products of weighted rows,
  // or, where a decay within the chunk is too strong for that, pair by pair
#pragma unroll 1
  for (int half = 0; half < 2; ++half) {
    const int j = half ? CC_Q - 1 - warp : warp;
    float kj[VL], acc[MR];
#pragma unroll
    for (int i = 0; i < MR; ++i) acc[i] = 0.f;
    if (!strong) {
      cc_row<VL>(hi + j * DKP, lane, kj);
#pragma unroll
      for (int i = 0; i < CC_Q; ++i)
        if (i >= j) {
          float qi[VL], ki[VL];
          cc_row<VL>(qs + i * DKP, lane, qi);
          if (DELTA) cc_row<VL>(ks + i * DKP, lane, ki);
#pragma unroll
          for (int e = 0; e < VL; ++e) {
            acc[i] = fmaf(qi[e], kj[e], acc[i]);
            if constexpr (DELTA) acc[CC_Q + i] = fmaf(ki[e], kj[e], acc[CC_Q + i]);
          }
        }
    } else {
      float hj[VL], lj[VL];
      cc_row<VL>(ks + j * DKP, lane, kj);
      cc_row<VL>(hi + j * DKP, lane, hj);
      cc_row<VL>(lo + j * DKP, lane, lj);
#pragma unroll
      for (int i = 0; i < CC_Q; ++i)
        if (i >= j) {
          float qi[VL], ki[VL], hv[VL], lv[VL];
          cc_row<VL>(qs + i * DKP, lane, qi);
          if (DELTA) cc_row<VL>(ks + i * DKP, lane, ki);
          cc_row<VL>(hi + i * DKP, lane, hv);
          cc_row<VL>(lo + i * DKP, lane, lv);
#pragma unroll
          for (int e = 0; e < VL; ++e) {
            const float f = kj[e] * cc_exp2((hv[e] - hj[e]) + (lv[e] - lj[e]));
            acc[i] = fmaf(qi[e], f, acc[i]);
            if constexpr (DELTA) acc[CC_Q + i] = fmaf(ki[e], f, acc[CC_Q + i]);
          }
        }
    }
    const float sum = cc_transpose_sum<MR>(acc, lane);
    const int i = lane & (CC_Q - 1);
    if (lane < CC_Q) bm[i][j] = sum;                       // (zero above the diagonal)
    else if (DELTA) sys[i][j] = i > j ? bs[i] * sum : 0.f;
  }
  __syncthreads();
  if (strong) weigh();

  // the system, one column a thread: W from the weighted keys, w0 from the values
  for (int col = threadIdx.x; col < DKP + dvp; col += CC_THREADS) {
    if (col < DKP) {
      float x[CC_Q];
      if constexpr (DELTA) {
#pragma unroll
        for (int i = 0; i < CC_Q; ++i) x[i] = bs[i] * ks[i * DKP + col];
        cc_solve(sys, x);
#pragma unroll
        for (int i = 0; i < CC_Q; ++i) wa[i * AP + col] = x[i];
      }
#pragma unroll
      for (int i = 0; i < CC_Q; ++i) {
        const float q = qs[i * DKP + col];
        wa[(MR - CC_Q + i) * AP + col] = DELTA ? q - cc_apply(bm, x, i) : q;
      }
    } else {
      const int c = col - DKP;
      float* dst = wv + (size_t)(c / CC_COLS) * 2 * CC_Q * CC_COLS + c % CC_COLS;
      float x[CC_Q];
      if (col == threadIdx.x) {
#pragma unroll
        for (int i = 0; i < CC_Q; ++i) x[i] = ahead[i];
      } else {
        values(c, x);
      }
      if constexpr (DELTA) {
#pragma unroll
        for (int i = 0; i < CC_Q; ++i) x[i] *= bs[i];
        cc_solve(sys, x);
      }
#pragma unroll
      for (int i = 0; i < CC_Q; ++i) {
        dst[i * CC_COLS] = x[i];
        dst[(CC_Q + i) * CC_COLS] = cc_apply(bm, x, i);
      }
    }
  }
}

__device__ __forceinline__ void cc_cp_async16(void* smem, const void* gmem) {
  const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(gmem));
}
// Two floats in one register pair, and the multiply-add on both at once.
__device__ __forceinline__ unsigned long long cc_pair(float a, float b) {
  unsigned long long r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 cc_both(unsigned long long p) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(p));
  return r;
}
__device__ __forceinline__ void cc_fma2(unsigned long long& c, unsigned long long a, unsigned long long b) {
  asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(c) : "l"(a), "l"(b));
}

// One block per (segment, head, CC_COLS columns): S through the segment's chunks in order.  S lies twice: in the registers
// of threads 0 .. DKP-1 (four neighbouring rows, four columns each), which take it past a chunk, and transposed in shared
// memory for the product [W; q - B W] S, whose sum over S's rows is split over the eight warps.  That product runs on
// pairs of neighbouring rows, S's step on pairs of rows with w doubled: no operand is shuffled.
template <bool DELTA, int DKP>
__global__ void __launch_bounds__(CC_THREADS, DKP <= 128 ? 2 : 1)
channel_scan_kernel(const float* __restrict__ work, const int4* __restrict__ pieces, const int* __restrict__ cu_pieces,
                    const int* __restrict__ seg_start, const int* __restrict__ seg_slot, float* __restrict__ state,
                    float* __restrict__ out, int H, int dk, int dv, int dvp) {
  pdl_begin();
  extern __shared__ __align__(16) float cc_sh[];
  constexpr int MR = cc_rows(DELTA), TR = MR / 8, AP = DKP + 8, KP = DKP + 4;    // TR: rows of the product a lane holds
  constexpr int KEEP = cc_shared(DELTA, DKP), VALS = 2 * CC_Q * CC_COLS, BUF = KEEP + VALS;
  constexpr int KW = DKP / 8;                              // rows of S a warp takes in the product
  float* St = cc_sh + 2 * BUF;                             // [16][AP]
  float* part = St + CC_COLS * AP;                         // [8 warps][TR][32 lanes][4]
  float* ws = part + 8 * TR * 128;                         // [16][16][2]
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * CC_COLS;
  const int p0 = cu_pieces[b], p1 = cu_pieces[b + 1];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const size_t step = (size_t)cc_floats(DELTA, DKP, dvp);

  auto load = [&](int p) {
    if (p < p1) {
      const float* src = work + ((size_t)p * H + h) * step;
      float* dst = cc_sh + ((p - p0) & 1) * BUF;
#pragma unroll
      for (int n = 0; n < (KEEP / 4 + CC_THREADS - 1) / CC_THREADS; ++n) {
        const int i = tid + n * CC_THREADS;
        if (i < KEEP / 4) cc_cp_async16(dst + 4 * i, src + 4 * i);
      }
      if (tid < VALS / 4) cc_cp_async16(dst + KEEP + 4 * tid, src + KEEP + (size_t)blockIdx.z * VALS + 4 * tid);
    }
    asm volatile("cp.async.commit_group;");
  };
  load(p0);

  const int sr = 4 * (tid >> 2), sc = 4 * (tid & 3);       // my rows and columns of S
  float* slot = state + ((size_t)seg_slot[b] * H + h) * dk * dv;
  float S[4][4];                                           // [column][row]
  if (tid < DKP) {
    const bool fresh = seg_start[b] == 0;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        S[j][e] = !fresh && sr + e < dk && col0 + sc + j < dv ? slot[(size_t)(sr + e) * dv + col0 + sc + j] : 0.f;
      *reinterpret_cast<float4*>(St + (sc + j) * AP + sr) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
    }
  }
  // the element (i, c) of the chunk's 16 x 16 outputs that lies at place tid of the partial sums
  const int i = ((tid & 127) >> 4) + 8 * (tid >> 7), c = ((tid >> 2) & 3) + 4 * (tid & 3);

  for (int p = p0; p < p1; ++p) {
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();
    load(p + 1);
    const int4 piece = pieces[p];
    const float* buf = cc_sh + ((p - p0) & 1) * BUF;
    const float *ka = buf + MR * AP, *ea = ka + CC_Q * KP, *va = buf + KEEP;
    {
      unsigned long long acc[TR][4];                       // rows g + 8 r, columns ct + 4 cc: sums of even and odd rows of S
#pragma unroll
      for (int r = 0; r < TR; ++r)
#pragma unroll
        for (int cc = 0; cc < 4; ++cc) acc[r][cc] = 0ull;
      const float* arow = buf + (lane >> 2) * AP + warp * KW;
      const float* srow = St + (lane & 3) * AP + warp * KW;
#pragma unroll
      for (int k = 0; k < KW; k += 4) {
        ulonglong2 a[TR], s[4];
#pragma unroll
        for (int cc = 0; cc < 4; ++cc) s[cc] = *reinterpret_cast<const ulonglong2*>(srow + 4 * cc * AP + k);
#pragma unroll
        for (int r = 0; r < TR; ++r) a[r] = *reinterpret_cast<const ulonglong2*>(arow + 8 * r * AP + k);
#pragma unroll
        for (int r = 0; r < TR; ++r)
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) {
            cc_fma2(acc[r][cc], a[r].x, s[cc].x);
            cc_fma2(acc[r][cc], a[r].y, s[cc].y);
          }
      }
#pragma unroll
      for (int r = 0; r < TR; ++r) {
        float v[4];
#pragma unroll
        for (int cc = 0; cc < 4; ++cc) {
          const float2 t = cc_both(acc[r][cc]);
          v[cc] = t.x + t.y;
        }
        *reinterpret_cast<float4*>(part + ((warp * TR + r) * 32 + lane) * 4) = make_float4(v[0], v[1], v[2], v[3]);
      }
    }
    if (!DELTA) *reinterpret_cast<float2*>(ws + 2 * (i * CC_COLS + c)) = make_float2(va[i * CC_COLS + c], va[i * CC_COLS + c]);
    __syncthreads();
    float o = va[(CC_Q + i) * CC_COLS + c];
    if constexpr (DELTA) {
      float w = va[i * CC_COLS + c], known = 0.f;
#pragma unroll
      for (int n = 0; n < 8; ++n) known += part[n * TR * 128 + tid];
      w -= known;
      *reinterpret_cast<float2*>(ws + 2 * (i * CC_COLS + c)) = make_float2(w, w);
      __syncthreads();
    }
    if (tid < DKP) {                                       // S past the chunk
      unsigned long long acc[4][2];
      const ulonglong2 e2 = *reinterpret_cast<const ulonglong2*>(ea + sr);
      const float2 ex = cc_both(e2.x), ey = cc_both(e2.y);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[j][0] = cc_pair(ex.x * S[j][0], ex.y * S[j][1]);
        acc[j][1] = cc_pair(ey.x * S[j][2], ey.y * S[j][3]);
      }
#pragma unroll
      for (int t = 0; t < CC_Q; ++t) {
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(ka + t * KP + sr);
        const ulonglong2 w01 = *reinterpret_cast<const ulonglong2*>(ws + 2 * (t * CC_COLS + sc));
        const ulonglong2 w23 = *reinterpret_cast<const ulonglong2*>(ws + 2 * (t * CC_COLS + sc) + 4);
        cc_fma2(acc[0][0], k2.x, w01.x); cc_fma2(acc[0][1], k2.y, w01.x);
        cc_fma2(acc[1][0], k2.x, w01.y); cc_fma2(acc[1][1], k2.y, w01.y);
        cc_fma2(acc[2][0], k2.x, w23.x); cc_fma2(acc[2][1], k2.y, w23.x);
        cc_fma2(acc[3][0], k2.x, w23.y); cc_fma2(acc[3][1], k2.y, w23.y);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 a = cc_both(acc[j][0]), d = cc_both(acc[j][1]);
        S[j][0] = a.x; S[j][1] = a.y; S[j][2] = d.x; S[j][3] = d.y;
        *reinterpret_cast<float4*>(St + (sc + j) * AP + sr) = make_float4(a.x, a.y, d.x, d.y);
      }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) o += part[n * TR * 128 + (DELTA ? 256 : 0) + tid];
    if (i < piece.z && col0 + c < dv) out[((size_t)(piece.y + i) * H + h) * dv + col0 + c] = o;
  }
  if (tid < DKP && p1 > p0)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (sr + e < dk && col0 + sc + j < dv) slot[(size_t)(sr + e) * dv + col0 + sc + j] = S[j][e];
}

// The same on the tensor cores, for bfloat16 models: S^T in the accumulators of mma.sync m16n8k16 (warp w holds 16 KS rows of S
// by 16 columns).  Every float factor goes in as three bfloat16 terms that add up to its 24 bits, and of the nine products
// of terms the six largest are formed: what is left out lies below float's last bit.
__device__ __forceinline__ void cc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two floats as three packed pairs of bfloat16 whose sums are the floats: each term the top half of what is left.
__device__ __forceinline__ void cc_split3(float a, float b, uint32_t& t0, uint32_t& t1, uint32_t& t2) {
  uint32_t ua = __float_as_uint(a), ub = __float_as_uint(b);
  t0 = __byte_perm(ua, ub, 0x7632);
  a -= __uint_as_float(ua & 0xffff0000u);
  b -= __uint_as_float(ub & 0xffff0000u);
  ua = __float_as_uint(a);
  ub = __float_as_uint(b);
  t1 = __byte_perm(ua, ub, 0x7632);
  a -= __uint_as_float(ua & 0xffff0000u);
  b -= __uint_as_float(ub & 0xffff0000u);
  t2 = __byte_perm(__float_as_uint(a), __float_as_uint(b), 0x7632);
}
// c_n += a b_n over the six largest products of terms, the small ones first; the N sums take turns, so that no product waits
// for the one before it
template <int N>
__device__ __forceinline__ void cc_mma6(float (*__restrict__ c)[4], const uint32_t (&a)[3][4], const uint32_t (&b)[N][2][3]) {
  constexpr int TA[6] = {2, 1, 0, 1, 0, 0}, TB[6] = {0, 1, 2, 0, 1, 0};
#pragma unroll
  for (int q = 0; q < 6; ++q)
#pragma unroll
    for (int n = 0; n < N; ++n) cc_mma(c[n], a[TA[q]], b[n][0][TB[q]], b[n][1][TB[q]]);
}

#define CC_PS 20               // floats per row of the partial sums
#define CC_WS 24               // bfloat16 per column of w's terms
template <bool DELTA, int DKP>
__host__ __device__ constexpr int cc_mma_warps() { return DKP / 16 < 8 ? DKP / 16 : 8; }

template <bool DELTA, int DKP>
__global__ void __launch_bounds__(CC_THREADS, DKP <= 128 ? 2 : 1)
channel_scan_mma_kernel(const float* __restrict__ work, const int4* __restrict__ pieces, const int* __restrict__ cu_pieces,
                        const int* __restrict__ seg_start, const int* __restrict__ seg_slot, float* __restrict__ state,
                        float* __restrict__ out, int H, int dk, int dv, int dvp) {
  pdl_begin();
  extern __shared__ __align__(16) float cc_sh[];
  constexpr int MR = cc_rows(DELTA), AP = DKP + 8, KP = DKP + 4;
  constexpr int NW = cc_mma_warps<DELTA, DKP>(), KS = DKP / (16 * NW);     // warps that hold S, 16-row steps of each
  constexpr int KEEP = cc_shared(DELTA, DKP), VALS = 2 * CC_Q * CC_COLS, BUF = KEEP + VALS;
  float* part = cc_sh + 2 * BUF;                           // [NW][MR][CC_PS]
  bf16* ws = reinterpret_cast<bf16*>(part + NW * MR * CC_PS);      // [3 terms][16 columns][CC_WS]
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * CC_COLS;
  const int p0 = cu_pieces[b], p1 = cu_pieces[b + 1];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const size_t step = (size_t)cc_floats(DELTA, DKP, dvp);

  auto load = [&](int p) {
    if (p < p1) {
      const float* src = work + ((size_t)p * H + h) * step;
      float* dst = cc_sh + ((p - p0) & 1) * BUF;
#pragma unroll
      for (int n = 0; n < (KEEP / 4 + CC_THREADS - 1) / CC_THREADS; ++n) {
        const int i = tid + n * CC_THREADS;
        if (i < KEEP / 4) cc_cp_async16(dst + 4 * i, src + 4 * i);
      }
      if (tid < VALS / 4) cc_cp_async16(dst + KEEP + 4 * tid, src + KEEP + (size_t)blockIdx.z * VALS + 4 * tid);
    }
    asm volatile("cp.async.commit_group;");
  };
  load(p0);

  // S[k][n]: rows row0 + 16 k + 8 n + 2 t + {0, 1}, columns g (elements 0, 1) and g + 8 (2, 3)
  float S[KS][2][4];
  const int row0 = warp * 16 * KS;
  float* slot = state + ((size_t)seg_slot[b] * H + h) * dk * dv;
  if (warp < NW) {
    const bool fresh = seg_start[b] == 0;
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = row0 + 16 * k + 8 * n + 2 * t + (e & 1), c = col0 + g + 8 * (e >> 1);
          S[k][n][e] = !fresh && r < dk && c < dv ? slot[(size_t)r * dv + c] : 0.f;
        }
  }
  const int i = tid >> 4, c = tid & 15;                    // my element of the chunk's 16 x 16 outputs

  for (int p = p0; p < p1; ++p) {
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();
    load(p + 1);
    const int4 piece = pieces[p];
    const float* buf = cc_sh + ((p - p0) & 1) * BUF;
    const float *ka = buf + MR * AP, *ea = ka + CC_Q * KP, *va = buf + KEEP;
    uint32_t kb[KS][2][2][3];                              // K's terms: tokens 2 t, 2 t + 1 (and + 8), row g of each tile
    if (warp < NW) {
      float acc[MR / 8][4];                                // columns g, g + 8; rows 2 t, 2 t + 1 of the product
#pragma unroll
      for (int m = 0; m < MR / 8; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[m][e] = 0.f;
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t sa[3][4];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          cc_split3(S[k][n][0], S[k][n][1], sa[0][2 * n], sa[1][2 * n], sa[2][2 * n]);
          cc_split3(S[k][n][2], S[k][n][3], sa[0][2 * n + 1], sa[1][2 * n + 1], sa[2][2 * n + 1]);
        }
        const float* arow = buf + g * AP + row0 + 16 * k + 2 * t;
        uint32_t ab[MR / 8][2][3];
#pragma unroll
        for (int m = 0; m < MR / 8; ++m)
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const float2 v = *reinterpret_cast<const float2*>(arow + 8 * m * AP + 8 * q);
            cc_split3(v.x, v.y, ab[m][q][0], ab[m][q][1], ab[m][q][2]);
          }
        cc_mma6<MR / 8>(acc, sa, ab);
      }
      float* at = part + (warp * MR + 2 * t) * CC_PS + g;
#pragma unroll
      for (int m = 0; m < MR / 8; ++m) {
        at[8 * m * CC_PS] = acc[m][0];
        at[(8 * m + 1) * CC_PS] = acc[m][1];
        at[8 * m * CC_PS + 8] = acc[m][2];
        at[(8 * m + 1) * CC_PS + 8] = acc[m][3];
      }
#pragma unroll
      for (int k = 0; k < KS; ++k)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const float* kr = ka + (2 * t + 8 * q) * KP + row0 + 16 * k + 8 * n + g;
            cc_split3(kr[0], kr[KP], kb[k][n][q][0], kb[k][n][q][1], kb[k][n][q][2]);
          }
    }
    __syncthreads();
    float o = va[(CC_Q + i) * CC_COLS + c], w = va[i * CC_COLS + c];
    if constexpr (DELTA) {
      float known = 0.f;
#pragma unroll
      for (int n = 0; n < NW; ++n) known += part[(n * MR + i) * CC_PS + c];
      w -= known;
    }
    {
      uint32_t t0, t1, t2;
      cc_split3(w, 0.f, t0, t1, t2);
      unsigned short* at = reinterpret_cast<unsigned short*>(ws) + c * CC_WS + i;
      at[0] = (unsigned short)t0;
      at[16 * CC_WS] = (unsigned short)t1;
      at[32 * CC_WS] = (unsigned short)t2;
    }
    __syncthreads();
    if (warp < NW) {                                       // S past the chunk
      uint32_t wa[3][4];
#pragma unroll
      for (int q = 0; q < 3; ++q) {
        const bf16* at = ws + (q * 16 + g) * CC_WS + 2 * t;
        wa[q][0] = *reinterpret_cast<const uint32_t*>(at);
        wa[q][1] = *reinterpret_cast<const uint32_t*>(at + 8 * CC_WS);
        wa[q][2] = *reinterpret_cast<const uint32_t*>(at + 8);
        wa[q][3] = *reinterpret_cast<const uint32_t*>(at + 8 * CC_WS + 8);
      }
#pragma unroll
      for (int k = 0; k < KS; ++k)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const float2 e2 = *reinterpret_cast<const float2*>(ea + row0 + 16 * k + 8 * n + 2 * t);
          S[k][n][0] *= e2.x; S[k][n][1] *= e2.y; S[k][n][2] *= e2.x; S[k][n][3] *= e2.y;
        }
#pragma unroll
      for (int k = 0; k < KS; ++k) cc_mma6<2>(S[k], wa, kb[k]);
    }
#pragma unroll
    for (int n = 0; n < NW; ++n) o += part[(n * MR + MR - CC_Q + i) * CC_PS + c];
    if (i < piece.z && col0 + c < dv) out[((size_t)(piece.y + i) * H + h) * dv + col0 + c] = o;
  }
  if (warp < NW && p1 > p0)
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = row0 + 16 * k + 8 * n + 2 * t + (e & 1), cc = col0 + g + 8 * (e >> 1);
          if (r < dk && cc < dv) slot[(size_t)r * dv + cc] = S[k][n][e];
        }
}

// ---------------------------------------------------------------------------------------------
static int cm_rows_padded(int dk) { return dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 128 ? 128 : 256)); }

// Floats of `work` per chunk for these sizes.
SNK_API long long snk_channel_memory_work(int delta, int H, int dk, int dv) {
  return (long long)H * cc_floats(delta != 0, cm_rows_padded(dk), (dv + CC_COLS - 1) / CC_COLS * CC_COLS);
}

template <bool DELTA>
static int channel_memory(const MemoryIn& in, const int* cu_seqlens, const int* seg_start, const int* seg_slot,
                          float* state, float* out, int B, int max_len, const int* pieces, const int* cu_pieces,
                          int n_pieces, float* work, int dtype, cudaStream_t stream) {
  const int H = in.H, dk = in.dk, dv = in.dv;
  if (n_pieces > 0) {
    const int dvp = (dv + CC_COLS - 1) / CC_COLS * CC_COLS, slices = dvp / CC_COLS;
    if (slices > 65535) return SNK_ERR_SIZE;
    const int4* table = reinterpret_cast<const int4*>(pieces);
#define CC_LAUNCH(DKP_)                                                                                        \
  do {                                                                                                         \
    auto prepare = channel_prepare_kernel<DELTA, T, DKP_>;                                                     \
    const size_t psmem = (size_t)4 * CC_Q * DKP_ * sizeof(float);                                              \
    if (psmem > 48 * 1024) cudaFuncSetAttribute(prepare, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)psmem); \
    snk_launch(prepare, dim3(n_pieces, H), dim3(CC_THREADS), psmem, stream, in, table, work, dvp);             \
    SNK_LAUNCH_CHECK();                                                                                        \
    const bool mma = dtype == SNK_BF16;                                                                        \
    auto scan = mma ? channel_scan_mma_kernel<DELTA, DKP_> : channel_scan_kernel<DELTA, DKP_>;                 \
    size_t ssmem = (size_t)2 * (cc_shared(DELTA, DKP_) + 2 * CC_Q * CC_COLS) * sizeof(float);                  \
    if (mma) ssmem += (size_t)cc_mma_warps<DELTA, DKP_>() * cc_rows(DELTA) * CC_PS * sizeof(float) + 48 * CC_WS * sizeof(bf16); \
    else ssmem += (size_t)(CC_COLS * (DKP_ + 8) + cc_rows(DELTA) * 128 + 2 * CC_Q * CC_COLS) * sizeof(float);  \
    if (ssmem > 48 * 1024) cudaFuncSetAttribute(scan, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ssmem); \
    snk_launch(scan, dim3(B, H, slices), dim3(CC_THREADS), ssmem, stream, (const float*)work, table, cu_pieces, \
               seg_start, seg_slot, state, out, H, dk, dv, dvp);                                               \
  } while (0)
    SNK_DISPATCH(dtype, {
      if (dk <= 32) CC_LAUNCH(32);
      else if (dk <= 64) CC_LAUNCH(64);
      else if (dk <= 128) CC_LAUNCH(128);
      else CC_LAUNCH(256);
    });
#undef CC_LAUNCH
    SNK_LAUNCH_CHECK();
    return 0;
  }
  const bool wide = (dv & 3) == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)out % 16 == 0;
  int lpr = 1;                                             // lanes a row of S
  while (lpr < 32 && 4 * lpr < dv) lpr *= 2;
  const int per_thread = (dk * lpr + CS_THREADS - 1) / CS_THREADS;
  if (max_len == 1 && wide && per_thread <= 16) {
    const dim3 grid(B, H, (dv + 127) / 128);
#define CS_LAUNCH(RPT_)                                                                                        \
  snk_launch(channel_step_kernel<DELTA, T, RPT_>, grid, dim3(CS_THREADS), 0, stream, in, cu_seqlens, seg_start, \
             seg_slot, state, out, lpr)
    SNK_DISPATCH(dtype, {
      if (per_thread <= 2) CS_LAUNCH(2);
      else if (per_thread <= 4) CS_LAUNCH(4);
      else if (per_thread <= 8) CS_LAUNCH(8);
      else CS_LAUNCH(16);
    });
#undef CS_LAUNCH
    SNK_LAUNCH_CHECK();
    return 0;
  }
  const int cpt = dv > 2 * CM_GROUPS && wide ? 4 : 1;
  const int cols = CM_GROUPS * cpt, slices = (dv + cols - 1) / cols;
  const int dkp = (dk + 4 * CM_TPC - 1) / (4 * CM_TPC) * (4 * CM_TPC);
  const int tokens = max_len < CM_TOKENS ? max_len : CM_TOKENS;
  const size_t smem = (size_t)tokens * (3 * dkp + cols + 1) * sizeof(float);
#define CM_LAUNCH(DKR_, CPT_)                                                                                  \
  do {                                                                                                         \
    auto kernel = channel_walk_kernel<DELTA, T, DKR_, CPT_>;                                                   \
    if (smem > 48 * 1024)                                                                                      \
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                    \
    snk_launch(kernel, dim3(B, H, slices), dim3(CM_THREADS), smem, stream, in, cu_seqlens, seg_start, seg_slot, \
               state, out, tokens);                                                                            \
  } while (0)
#define CM_SIZES(CPT_)                                                                                         \
  do {                                                                                                         \
    if (dk <= 32) CM_LAUNCH(32, CPT_);                                                                         \
    else if (dk <= 64) CM_LAUNCH(64, CPT_);                                                                    \
    else if (dk <= 128) CM_LAUNCH(128, CPT_);                                                                  \
    else CM_LAUNCH(256, CPT_);                                                                                 \
  } while (0)
  SNK_DISPATCH(dtype, {
    if (cpt == 4) CM_SIZES(4);
    else CM_SIZES(1);
  });
#undef CM_SIZES
#undef CM_LAUNCH
  SNK_LAUNCH_CHECK();
  return 0;
}

// u: compute dtype [M, u_ld].  z: float, beta: compute dtype (null: the linear form), both from their first column on.
// bias float [H*dk]; rate float [H] (delta form).  state: float [slots, H, dk, dv].  out: float [M, H*dv].  max_len: the
// longest segment.  n_pieces 0: step or walk.  Otherwise pieces int32 [n_pieces, 4] (segment, first row, rows up to 16,
// flags), cu_pieces int32 [B+1] (first piece of each segment) and work (snk_channel_memory_work floats per piece).
SNK_API int snk_channel_memory(const void* u, long long u_ld, int q_off, int k_off, int v_off, const float* z,
                               long long z_ld, const float* bias, const float* rate, const void* beta, long long b_ld,
                               float sharp, float q_scale, float unit_eps, const int* cu_seqlens, const int* seg_start,
                               const int* seg_slot, float* state, float* out, int B, int H, int G, int dk, int dv,
                               int max_len, const int* pieces, const int* cu_pieces, int n_pieces, float* work,
                               int dtype, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H <= 0 || H > 65535 || G <= 0 || H % G || dk <= 0 || dk > 256 || dv <= 0 || dv > 32 * 65535 || max_len <= 0 ||
      z_ld < (long long)H * dk || !bias || (beta && !rate) || n_pieces < 0)
    return SNK_ERR_SIZE;
  if (n_pieces && (!pieces || !cu_pieces || !work)) return SNK_ERR_SIZE;
  if (n_pieces && (((uintptr_t)pieces | (uintptr_t)work) & 15)) return SNK_ERR_ALIGN;
  const MemoryIn in{u, u_ld, q_off, k_off, v_off, z, z_ld, bias, rate, beta, b_ld, sharp, q_scale, unit_eps, H, G, dk, dv};
  return beta ? channel_memory<true>(in, cu_seqlens, seg_start, seg_slot, state, out, B, max_len, pieces, cu_pieces,
                                     n_pieces, work, dtype, stream)
              : channel_memory<false>(in, cu_seqlens, seg_start, seg_slot, state, out, B, max_len, pieces, cu_pieces,
                                      n_pieces, work, dtype, stream);
}
