// The gated delta rule over a flat batch of segments: a matrix memory that takes off what it already answers to a key
// before it writes.
//
// Per head a float matrix S [dk, dv], zero for a fresh request, kept in the request's state slot between steps:
//
//   S <- diag(a_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
//
//   q, k  unit vectors per head, x / sqrt(sum(x^2) + unit_eps), q times q_scale; head h reads q/k head h / (H / G)
//   a_t   exp(rate[h] * softplus(z_t + bias)) per head and channel (rate = -exp(A_log)), z float rows of their own
//   beta  sigmoid of a logit per head
//
// q, k and v are columns of the convolved rows `u` in the compute dtype; lengths, decays, betas, state, sums and outputs
// are float.
//
// The walk (any step): a block serves one (segment, head, slice of columns of S).  Eight neighbouring threads share a
// group of one or four columns, each holding an eighth of its rows in registers over the whole segment; up to DL_TOKENS
// tokens' q, k, decays, v and beta come into shared memory at a time.
#include "common.cuh"

#define DL_TOKENS 16
#define DL_TPC 8               // threads per column group
#define DL_GROUPS 32           // column groups per block
#define DL_THREADS (DL_TPC * DL_GROUPS)

struct DeltaIn {
  const void* u;                 // compute dtype, row pitch u_ld
  long long u_ld;
  int q_off, k_off, v_off;
  const float* z;                // row pitch z_ld
  long long z_ld;
  const float* bias;             // [H*dk]
  const float* rate;             // [H]
  const void* beta;              // compute dtype, row pitch b_ld
  long long b_ld;
  float q_scale, unit_eps;
  int H, G, dk, dv;
};

// log(1 + e^z)
__device__ __forceinline__ float dl_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T, int DKR, int CPT>
__global__ void __launch_bounds__(DL_THREADS)
delta_walk_kernel(const DeltaIn in, const int* __restrict__ cu_seqlens, const int* __restrict__ seg_start,
                  const int* __restrict__ seg_slot, float* __restrict__ state, float* __restrict__ out, int tokens) {
  pdl_begin();
  extern __shared__ __align__(16) float dl_sh[];
  constexpr int RPT = DKR / DL_TPC;                        // rows of S per thread
  constexpr int COLS = DL_GROUPS * CPT;
  const int dk = in.dk, dv = in.dv, H = in.H;
  const int dkp = (dk + 4 * DL_TPC - 1) / (4 * DL_TPC) * (4 * DL_TPC);
  float* qs = dl_sh;                                       // [tokens][dkp]
  float* ks = qs + tokens * dkp;
  float* as = ks + tokens * dkp;
  float* vs = as + tokens * dkp;                           // [tokens][COLS]
  float* bs = vs + tokens * COLS;                          // [tokens]
  const int b = blockIdx.x, h = blockIdx.y, g = h / (H / in.G);
  const int sub = threadIdx.x & (DL_TPC - 1), group = threadIdx.x / DL_TPC;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col0 = blockIdx.z * COLS, c = col0 + group * CPT;
  const int row0 = cu_seqlens[b], row1 = cu_seqlens[b + 1];
  if (row1 <= row0) return;
  float* slot = state + ((size_t)seg_slot[b] * H + h) * dk * dv;
  const bool fresh = seg_start[b] == 0;
  const bool wide = CPT == 4 && (dv & 3) == 0;             // my four columns as one 16-byte access (all or none exist)

  // registers [i*4 + e][j] hold row 4 DL_TPC i + 4 sub + e, column c + j
  float S[RPT][CPT];
#pragma unroll
  for (int i = 0; i < RPT / 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = 4 * DL_TPC * i + 4 * sub + e;
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
  const float rate = in.rate[h];
  const T* u = static_cast<const T*>(in.u);
  for (int t0 = row0; t0 < row1; t0 += tokens) {
    const int nt = min(tokens, row1 - t0);
    __syncthreads();                                       // everyone is done with the previous tokens
    for (int i = threadIdx.x; i < nt * dkp; i += DL_THREADS) {
      const int t = i / dkp, r = i - t * dkp;
      float qv = 0.f, kv = 0.f, av = 0.f;
      if (r < dk) {
        const T* row = u + (size_t)(t0 + t) * in.u_ld;
        qv = to_f<T>(row[in.q_off + g * dk + r]);
        kv = to_f<T>(row[in.k_off + g * dk + r]);
        av = expf(rate * dl_softplus(in.z[(size_t)(t0 + t) * in.z_ld + h * dk + r] + in.bias[h * dk + r]));
      }
      qs[i] = qv;
      ks[i] = kv;
      as[i] = av;
    }
    for (int i = threadIdx.x; i < nt * COLS; i += DL_THREADS) {
      const int t = i / COLS, d = i - t * COLS;
      vs[i] = col0 + d < dv ? to_f<T>(u[(size_t)(t0 + t) * in.u_ld + in.v_off + h * dv + col0 + d]) : 0.f;
    }
    if (threadIdx.x < nt) {
      const float z = to_f<T>(static_cast<const T*>(in.beta)[(size_t)(t0 + threadIdx.x) * in.b_ld + h]);
      bs[threadIdx.x] = 1.f / (1.f + expf(-z));
    }
    __syncthreads();
    for (int t = warp; t < nt; t += DL_THREADS / 32) {     // unit lengths, a warp per token
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
        if (4 * DL_TPC * i < dk) {
          const float4 k4 = *reinterpret_cast<const float4*>(kt + 4 * DL_TPC * i + 4 * sub);
          const float4 a4 = *reinterpret_cast<const float4*>(at + 4 * DL_TPC * i + 4 * sub);
          const float kv[4] = {k4.x, k4.y, k4.z, k4.w}, av[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
          for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int j = 0; j < CPT; ++j) {
              S[i * 4 + e][j] *= av[e];
              known[j] = fmaf(S[i * 4 + e][j], kv[e], known[j]);
            }
        }
#pragma unroll
      for (int w = 1; w < DL_TPC; w <<= 1)
#pragma unroll
        for (int j = 0; j < CPT; ++j) known[j] += __shfl_xor_sync(0xffffffffu, known[j], w);
      const float beta = bs[t];
      float write[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) write[j] = beta * (vs[t * COLS + group * CPT + j] - known[j]);
#pragma unroll
      for (int i = 0; i < RPT / 4; ++i)
        if (4 * DL_TPC * i < dk) {
          const float4 k4 = *reinterpret_cast<const float4*>(kt + 4 * DL_TPC * i + 4 * sub);
          const float4 q4 = *reinterpret_cast<const float4*>(qt + 4 * DL_TPC * i + 4 * sub);
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
      for (int w = 1; w < DL_TPC; w <<= 1)
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
      const int r = 4 * DL_TPC * i + 4 * sub + e;
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

// u: compute dtype [M, u_ld].  z: float, beta: compute dtype, both from their first column on.  bias float [H*dk], rate
// float [H].  state: float [slots, H, dk, dv].  out: float [M, H*dv].  max_len: the longest segment.
SNK_API int snk_delta_memory(const void* u, long long u_ld, int q_off, int k_off, int v_off, const float* z,
                             long long z_ld, const float* bias, const float* rate, const void* beta, long long b_ld,
                             float q_scale, float unit_eps, const int* cu_seqlens, const int* seg_start,
                             const int* seg_slot, float* state, float* out, int B, int H, int G, int dk, int dv,
                             int max_len, int dtype, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H <= 0 || H > 65535 || G <= 0 || H % G || dk <= 0 || dk > 256 || dv <= 0 || dv > 32 * 65535 || max_len <= 0)
    return SNK_ERR_SIZE;
  const DeltaIn in{u, u_ld, q_off, k_off, v_off, z, z_ld, bias, rate, beta, b_ld, q_scale, unit_eps, H, G, dk, dv};
  const int cpt = dv > 2 * DL_GROUPS && (dv & 3) == 0 && (uintptr_t)state % 16 == 0 ? 4 : 1;
  const int cols = DL_GROUPS * cpt, slices = (dv + cols - 1) / cols;
  const int dkp = (dk + 4 * DL_TPC - 1) / (4 * DL_TPC) * (4 * DL_TPC);
  const int tokens = max_len < DL_TOKENS ? max_len : DL_TOKENS;
  const size_t smem = (size_t)tokens * (3 * dkp + cols + 1) * sizeof(float);
#define DL_LAUNCH(DKR_, CPT_)                                                                                 \
  do {                                                                                                        \
    auto kernel = delta_walk_kernel<T, DKR_, CPT_>;                                                           \
    if (smem > 48 * 1024)                                                                                     \
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                   \
    snk_launch(kernel, dim3(B, H, slices), dim3(DL_THREADS), smem, stream, in, cu_seqlens, seg_start, seg_slot, \
               state, out, tokens);                                                                           \
  } while (0)
#define DL_ROWS(CPT_)                                                                                         \
  do {                                                                                                        \
    if (dk <= 32) DL_LAUNCH(32, CPT_);                                                                        \
    else if (dk <= 64) DL_LAUNCH(64, CPT_);                                                                   \
    else if (dk <= 128) DL_LAUNCH(128, CPT_);                                                                 \
    else DL_LAUNCH(256, CPT_);                                                                                \
  } while (0)
  SNK_DISPATCH(dtype, {
    if (cpt == 4) DL_ROWS(4);
    else DL_ROWS(1);
  });
#undef DL_ROWS
#undef DL_LAUNCH
  SNK_LAUNCH_CHECK();
  return 0;
}
