// Selective state-space recurrence (Mamba-2) over a flat batch of segments, and the gated norm that follows it.
//
// Per head a float matrix S [N, P], zero for a fresh request, kept in the request's state slot between steps:
//
//   step = softplus(dt + dt_bias),  S_t = exp(-exp(a_log) step) S_(t-1) + step B_t x_t^T,  y_t = S_t^T C_t + D x_t
//
// x [H, P], B and C [G, N] (head h reads group h / (H / G)) are columns of the convolved rows `u` in the compute
// dtype; dt [H] is a column block of the projection.  Steps, decays, state, sums and outputs are float.
//
// The walk: a block serves one (segment, head, slice of 16 vectors of columns).  16 neighbouring threads share a row
// of S, 16 such groups take the rows in turns, each thread keeping its part of S in registers over the whole
// segment.  Up to SS_TOKENS tokens' inputs come into shared memory at a time; the groups' parts of S^T C are added
// within a warp by a shuffle, across warps through shared memory, once per such chunk.
#include "common.cuh"

#define SS_TOKENS 32
#define SS_LANES 16            // threads per row of S
#define SS_GROUPS 16           // rows of S at a time
#define SS_WARPS (SS_LANES * SS_GROUPS / 32)

// log(1 + e^z)
__device__ __forceinline__ float ss_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T, int VEC, int NI>
__global__ void __launch_bounds__(SS_LANES * SS_GROUPS)
state_space_walk_kernel(const T* __restrict__ u, long long u_ld, int x_off, int b_off, int c_off,
                        const void* __restrict__ dt, int dt_f32, long long dt_ld, const float* __restrict__ dt_bias,
                        const float* __restrict__ rate, const float* __restrict__ skip,
                        const int* __restrict__ cu_seqlens, const int* __restrict__ seg_start,
                        const int* __restrict__ seg_slot, float* __restrict__ state, float* __restrict__ out, int H,
                        int G, int N, int P, int tokens) {
  pdl_begin();
  extern __shared__ __align__(16) float ss_sh[];
  constexpr int COLS = SS_LANES * VEC;
  const int Np = SS_GROUPS * NI;
  float* bs = ss_sh;                                     // [tokens][Np]  step * B
  float* cs = bs + tokens * Np;                          // [tokens][Np]
  float* xs = cs + tokens * Np;                          // [tokens][COLS]
  float* part = xs + tokens * COLS;                      // [tokens][SS_WARPS][COLS]
  float* as = part + tokens * SS_WARPS * COLS;           // [tokens] decay
  float* st = as + tokens;                               // [tokens] step
  const int b = blockIdx.x, h = blockIdx.y;
  const int g = h / (H / G);
  const int lane = threadIdx.x % SS_LANES, group = threadIdx.x / SS_LANES;
  const int warp = threadIdx.x >> 5;
  const int c0 = blockIdx.z * COLS, c = c0 + lane * VEC;
  const int row0 = cu_seqlens[b], row1 = cu_seqlens[b + 1];
  if (row1 <= row0) return;
  float* slot = state + ((size_t)seg_slot[b] * H + h) * N * P;
  const bool fresh = seg_start[b] == 0;
  float S[NI][VEC];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int r = group + SS_GROUPS * i;
    if (!fresh && r < N && c < P) {
      if constexpr (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4*>(slot + (size_t)r * P + c);
        S[i][0] = v.x; S[i][1] = v.y; S[i][2] = v.z; S[i][3] = v.w;
      } else {
        S[i][0] = slot[(size_t)r * P + c];
      }
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) S[i][e] = 0.f;
    }
  }
  const float my_bias = dt_bias[h], my_rate = rate[h], my_skip = skip[h];
  for (int t0 = row0; t0 < row1; t0 += tokens) {
    const int nt = min(tokens, row1 - t0);
    __syncthreads();
    if (threadIdx.x < nt) {
      const size_t at = (size_t)(t0 + threadIdx.x) * dt_ld + h;
      const float z = dt_f32 ? static_cast<const float*>(dt)[at] : to_f<T>(static_cast<const T*>(dt)[at]);
      const float s = ss_softplus(z + my_bias);
      st[threadIdx.x] = s;
      as[threadIdx.x] = expf(my_rate * s);
    }
    for (int i = threadIdx.x; i < nt * COLS; i += blockDim.x) {
      const int t = i / COLS, d = i - t * COLS;
      xs[i] = c0 + d < P ? to_f<T>(u[(size_t)(t0 + t) * u_ld + x_off + (size_t)h * P + c0 + d]) : 0.f;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * Np; i += blockDim.x) {
      const int t = i / Np, r = i - t * Np;
      const T* row = u + (size_t)(t0 + t) * u_ld + (size_t)g * N;
      bs[i] = r < N ? st[t] * to_f<T>(row[b_off + r]) : 0.f;
      cs[i] = r < N ? to_f<T>(row[c_off + r]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float a = as[t];
      float x[VEC], acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        x[e] = xs[t * COLS + lane * VEC + e];
        acc[e] = 0.f;
      }
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float bv = bs[t * Np + group + SS_GROUPS * i], cv = cs[t * Np + group + SS_GROUPS * i];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          S[i][e] = fmaf(a, S[i][e], bv * x[e]);
          acc[e] = fmaf(S[i][e], cv, acc[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 16);
      if ((threadIdx.x & 31) < 16) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) part[(t * SS_WARPS + warp) * COLS + lane * VEC + e] = acc[e];
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * COLS; i += blockDim.x) {
      const int t = i / COLS, d = i - t * COLS;
      if (c0 + d >= P) continue;
      float y = 0.f;
#pragma unroll
      for (int w = 0; w < SS_WARPS; ++w) y += part[(t * SS_WARPS + w) * COLS + d];
      out[((size_t)(t0 + t) * H + h) * P + c0 + d] = fmaf(my_skip, xs[i], y);
    }
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int r = group + SS_GROUPS * i;
    if (r < N && c < P) {
      if constexpr (VEC == 4) *reinterpret_cast<float4*>(slot + (size_t)r * P + c) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
      else slot[(size_t)r * P + c] = S[i][0];
    }
  }
}

// u: compute dtype [M, u_ld].  dt: [M, dt_ld] from the first of its H columns on, float (dt_f32) or the compute
// dtype.  rate = -exp(a_log), dt_bias, skip: float [H].  state: float [slots, H, N, P].  out: float [M, H*P].
// max_len: the longest segment.
SNK_API int snk_state_space(const void* u, long long u_ld, int x_off, int b_off, int c_off, const void* dt, int dt_f32,
                            long long dt_ld, const float* dt_bias, const float* rate, const float* skip,
                            const int* cu_seqlens, const int* seg_start, const int* seg_slot, float* state, float* out,
                            int B, int H, int G, int N, int P, int max_len, int dtype, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (H <= 0 || H > 65535 || G <= 0 || H % G || N <= 0 || N > 256 || P <= 0 || max_len <= 0) return SNK_ERR_SIZE;
  const bool wide = P % 4 == 0 && (uintptr_t)state % 16 == 0;
  const int vec = wide ? 4 : 1, cols = SS_LANES * vec;
  const int slices = (P + cols - 1) / cols;
  if (slices > 65535) return SNK_ERR_SIZE;
  const int ni = N <= 16 ? 1 : (N <= 32 ? 2 : (N <= 64 ? 4 : (N <= 128 ? 8 : 16)));
  const int tokens = max_len < SS_TOKENS ? max_len : SS_TOKENS;
  const size_t smem = (size_t)tokens * (2 * SS_GROUPS * ni + cols + SS_WARPS * cols + 2) * sizeof(float);
#define SS_LAUNCH(VEC_, NI_)                                                                                  \
  do {                                                                                                        \
    auto kernel = state_space_walk_kernel<T, VEC_, NI_>;                                                      \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    snk_launch(kernel, dim3(B, H, slices), dim3(SS_LANES * SS_GROUPS), smem, stream, static_cast<const T*>(u), u_ld, \
               x_off, b_off, c_off, dt, dt_f32, dt_ld, dt_bias, rate, skip, cu_seqlens, seg_start, seg_slot, state,   \
               out, H, G, N, P, tokens);                                                                      \
  } while (0)
#define SS_ROWS(VEC_)                                                                                         \
  do {                                                                                                        \
    if (ni == 1) SS_LAUNCH(VEC_, 1);                                                                          \
    else if (ni == 2) SS_LAUNCH(VEC_, 2);                                                                     \
    else if (ni == 4) SS_LAUNCH(VEC_, 4);                                                                     \
    else if (ni == 8) SS_LAUNCH(VEC_, 8);                                                                     \
    else SS_LAUNCH(VEC_, 16);                                                                                 \
  } while (0)
  SNK_DISPATCH(dtype, {
    if (wide) SS_ROWS(4);
    else SS_ROWS(1);
  });
#undef SS_ROWS
#undef SS_LAUNCH
  SNK_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------------------------
// The gate before the norm: v = y * silu(z), each of `groups` equal parts of a row over its own
// sqrt(mean(v^2) + eps), times w, in the compute dtype.  y float [M, n]; z in the compute dtype, row pitch z_ld.
// One block per (row, part).
template <typename T, int VEC, int IT>
__global__ void gate_group_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, long long z_ld, SmallVec w,
                                       T* __restrict__ out, int n, int part, float eps) {
  pdl_begin();
  __shared__ float red[33];
  const size_t m = blockIdx.x;
  const int p0 = blockIdx.y * part;
  const float* yr = y + m * n + p0;
  const T* zr = z + m * z_ld + p0;
  float v[IT][VEC];
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = (threadIdx.x + it * blockDim.x) * VEC;
    if (i < part) {
      float yv[VEC], zv[VEC];
      if constexpr (VEC == 4) {
        const float4 a = *reinterpret_cast<const float4*>(yr + i);
        yv[0] = a.x; yv[1] = a.y; yv[2] = a.z; yv[3] = a.w;
        if constexpr (sizeof(T) == 2) {
          const uint2 q = *reinterpret_cast<const uint2*>(zr + i);
          zv[0] = __uint_as_float(q.x << 16); zv[1] = __uint_as_float(q.x & 0xffff0000u);
          zv[2] = __uint_as_float(q.y << 16); zv[3] = __uint_as_float(q.y & 0xffff0000u);
        } else {
          const float4 q = *reinterpret_cast<const float4*>(zr + i);
          zv[0] = q.x; zv[1] = q.y; zv[2] = q.z; zv[3] = q.w;
        }
      } else {
        yv[0] = yr[i];
        zv[0] = to_f<T>(zr[i]);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        v[it][e] = yv[e] * (zv[e] / (1.f + expf(-zv[e])));
        ss = fmaf(v[it][e], v[it][e], ss);
      }
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[it][e] = 0.f;
    }
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)part + eps);
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = (threadIdx.x + it * blockDim.x) * VEC;
    if (i < part) {
      T* o = out + m * n + p0 + i;
      if constexpr (VEC == 4)
        store4<T>(o, v[it][0] * inv * w[p0 + i], v[it][1] * inv * w[p0 + i + 1], v[it][2] * inv * w[p0 + i + 2],
                  v[it][3] * inv * w[p0 + i + 3]);
      else
        *o = from_f<T>(v[it][0] * inv * w[p0 + i]);
    }
  }
}

SNK_API int snk_gate_group_norm(const float* y, const void* z, long long z_ld, const void* w, int w_f32, void* out, int M,
                                int n, int groups, float eps, int dtype, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (n <= 0 || groups <= 0 || groups > 65535 || n % groups) return SNK_ERR_SIZE;
  const int part = n / groups;
  const uintptr_t tv = dtype == SNK_F32 ? 16 : 8;
  const bool vec = part % 4 == 0 && z_ld % 4 == 0 && (uintptr_t)y % 16 == 0 && ((uintptr_t)z | (uintptr_t)out) % tv == 0;
  const int items = vec ? part / 4 : part;
  if (items > 1024 * 8) return SNK_ERR_SIZE;
  SmallVec wv{w, w_f32};
#define GG_LAUNCH(VEC_, IT_, THREADS_)                                                                         \
  snk_launch(gate_group_norm_kernel<T, VEC_, IT_>, dim3(M, groups), dim3(THREADS_), 0, stream, y,              \
             static_cast<const T*>(z), z_ld, wv, static_cast<T*>(out), n, part, eps)
#define GG_SIZES(VEC_)                                                                                         \
  do {                                                                                                         \
    if (items <= 64) GG_LAUNCH(VEC_, 1, 64);                                                                   \
    else if (items <= 256) GG_LAUNCH(VEC_, 1, 256);                                                            \
    else if (items <= 1024) GG_LAUNCH(VEC_, 4, 256);                                                           \
    else if (items <= 2048) GG_LAUNCH(VEC_, 4, 512);                                                           \
    else GG_LAUNCH(VEC_, 8, 1024);                                                                             \
  } while (0)
  SNK_DISPATCH(dtype, {
    if (vec) GG_SIZES(4);
    else GG_SIZES(1);
  });
#undef GG_SIZES
#undef GG_LAUNCH
  SNK_LAUNCH_CHECK();
  return 0;
}
