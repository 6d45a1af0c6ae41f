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
//
// Chunks (bfloat16 rows, steps with long segments): the same recurrence in its chunked form on the tensor cores.  With
// c_t = sum of the log decays up to t inside a chunk of 64 tokens,
//   y_t = exp(c_t) C_t S_in + sum_(s <= t) exp(c_t - c_s) step_s (C_t . B_s) x_s + D x_t
//   S_out = exp(c_end) S_in + sum_s exp(c_end - c_s) step_s B_s x_s^T
// A block serves one (segment, head, 32 columns of P) and walks the segment's chunks in order, S in the accumulators of
// mma.sync m16n8k16 (N up to 128).  x, B and C are bfloat16 as they come, so C B^T is exact in float; every float factor (S, the
// masked weights, the weighted x) goes in as three bfloat16 terms that add up to its 24 bits, so the sums are 32-bit
// sums in another order.  c_t is summed in double and kept as two floats: the difference of two of them is exact to
// float however long the chunk's decay is.
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

// ---------------------------------------------------------------------------------------------
#define SC_Q 64                // tokens per chunk
#define SC_COLS 32             // columns of P per block
#define SC_WORKERS 512         // threads of the sixteen warps that compute
#define SC_THREADS 544
#define SC_XS (SC_COLS + 8)    // elements per row of x, of the weighted x and of S in shared memory

__device__ __forceinline__ void sc_cp_async16(void* smem, const void* gmem, bool valid) {
  const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
  const int bytes = valid ? 16 : 0;                        // not valid: zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(gmem), "r"(bytes));
}
__device__ __forceinline__ void sc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void sc_ldsm4(uint32_t (&r)[4], const bf16* row) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(row);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void sc_ldsm4_trans(uint32_t (&r)[4], const bf16* row) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(row);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ float sc_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Two floats as three packed pairs of bfloat16: a = t[0].x + t[1].x + t[2].x to float's last bit (so b).
__device__ __forceinline__ void sc_split3(float a, float b, uint32_t (&t)[3]) {
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    t[i] = *reinterpret_cast<const uint32_t*>(&v);
    a -= __uint_as_float(t[i] << 16);
    b -= __uint_as_float(t[i] & 0xffff0000u);
  }
}

// Warps 0..7 form the chunk's y, 16 rows and 16 columns each; warps 8..15 hold S and take it to the next chunk; warp 16
// works out the next chunk's steps and decays.  The three work at the same time: y of chunk k reads S as it was before
// the chunk (three bfloat16 terms in shared memory, two buffers), while S moves past the chunk and its terms go into the
// other buffer.  One block-wide barrier per chunk.
// NT: 16-row tiles of S, rounded up to a power of two (N <= 16 NT).  EXACT: N is 16 NT, every address a constant away.
template <int NT, bool EXACT>
__global__ void __launch_bounds__(SC_THREADS)
state_space_chunk_kernel(const bf16* __restrict__ u, long long u_ld, int x_off, int b_off, int c_off,
                         const void* __restrict__ dt, int dt_f32, long long dt_ld, const float* __restrict__ dt_bias,
                         const float* __restrict__ rate, const float* __restrict__ skip,
                         const int* __restrict__ cu_seqlens, const int* __restrict__ seg_start,
                         const int* __restrict__ seg_slot, float* __restrict__ state, float* __restrict__ out, int H,
                         int G, int N_, int P) {
  pdl_begin();
  const int N = EXACT ? 16 * NT : N_;
  extern __shared__ __align__(16) unsigned char sc_raw[];
  // of a chunk: c_t (two floats), step_t, exp(c_end)
  __shared__ __align__(8) float s_hi[2][SC_Q], s_lo[2][SC_Q], s_step[2][SC_Q];
  __shared__ float s_end[2];
  const int NS = N + 8;                                    // elements per row of B and C
  bf16* sm_c = reinterpret_cast<bf16*>(sc_raw);            // [2][SC_Q][NS]
  bf16* sm_b = sm_c + 2 * SC_Q * NS;                       // [2][SC_Q][NS]
  bf16* sm_x = sm_b + 2 * SC_Q * NS;                       // [2][SC_Q][SC_XS]
  bf16* sm_w = sm_x + 2 * SC_Q * SC_XS;                    // [3][SC_Q][SC_XS]  the terms of the weighted x
  bf16* sm_s = sm_w + 3 * SC_Q * SC_XS;                    // [2][3][N][SC_XS]  the terms of S before a chunk
  const int b = blockIdx.x, h = blockIdx.y;
  const int g = h / (H / G);
  const int col0 = blockIdx.z * SC_COLS;
  const int row0 = cu_seqlens[b], row1 = cu_seqlens[b + 1];
  if (row1 <= row0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad = lane >> 2, tq = lane & 3;
  const int n_chunks = (row1 - row0 + SC_Q - 1) / SC_Q;
  const int tiles = N / 16;

  auto load = [&](int k) {                                 // by the threads of warps 0..15
    if (k < n_chunks) {
      const int t0 = row0 + k * SC_Q, nt = min(SC_Q, row1 - t0), buf = k & 1;
      const int nv = N / 8;
      // eight threads a row: B and C in 16-byte vectors, eight at a time; x by half of them
      const int t = threadIdx.x >> 3, c0 = threadIdx.x & 7;
      const bool live = t < nt;
      const bf16* row = u + (size_t)(t0 + (live ? t : 0)) * u_ld;
      const bf16 *gb = row + b_off + (size_t)g * N, *gc = row + c_off + (size_t)g * N;
      bf16 *db = sm_b + (buf * SC_Q + t) * NS, *dc = sm_c + (buf * SC_Q + t) * NS;
#pragma unroll
      for (int i = 0; i < (2 * NT + 7) / 8; ++i) {
        const int c = c0 + 8 * i;
        if (c < nv) {
          sc_cp_async16(db + c * 8, gb + c * 8, live);
          sc_cp_async16(dc + c * 8, gc + c * 8, live);
        }
      }
      if (c0 < SC_COLS / 8) {
        const bool ok = live && col0 + c0 * 8 < P;
        sc_cp_async16(sm_x + (buf * SC_Q + t) * SC_XS + c0 * 8, row + x_off + (size_t)h * P + (ok ? col0 + c0 * 8 : 0), ok);
      }
    }
    asm volatile("cp.async.commit_group;");
  };

  if (warp == SC_WORKERS / 32) {
    // steps and summed log decays (as powers of two), two tokens a lane, a chunk ahead of the others; the raw values of
    // the chunk after that are on their way meanwhile
    const float my_bias = dt_bias[h];
    const double rate2 = (double)rate[h] * 1.4426950408889634;
    auto raw = [&](int k, int i) {
      const int t = row0 + k * SC_Q + 2 * lane + i;
      if (t >= row1) return 0.f;
      const size_t at = (size_t)t * dt_ld + h;
      return dt_f32 ? static_cast<const float*>(dt)[at] : __bfloat162float(static_cast<const bf16*>(dt)[at]);
    };
    float z0 = raw(0, 0), z1 = raw(0, 1);
    for (int k = 0; k <= n_chunks; ++k) {                  // chunk k's values, before the barrier that opens chunk k
      if (k < n_chunks) {
        const int buf = k & 1, t = row0 + k * SC_Q + 2 * lane;
        const float step0 = t < row1 ? ss_softplus(z0 + my_bias) : 0.f, step1 = t + 1 < row1 ? ss_softplus(z1 + my_bias) : 0.f;
        z0 = raw(k + 1, 0);
        z1 = raw(k + 1, 1);
        const double d0 = rate2 * (double)step0, pair = d0 + rate2 * (double)step1;
        double run = pair;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const double other = __shfl_up_sync(0xffffffffu, run, o);
          if (lane >= o) run += other;
        }
        const double c0 = run - pair + d0;
        const float hi0 = (float)c0, hi1 = (float)run;
        *reinterpret_cast<float2*>(&s_hi[buf][2 * lane]) = make_float2(hi0, hi1);
        *reinterpret_cast<float2*>(&s_lo[buf][2 * lane]) = make_float2((float)(c0 - (double)hi0), (float)(run - (double)hi1));
        *reinterpret_cast<float2*>(&s_step[buf][2 * lane]) = make_float2(step0, step1);
        if (lane == 31) s_end[buf] = sc_exp2(hi1);
      }
      __syncthreads();
    }
    return;
  }
  load(0);

  if (warp >= 8) {
    // S: warp w of these holds 16-row tile w % tiles, all of the block's columns or a share of them
    const int w = warp - 8;
    const int shares = tiles <= 2 ? 4 : (tiles <= 4 ? 2 : 1);      // warps that share a tile's columns
    const int tile = w % tiles, share = w / tiles;
    const int nt_first = share * (4 / shares), nt_count = share < shares ? 4 / shares : 0;   // (past the last share: none)
    const bool fresh = seg_start[b] == 0;
    float* slot = state + ((size_t)seg_slot[b] * H + h) * N * P + (size_t)(tile * 16 + quad) * P + col0 + nt_first * 8 + tq * 2;
    float S[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float2 v = make_float2(0.f, 0.f);
        if (!fresh && j < nt_count && col0 + (nt_first + j) * 8 + tq * 2 < P)
          v = *reinterpret_cast<const float2*>(slot + (size_t)8 * r * P + j * 8);
        S[j][2 * r] = v.x;
        S[j][2 * r + 1] = v.y;
      }
    auto put = [&](int buf) {                              // the terms of S
      bf16* at = sm_s + ((size_t)buf * 3 * N + tile * 16 + quad) * SC_XS + nt_first * 8 + tq * 2;
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j < nt_count)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            uint32_t term[3];
            sc_split3(S[j][2 * r], S[j][2 * r + 1], term);
#pragma unroll
            for (int q = 0; q < 3; ++q) *reinterpret_cast<uint32_t*>(at + (q * N + 8 * r) * SC_XS + j * 8) = term[q];
          }
    };
    put(0);
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();                                       // opens chunk 0
    for (int k = 0; k < n_chunks; ++k) {
      const int buf = k & 1;
      load(k + 1);
      const bf16* bb = sm_b + buf * SC_Q * NS;
      {
        // x weighted by exp(c_end - c_s) step_s, eight columns a thread; c_end is the last token's
        const int i = threadIdx.x - 256, t = i >> 2, c = (i & 3) * 8;
        const float wt = s_step[buf][t] * sc_exp2((s_hi[buf][SC_Q - 1] - s_hi[buf][t]) + (s_lo[buf][SC_Q - 1] - s_lo[buf][t]));
        const uint4 raw = *reinterpret_cast<const uint4*>(sm_x + (buf * SC_Q + t) * SC_XS + c);
        const uint32_t xr[4] = {raw.x, raw.y, raw.z, raw.w};
        uint32_t term[4][3];
#pragma unroll
        for (int e = 0; e < 4; ++e)
          sc_split3(wt * __uint_as_float(xr[e] << 16), wt * __uint_as_float(xr[e] & 0xffff0000u), term[e]);
#pragma unroll
        for (int q = 0; q < 3; ++q)
          *reinterpret_cast<uint4*>(sm_w + (q * SC_Q + t) * SC_XS + c) = make_uint4(term[0][q], term[1][q], term[2][q], term[3][q]);
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");       // among these eight warps
      const float end = s_end[buf];
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[j][e] *= end;
      if (nt_count > 0) {
#pragma unroll
        for (int kk = 0; kk < SC_Q / 16; ++kk) {           // (rows past the segment's end are zeros)
          uint32_t a[4];
          // B as it lies, token by token, read transposed: lane L reads token (L / 16) * 8 + L % 8, columns (L / 8 % 2) * 8
          sc_ldsm4_trans(a, bb + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * NS + tile * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
          for (int q = 0; q < 3; ++q) {
            const bf16* w_row = sm_w + (q * SC_Q + kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * SC_XS + (lane >> 4) * 8;
            if (nt_count == 1) {
              uint32_t f[4];
              sc_ldsm4_trans(f, w_row + (nt_first & ~1) * 8);
              if (nt_first & 1) sc_mma(S[0], a, f[2], f[3]);
              else sc_mma(S[0], a, f[0], f[1]);
            } else {
#pragma unroll
              for (int j = 0; j < 4; j += 2)
                if (j < nt_count) {
                  uint32_t f[4];
                  sc_ldsm4_trans(f, w_row + (nt_first + j) * 8);
                  sc_mma(S[j], a, f[0], f[1]);
                  sc_mma(S[j + 1], a, f[2], f[3]);
                }
            }
          }
        }
      }
      put(buf ^ 1);
      asm volatile("cp.async.wait_group 0;");
      __syncthreads();                                     // opens chunk k + 1
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (j < nt_count && col0 + (nt_first + j) * 8 + tq * 2 < P)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          *reinterpret_cast<float2*>(slot + (size_t)8 * r * P + j * 8) = make_float2(S[j][2 * r], S[j][2 * r + 1]);
    return;
  }

  // y: rows 16 yi .. of the chunk, so dealt that the warps of one scheduler have equal work under the causal triangle,
  // columns 16 yh ..
  const int yi = warp < 4 ? warp : 7 - warp, yh = warp >> 2;
  const float my_skip = skip[h];
  asm volatile("cp.async.wait_group 0;");
  __syncthreads();                                         // opens chunk 0
  for (int k = 0; k < n_chunks; ++k) {
    const int t0 = row0 + k * SC_Q, nt = min(SC_Q, row1 - t0), buf = k & 1;
    load(k + 1);
    if (yi * 16 < nt) {
      const bf16* bb = sm_b + buf * SC_Q * NS;
      const bf16* xb = sm_x + buf * SC_Q * SC_XS;
      uint32_t ca[NT][4];                                  // this warp's rows of C
      const bf16* c_row = sm_c + (buf * SC_Q + yi * 16 + (lane & 15)) * NS + (lane >> 4) * 8;
#pragma unroll
      for (int kk = 0; kk < NT; ++kk)
        if (EXACT || kk < tiles) sc_ldsm4(ca[kk], c_row + kk * 16);
      float part[3][2][4];                                 // C S_in, term by term
#pragma unroll
      for (int q = 0; q < 3; ++q)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) part[q][j][e] = 0.f;
      const bf16* s_row = sm_s + ((size_t)buf * 3 * N + ((lane >> 3) & 1) * 8 + (lane & 7)) * SC_XS + yh * 16 + (lane >> 4) * 8;
#pragma unroll
      for (int kk = 0; kk < NT; ++kk)
        if (EXACT || kk < tiles) {
#pragma unroll
          for (int q = 0; q < 3; ++q) {
            uint32_t f[4];
            sc_ldsm4_trans(f, s_row + (q * N + kk * 16) * SC_XS);
            sc_mma(part[q][0], ca[kk], f[0], f[1]);
            sc_mma(part[q][1], ca[kk], f[2], f[3]);
          }
        }
      float hi[2], lo[2];                                  // c_t of this thread's two rows
      float acc[2][4];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        hi[r] = s_hi[buf][yi * 16 + quad + 8 * r];
        lo[r] = s_lo[buf][yi * 16 + quad + 8 * r];
        const float f = sc_exp2(hi[r]);
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 2 * r; e < 2 * r + 2; ++e) acc[j][e] = f * ((part[2][j][e] + part[1][j][e]) + part[0][j][e]);
      }
#pragma unroll
      for (int sj = 0; sj < SC_Q / 16; ++sj) {             // 16 tokens s at a time
        if (sj > yi) break;
        float m[2][2][4];                                  // even and odd steps apart: shorter chains
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) m[p][j][e] = 0.f;
        // rows s of B as the columns of the product: lane L reads token (L / 16) * 8 + L % 8, eight elements from
        // (L / 8 % 2) * 8 on
        const bf16* b_row = bb + (sj * 16 + (lane >> 4) * 8 + (lane & 7)) * NS + ((lane >> 3) & 1) * 8;
#pragma unroll
        for (int kk = 0; kk < NT; ++kk)
          if (EXACT || kk < tiles) {
            uint32_t f[4];
            sc_ldsm4(f, b_row + kk * 16);
            sc_mma(m[kk & 1][0], ca[kk], f[0], f[1]);
            sc_mma(m[kk & 1][1], ca[kk], f[2], f[3]);
          }
        uint32_t wa[3][4];                                 // the weights' terms as the rows of the next product
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int s = sj * 16 + j * 8 + tq * 2;
          const float2 sh = *reinterpret_cast<const float2*>(&s_hi[buf][s]), sl = *reinterpret_cast<const float2*>(&s_lo[buf][s]);
          const float2 st = *reinterpret_cast<const float2*>(&s_step[buf][s]);
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int t = yi * 16 + quad + 8 * r;
            float w0 = (m[0][j][2 * r] + m[1][j][2 * r]) * st.x * sc_exp2((hi[r] - sh.x) + (lo[r] - sl.x));
            float w1 = (m[0][j][2 * r + 1] + m[1][j][2 * r + 1]) * st.y * sc_exp2((hi[r] - sh.y) + (lo[r] - sl.y));
            if (s > t) w0 = 0.f;
            if (s + 1 > t) w1 = 0.f;
            uint32_t term[3];
            sc_split3(w0, w1, term);
#pragma unroll
            for (int q = 0; q < 3; ++q) wa[q][2 * j + r] = term[q];
          }
        }
        uint32_t f[4];
        sc_ldsm4_trans(f, xb + (sj * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * SC_XS + yh * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int q = 0; q < 3; ++q) {
          sc_mma(acc[0], wa[q], f[0], f[1]);
          sc_mma(acc[1], wa[q], f[2], f[3]);
        }
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = yi * 16 + quad + 8 * r;
        if (t < nt) {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int c = yh * 16 + j * 8 + tq * 2;
            if (col0 + c < P) {
              const uint32_t x2 = *reinterpret_cast<const uint32_t*>(xb + t * SC_XS + c);
              float2 y;
              y.x = fmaf(my_skip, __uint_as_float(x2 << 16), acc[j][2 * r]);
              y.y = fmaf(my_skip, __uint_as_float(x2 & 0xffff0000u), acc[j][2 * r + 1]);
              *reinterpret_cast<float2*>(out + ((size_t)(t0 + t) * H + h) * P + col0 + c) = y;
            }
          }
        }
      }
    }
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();                                       // opens chunk k + 1
  }
}

#define SC_MIN_LEN 32          // a step whose longest segment is shorter walks token by token

// Whether the chunked kernel takes a step.
static bool sc_ok(int dtype, const void* u, long long u_ld, int x_off, int b_off, int c_off, const void* state, const void* out,
                  int N, int P, int max_len) {
  static int on = -1;                                      // SNOWLLM_B200_STATE_SPACE_MMA=0: never (A/B runs)
  if (on < 0) {
    const char* e = getenv("SNOWLLM_B200_STATE_SPACE_MMA");
    on = !(e && e[0] == '0');
  }
  return on && dtype == SNK_BF16 && max_len >= SC_MIN_LEN && N % 16 == 0 && N <= 128 && P % 8 == 0 && u_ld % 8 == 0 &&
         x_off % 8 == 0 && b_off % 8 == 0 && c_off % 8 == 0 && (uintptr_t)u % 16 == 0 && (uintptr_t)state % 8 == 0 &&
         (uintptr_t)out % 8 == 0;
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
  if (sc_ok(dtype, u, u_ld, x_off, b_off, c_off, state, out, N, P, max_len)) {
    const int cslices = (P + SC_COLS - 1) / SC_COLS;
    if (cslices > 65535) return SNK_ERR_SIZE;
    const size_t csmem = (size_t)(4 * SC_Q * (N + 8) + 5 * SC_Q * SC_XS + 6 * N * SC_XS) * sizeof(bf16);
#define SC_LAUNCH_(NT_, EXACT_)                                                                                \
  do {                                                                                                         \
    auto kernel = state_space_chunk_kernel<NT_, EXACT_>;                                                       \
    if (csmem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)csmem); \
    snk_launch(kernel, dim3(B, H, cslices), dim3(SC_THREADS), csmem, stream,                                   \
               static_cast<const bf16*>(u), u_ld, x_off, b_off, c_off, dt, dt_f32, dt_ld, dt_bias, rate, skip, \
               cu_seqlens, seg_start, seg_slot, state, out, H, G, N, P);                                       \
  } while (0)
#define SC_LAUNCH(NT_)                                                                                         \
  do {                                                                                                         \
    if (N == 16 * NT_) SC_LAUNCH_(NT_, true);                                                                  \
    else SC_LAUNCH_(NT_, false);                                                                               \
  } while (0)
    if (N <= 16) SC_LAUNCH_(1, true);
    else if (N <= 32) SC_LAUNCH(2);
    else if (N <= 64) SC_LAUNCH(4);
    else SC_LAUNCH(8);
#undef SC_LAUNCH
#undef SC_LAUNCH_
    SNK_LAUNCH_CHECK();
    return 0;
  }
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
    else if (items <= 128) GG_LAUNCH(VEC_, 1, 128);                                                            \
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
