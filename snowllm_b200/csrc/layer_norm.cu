// Layer norm fused with the residual sum that precedes it, and the gate of a layer's side input from the token ids.
//
//   d   = ca * a + cb * b  (+ the routed experts' weighted rows, still in pieces)     every term optional
//   d   = d / rms(d) * w1                                                             where the update has a norm
//   x  += d
//   out = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w2 * gain                     in the compute dtype; without
//         w2: x itself in the compute dtype (what a product on the raw stream reads)
//
// With `rows` only those rows come out and the residual is not written (a model's last norm on the rows whose logits
// are wanted).  Sums, statistics and the residual are float.  A block keeps one row in registers; its size depends on W
// and, through one threshold, on the number of rows (the order of a row's sums with it).
#include "common.cuh"

#define LN_MANY_ROWS 160       // from here on rows fill the SMs: blocks with fewer registers, more of them on an SM

struct LayerNormArgs {
  float* residual;
  const float* a;                 // [M, W], null: no such term
  const float* b;
  float ca, cb;
  const float* y;                 // the experts' rows, null: none
  const int* pair_pos;            // [M, k]
  const float* pair_w;            // [M, k]
  int k;
  const float* w1;                // [W], null: the update has no norm
  float eps1;
  const float* w2;                // [W], null: no norm, the sum itself comes out
  float eps2, gain;
  const int* rows;
  int W;
};

template <int VEC>
__device__ __forceinline__ void ln_load(const float* __restrict__ p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else {
    v[0] = *p;
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void ln_store(T* __restrict__ p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) store4<T>(p, v[0], v[1], v[2], v[3]);
  else *p = from_f<T>(v[0]);
}

// EARLY: for the few rows of a decode step, where a row's latency counts: every load that depends on nothing goes out
// ahead.
template <typename T, int VEC, int IT, bool EARLY>
__global__ void __launch_bounds__(VEC == 4 ? 512 : 1024) layer_norm_kernel(const LayerNormArgs p, T* __restrict__ out) {
  __shared__ float red[33];
  const int W = p.W;
  const int step = blockDim.x * VEC;
  float w1[EARLY ? IT : 1][VEC], w2[EARLY ? IT : 1][VEC];
  if constexpr (EARLY) {                                   // weights are constants: they need not wait for the kernel before
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = threadIdx.x * VEC + it * step;
#pragma unroll
      for (int e = 0; e < VEC; ++e) w1[it][e] = w2[it][e] = 0.f;
      if (i < W) {
        if (p.w1) ln_load<VEC>(p.w1 + i, w1[it]);
        if (p.w2) ln_load<VEC>(p.w2 + i, w2[it]);
      }
    }
  }
  pdl_begin();
  const size_t m = p.rows ? (size_t)p.rows[blockIdx.x] : (size_t)blockIdx.x;
  float x[IT][VEC], d[IT][VEC];
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = threadIdx.x * VEC + it * step;
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[it][e] = d[it][e] = 0.f;
    if (i < W) {
      ln_load<VEC>(p.residual + m * W + i, x[it]);
      float t[VEC];
      if (p.a) {
        ln_load<VEC>(p.a + m * W + i, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) d[it][e] = p.ca * t[e];
      }
      if (p.b) {
        ln_load<VEC>(p.b + m * W + i, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) d[it][e] = fmaf(p.cb, t[e], d[it][e]);
      }
    }
  }
  if (p.y) {
#pragma unroll 4
    for (int j = 0; j < p.k; ++j) {
      const float w = p.pair_w[m * p.k + j];
      const float* yr = p.y + (size_t)p.pair_pos[m * p.k + j] * W;
#pragma unroll
      for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * VEC + it * step;
        if (i < W) {
          float t[VEC];
          ln_load<VEC>(yr + i, t);
#pragma unroll
          for (int e = 0; e < VEC; ++e) d[it][e] = fmaf(w, t[e], d[it][e]);
        }
      }
    }
  }
  if (p.w1) {
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < IT; ++it)
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(d[it][e], d[it][e], ss);
    ss = block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)W + p.eps1);
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = threadIdx.x * VEC + it * step;
      if (i < W) {
        float w[VEC];
        if constexpr (EARLY) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) w[e] = w1[it][e];
        } else {
          ln_load<VEC>(p.w1 + i, w);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) d[it][e] = d[it][e] * inv * w[e];
      }
    }
  }
  const bool changed = p.a || p.b || p.y;
  float sum = 0.f;
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = threadIdx.x * VEC + it * step;
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      x[it][e] += d[it][e];
      sum += x[it][e];
    }
    if (changed && !p.rows && i < W) ln_store<float, VEC>(p.residual + m * W + i, x[it]);
  }
  float mean = 0.f, inv = 1.f;
  if (p.w2) {
    mean = block_sum(sum, red) / (float)W;
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = threadIdx.x * VEC + it * step;
      if (i < W) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          x[it][e] -= mean;
          ss = fmaf(x[it][e], x[it][e], ss);
        }
      }
    }
    ss = block_sum(ss, red);
    inv = p.gain / sqrtf(ss / (float)W + p.eps2);
  }
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = threadIdx.x * VEC + it * step;
    if (i < W) {
      float o[VEC];
      if (p.w2) {
        float w[VEC];
        if constexpr (EARLY) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) w[e] = w2[it][e];
        } else {
          ln_load<VEC>(p.w2 + i, w);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = x[it][e] * inv * w[e];
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = x[it][e];
      }
      ln_store<T, VEC>(out + (size_t)blockIdx.x * W + i, o);
    }
  }
}

SNK_API int snk_layer_norm(float* residual, const float* a, const float* b, float ca, float cb, const float* y,
                           const int* pair_pos, const float* pair_w, int k, const float* w1, float eps1, const float* w2,
                           float eps2, float gain, void* out, const int* rows, int R, int W, int dtype,
                           cudaStream_t stream) {
  if (R <= 0) return 0;
  if (W <= 0 || W > 16384 || !residual || !out || (y && (k <= 0 || !pair_pos || !pair_w)) || (w1 && !(a || b || y)))
    return SNK_ERR_SIZE;
  const LayerNormArgs args{residual, a, b, ca, cb, y, pair_pos, pair_w, k, w1, eps1, w2, eps2, gain, rows, W};
  const uintptr_t tv = dtype == SNK_F32 ? 16 : 8;          // four elements of the compute dtype
  const bool vec = W % 4 == 0 && (uintptr_t)out % tv == 0 &&
                   ((uintptr_t)residual | (uintptr_t)a | (uintptr_t)b | (uintptr_t)y | (uintptr_t)w1 | (uintptr_t)w2) % 16 == 0;
#define LN_LAUNCH_(VEC_, IT_, EARLY_, THREADS_)                                                               \
  snk_launch(layer_norm_kernel<T, VEC_, IT_, EARLY_>, dim3(R), dim3(THREADS_), 0, stream, args, static_cast<T*>(out))
#define LN_LAUNCH(VEC_, IT_, THREADS_) LN_LAUNCH_(VEC_, IT_, false, THREADS_)
  SNK_DISPATCH(dtype, {
    if (vec) {
      const int n4 = W / 4;
      if (R < LN_MANY_ROWS && n4 <= 1024) {
        if (n4 <= 64) LN_LAUNCH_(4, 1, true, 64);
        else if (n4 <= 256) LN_LAUNCH_(4, 1, true, 256);
        else if (n4 <= 512) LN_LAUNCH_(4, 1, true, 512);
        else LN_LAUNCH_(4, 2, true, 512);
      } else if (n4 <= 64) LN_LAUNCH(4, 1, 64);
      else if (n4 <= 256) LN_LAUNCH(4, 1, 256);
      else if (n4 <= 512) LN_LAUNCH(4, 2, 256);
      else if (n4 <= 1024) LN_LAUNCH(4, 4, 256);
      else if (n4 <= 2048) LN_LAUNCH(4, 4, 512);
      else LN_LAUNCH(4, 8, 512);
    } else {
      if (W <= 256) LN_LAUNCH(1, 1, 256);
      else if (W <= 1024) LN_LAUNCH(1, 4, 256);
      else if (W <= 4096) LN_LAUNCH(1, 4, 1024);
      else LN_LAUNCH(1, 16, 1024);
    }
  });
#undef LN_LAUNCH
#undef LN_LAUNCH_
  SNK_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------------------------
// out[m, j] = gelu(g[m, j]) * table[token(m), off + j], gelu in its tanh form, j < n.  g float; table in the compute
// dtype, row pitch ld.  A negative id -(i + 1) stands for pending[i], a token the host has not read yet.
template <typename T>
__global__ void side_gate_kernel(const float* __restrict__ g, const T* __restrict__ table, long long ld, int off,
                                 const int* __restrict__ ids, const int* __restrict__ pending, int num_pending,
                                 T* __restrict__ out, long long total, int n, int V) {
  pdl_begin();
  const long long stride = (long long)gridDim.x * blockDim.x;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) {
    const long long m = i / n;
    const int j = (int)(i - m * n);
    int id = ids[m];
    if (id < 0 && pending != nullptr && -(id + 1) < num_pending) id = pending[-(id + 1)];
    const bool ok = id >= 0 && id < V;                     // the host checks ids; a bad one reads nothing
    const float e = ok ? to_f<T>(table[(size_t)id * ld + off + j]) : 0.f;
    const float z = g[i];
    out[i] = from_f<T>(0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))) * e);
  }
}

SNK_API int snk_side_gate(const float* g, const void* table, long long ld, int off, const int* ids, const int* pending,
                          int num_pending, void* out, int M, int n, int V, int dtype, cudaStream_t stream) {
  if (M <= 0 || n <= 0) return 0;
  if (off < 0 || ld < off + n || V <= 0) return SNK_ERR_SIZE;
  const long long total = (long long)M * n;
  const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  SNK_DISPATCH(dtype, snk_launch(side_gate_kernel<T>, dim3(blocks), dim3(256), 0, stream, g,
                                 static_cast<const T*>(table), ld, off, ids, pending, num_pending, static_cast<T*>(out),
                                 total, n, V));
  SNK_LAUNCH_CHECK();
  return 0;
}
