// The seam between two sublayers of a layer with a norm on both sides of each sublayer: one kernel takes the
// residual row from a sublayer's raw output to the next sublayer's normalised input.
//
//   d  = y * sigmoid(g + b)            y: a float row, or routed experts' rows still in pieces (a piece without a
//                                      row of its own, place -1, stands for the sublayer's input row h);
//                                      g: the gate's logits per element in the compute dtype, b a float bias
//   x += d / rms(d) * w1               the norm on the sublayer's output
//   X_n = x;  x = sum_j a[j] X_j       (where a depth average is asked for) the layers' results X_0 .. X_n of the
//                                      step lie in `history` [n + 1, M, W]; this row's X_n is stored there
//   out = x / rms(x) * w2              the norm before the next sublayer, in the compute dtype
//
// Every step is optional (no y: the row is only recorded and normalised).  With `rows` only those rows come out
// and neither the residual nor the history is written (the model's last norm on the rows whose logits are wanted).
// Sums, statistics, gates and the residual are float.  A block takes one row and keeps it in registers; its size
// depends on W alone and, through one threshold, on the number of rows (the order of a row's sums with it).
#include "common.cuh"

#define SW_MANY_ROWS 160       // from here on rows fill the SMs: blocks with fewer registers, more of them on an SM

template <typename T> struct SwRaw;                       // four elements of the compute dtype
template <> struct SwRaw<float> {
  static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
};
template <> struct SwRaw<bf16> {
  static __device__ __forceinline__ float4 load(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                       __uint_as_float(u.y & 0xffff0000u));
  }
};

template <typename T, int VEC>
__device__ __forceinline__ void sw_load(const T* __restrict__ p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 t = SwRaw<T>::load(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else {
    v[0] = to_f<T>(*p);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void sw_store(T* __restrict__ p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) store4<T>(p, v[0], v[1], v[2], v[3]);
  else *p = from_f<T>(v[0]);
}

struct SandwichArgs {
  float* residual;
  const float* y;                 // float rows [M, W], or the experts' rows when pair_pos is given; null: no sublayer
  const int* pair_pos;            // [M, k] row of each pick, -1: the row h itself
  const float* pair_w;            // [M, k]
  int k;
  const void* h;                  // [M, W] compute dtype; null where no place is -1
  const void* gate;               // compute dtype, row pitch gate_ld; null: no gate
  long long gate_ld;
  const float* gate_bias;         // [W]
  const float* w1;                // [W], null: no norm on the output
  float eps1;
  float* history;                 // null: nothing kept
  long long history_step;         // elements from one entry to the next
  int n;                          // number of this row's entry
  const float* avg;               // [n + 1], null: no average
  const float* w2;                // [W]
  float eps2;
  const int* rows;
  int W;
};

// EARLY: for the few rows of a decode step, where a row's latency counts and not how many rows an SM holds.
template <typename T, int VEC, int IT, bool EARLY>
__global__ void __launch_bounds__(VEC == 4 ? 512 : 1024)
sandwich_norm_kernel(const SandwichArgs a, T* __restrict__ out) {
  pdl_begin();
  __shared__ float red[33];
  const int W = a.W;
  const size_t m = a.rows ? (size_t)a.rows[blockIdx.x] : (size_t)blockIdx.x;
  const int step = blockDim.x * VEC;
  float x[IT][VEC];
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = threadIdx.x * VEC + it * step;
    if (i < W) {
      sw_load<float, VEC>(a.residual + m * W + i, x[it]);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[it][e] = 0.f;
    }
  }
  float old[IT][VEC];                                      // the earlier layers' share of the average
#pragma unroll
  for (int it = 0; it < IT; ++it)
#pragma unroll
    for (int e = 0; e < VEC; ++e) old[it][e] = 0.f;
  auto earlier_layers = [&] {
    constexpr int JU = EARLY ? 8 : 4;                      // entries whose loads are in flight together
#pragma unroll JU
    for (int j = 0; j < a.n; ++j) {
      const float w = a.avg[j];
      const float* hx = a.history + (size_t)j * a.history_step + m * W;
#pragma unroll
      for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * VEC + it * step;
        if (i < W) {
          float t[VEC];
          sw_load<float, VEC>(hx + i, t);
#pragma unroll
          for (int e = 0; e < VEC; ++e) old[it][e] = fmaf(w, t[e], old[it][e]);
        }
      }
    }
  };
  // EARLY: the loads that depend on nothing go out before the sublayer's rows are looked up
  float g[EARLY ? IT : 1][VEC], gb[EARLY ? IT : 1][VEC], w1[EARLY ? IT : 1][VEC], w2[EARLY ? IT : 1][VEC];
  if constexpr (EARLY) {
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = threadIdx.x * VEC + it * step;
#pragma unroll
      for (int e = 0; e < VEC; ++e) g[it][e] = gb[it][e] = w1[it][e] = w2[it][e] = 0.f;
      if (i < W) {
        if (a.y && a.gate) {
          sw_load<T, VEC>(static_cast<const T*>(a.gate) + m * a.gate_ld + i, g[it]);
          sw_load<float, VEC>(a.gate_bias + i, gb[it]);
        }
        if (a.y && a.w1) sw_load<float, VEC>(a.w1 + i, w1[it]);
        sw_load<float, VEC>(a.w2 + i, w2[it]);
      }
    }
    if (a.avg) earlier_layers();
  }
  if (a.y) {
    float d[IT][VEC];
    if (a.pair_pos) {
#pragma unroll
      for (int it = 0; it < IT; ++it)
#pragma unroll
        for (int e = 0; e < VEC; ++e) d[it][e] = 0.f;
      float own = 0.f;                                    // the weight of the picks that stand for h itself
#pragma unroll 4
      for (int j = 0; j < a.k; ++j) {
        const int at = a.pair_pos[m * a.k + j];
        const float w = a.pair_w[m * a.k + j];
        if (at < 0) {
          own += w;
          continue;
        }
        const float* yr = a.y + (size_t)at * W;
#pragma unroll
        for (int it = 0; it < IT; ++it) {
          const int i = threadIdx.x * VEC + it * step;
          if (i < W) {
            float t[VEC];
            sw_load<float, VEC>(yr + i, t);
#pragma unroll
            for (int e = 0; e < VEC; ++e) d[it][e] = fmaf(w, t[e], d[it][e]);
          }
        }
      }
      if (own != 0.f && a.h) {
        const T* hr = static_cast<const T*>(a.h) + m * W;
#pragma unroll
        for (int it = 0; it < IT; ++it) {
          const int i = threadIdx.x * VEC + it * step;
          if (i < W) {
            float t[VEC];
            sw_load<T, VEC>(hr + i, t);
#pragma unroll
            for (int e = 0; e < VEC; ++e) d[it][e] = fmaf(own, t[e], d[it][e]);
          }
        }
      }
    } else {
#pragma unroll
      for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * VEC + it * step;
        if (i < W) {
          sw_load<float, VEC>(a.y + m * W + i, d[it]);
        } else {
#pragma unroll
          for (int e = 0; e < VEC; ++e) d[it][e] = 0.f;
        }
      }
    }
    if (a.gate) {
      const T* gr = static_cast<const T*>(a.gate) + m * a.gate_ld;
#pragma unroll
      for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * VEC + it * step;
        if constexpr (EARLY) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) d[it][e] /= 1.f + expf(-(g[it][e] + gb[it][e]));
        } else if (i < W) {
          float z[VEC], b[VEC];
          sw_load<T, VEC>(gr + i, z);
          sw_load<float, VEC>(a.gate_bias + i, b);
#pragma unroll
          for (int e = 0; e < VEC; ++e) d[it][e] /= 1.f + expf(-(z[e] + b[e]));
        }
      }
    }
    if (a.w1) {
      float ss = 0.f;
#pragma unroll
      for (int it = 0; it < IT; ++it)
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(d[it][e], d[it][e], ss);
      ss = block_sum(ss, red);
      const float inv = 1.f / sqrtf(ss / (float)W + a.eps1);
#pragma unroll
      for (int it = 0; it < IT; ++it) {
        const int i = threadIdx.x * VEC + it * step;
        if constexpr (EARLY) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) x[it][e] = fmaf(d[it][e] * inv, w1[it][e], x[it][e]);
        } else if (i < W) {
          float w[VEC];
          sw_load<float, VEC>(a.w1 + i, w);
#pragma unroll
          for (int e = 0; e < VEC; ++e) x[it][e] = fmaf(d[it][e] * inv, w[e], x[it][e]);
        }
      }
    } else {
#pragma unroll
      for (int it = 0; it < IT; ++it)
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[it][e] += d[it][e];
    }
  }
  if (a.history && !a.rows) {
    float* hx = a.history + (size_t)a.n * a.history_step + m * W;
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = threadIdx.x * VEC + it * step;
      if (i < W) sw_store<float, VEC>(hx + i, x[it]);
    }
  }
  if (a.avg) {
    if constexpr (!EARLY) earlier_layers();
    const float last = a.avg[a.n];
#pragma unroll
    for (int it = 0; it < IT; ++it)
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[it][e] = fmaf(last, x[it][e], old[it][e]);
  }
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = threadIdx.x * VEC + it * step;
    if (i < W) {
      if ((a.y || a.avg) && !a.rows) sw_store<float, VEC>(a.residual + m * W + i, x[it]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(x[it][e], x[it][e], ss);
    }
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)W + a.eps2);
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = threadIdx.x * VEC + it * step;
    if (i < W) {
      float w[VEC], o[VEC];
      if constexpr (!EARLY) sw_load<float, VEC>(a.w2 + i, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) o[e] = x[it][e] * inv * (EARLY ? w2[it][e] : w[e]);
      sw_store<T, VEC>(out + (size_t)blockIdx.x * W + i, o);
    }
  }
}

SNK_API int snk_sandwich_norm(float* residual, const float* y, const int* pair_pos, const float* pair_w, int k,
                              const void* h, const void* gate, long long gate_ld, const float* gate_bias,
                              const float* w1, float eps1, float* history, long long history_step, int n,
                              const float* avg, const float* w2, float eps2, void* out, const int* rows, int R, int W,
                              int dtype, cudaStream_t stream) {
  if (R <= 0) return 0;
  if (W <= 0 || W > 16384 || !residual || !w2 || (pair_pos && (k <= 0 || !pair_w || !y))) return SNK_ERR_SIZE;
  if ((gate && !gate_bias) || (avg && !history) || n < 0) return SNK_ERR_SIZE;
  const SandwichArgs args{residual, y, pair_pos, pair_w, k, h, gate, gate_ld, gate_bias, w1, eps1, history,
                          history_step, n, avg, w2, eps2, rows, W};
  const uintptr_t tv = dtype == SNK_F32 ? 16 : 8;         // four elements of the compute dtype
  const bool vec = W % 4 == 0 && gate_ld % 4 == 0 && history_step % 4 == 0 &&
                   ((uintptr_t)residual | (uintptr_t)y | (uintptr_t)gate_bias | (uintptr_t)w1 | (uintptr_t)history |
                    (uintptr_t)w2) % 16 == 0 &&
                   ((uintptr_t)h | (uintptr_t)gate | (uintptr_t)out) % tv == 0;
#define SW_LAUNCH_(VEC_, IT_, EARLY_, THREADS_)                                                               \
  snk_launch(sandwich_norm_kernel<T, VEC_, IT_, EARLY_>, dim3(R), dim3(THREADS_), 0, stream, args, static_cast<T*>(out))
#define SW_LAUNCH(VEC_, IT_, THREADS_) SW_LAUNCH_(VEC_, IT_, false, THREADS_)
  SNK_DISPATCH(dtype, {
    if (vec) {
      const int n4 = W / 4;
      if (R < SW_MANY_ROWS && n4 <= 1024) {
        if (n4 <= 64) SW_LAUNCH_(4, 1, true, 64);
        else if (n4 <= 256) SW_LAUNCH_(4, 1, true, 256);
        else if (n4 <= 512) SW_LAUNCH_(4, 1, true, 512);
        else SW_LAUNCH_(4, 2, true, 512);
      } else if (n4 <= 64) SW_LAUNCH(4, 1, 64);
      else if (n4 <= 256) SW_LAUNCH(4, 1, 256);
      else if (n4 <= 512) SW_LAUNCH(4, 2, 256);
      else if (n4 <= 1024) SW_LAUNCH(4, 4, 256);
      else if (n4 <= 2048) SW_LAUNCH(4, 4, 512);
      else SW_LAUNCH(4, 8, 512);
    } else {
      if (W <= 256) SW_LAUNCH(1, 1, 256);
      else if (W <= 1024) SW_LAUNCH(1, 4, 256);
      else if (W <= 4096) SW_LAUNCH(1, 4, 1024);
      else SW_LAUNCH(1, 16, 1024);
    }
  });
#undef SW_LAUNCH
#undef SW_LAUNCH_
  SNK_LAUNCH_CHECK();
  return 0;
}
