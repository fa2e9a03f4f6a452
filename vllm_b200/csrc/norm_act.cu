// RMSNorm / fused residual-add RMSNorm / LayerNorm / gated activations (sm_100a).
//
// Reference ops: csrc/libtorch_stable/layernorm_kernels.cu (rms_norm,
// fused_add_rms_norm), activation_kernels.cu (silu_and_mul, gelu_and_mul, ...).
// Our variants: one CTA per token, 16-byte vector access, the row stays in
// registers between the reduction and the scale pass (single HBM read), fp32 math.
#include "common.cuh"

namespace {

constexpr int MAXV = 4;  // 16B vectors per thread kept in registers

template <typename T, bool ADD, bool GEMMA>
__global__ void __launch_bounds__(1024) rms_norm_kernel(T* __restrict__ out, T* __restrict__ x,
                                                         T* __restrict__ residual, const T* __restrict__ w,
                                                         int H, float eps, int64_t x_stride) {
  constexpr int N = Vec16<T>::N;
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  T* xr = x + row * x_stride;
  T* rr = ADD ? residual + row * (int64_t)H : nullptr;
  T* orow = out + row * (ADD ? x_stride : (int64_t)H);
  const int nvec = H / N;
  Vec16<T> v[MAXV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      v[i] = ld16(xr + vi * N);
      if (ADD) {
        Vec16<T> r = ld16(rr + vi * N);
#pragma unroll
        for (int j = 0; j < N; ++j) v[i].e[j] = from_f32<T>(to_f32(v[i].e[j]) + to_f32(r.e[j]));
        st16(rr + vi * N, v[i]);
      }
#pragma unroll
      for (int j = 0; j < N; ++j) { float f = to_f32(v[i].e[j]); ss += f * f; }
    }
  }
  ss = block_sum(ss, red);
  const float inv = rsqrtf(ss / (float)H + eps);
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      Vec16<T> wv = ld16(w + vi * N), o;
#pragma unroll
      for (int j = 0; j < N; ++j) {
        float g = to_f32(wv.e[j]);
        if (GEMMA) g += 1.f;
        o.e[j] = from_f32<T>(to_f32(v[i].e[j]) * inv * g);
      }
      st16(orow + vi * N, o);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(1024) layer_norm_kernel(T* __restrict__ out, const T* __restrict__ x,
                                                           const T* __restrict__ w, const T* __restrict__ b, int H,
                                                           float eps) {
  constexpr int N = Vec16<T>::N;
  __shared__ float red[32];
  const int64_t row = blockIdx.x;
  const T* xr = x + row * H;
  const int nvec = H / N;
  Vec16<T> v[MAXV];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      v[i] = ld16(xr + vi * N);
#pragma unroll
      for (int j = 0; j < N; ++j) s += to_f32(v[i].e[j]);
    }
  }
  const float mean = block_sum(s, red) / (float)H;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
#pragma unroll
      for (int j = 0; j < N; ++j) { float d = to_f32(v[i].e[j]) - mean; ss += d * d; }
    }
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)H + eps);
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nvec) {
      Vec16<T> wv = ld16(w + vi * N), bv, o;
      if (b) bv = ld16(b + vi * N);
#pragma unroll
      for (int j = 0; j < N; ++j) {
        float y = (to_f32(v[i].e[j]) - mean) * inv * to_f32(wv.e[j]);
        if (b) y += to_f32(bv.e[j]);
        o.e[j] = from_f32<T>(y);
      }
      st16(out + row * H + vi * N, o);
    }
  }
}

enum : int { ACT_SILU = 0, ACT_GELU = 1, ACT_GELU_TANH = 2, ACT_RELU = 3, ACT_GELU_NEW = 4, ACT_GELU_FAST = 5,
             ACT_QUICK_GELU = 6, ACT_RELU2 = 7 };

template <int ACT> VB_DEVICE float act_fn(float x) {
  if (ACT == ACT_SILU) return x / (1.f + __expf(-x));
  if (ACT == ACT_GELU) return 0.5f * x * (1.f + erff(x * 0.70710678118654752f));
  if (ACT == ACT_GELU_TANH || ACT == ACT_GELU_NEW)
    return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
  if (ACT == ACT_GELU_FAST) return 0.5f * x * (1.f + tanhf(x * 0.7978845608f * (1.f + 0.044715f * x * x)));
  if (ACT == ACT_QUICK_GELU) return x / (1.f + __expf(-1.702f * x));
  if (ACT == ACT_RELU2) { float r = fmaxf(x, 0.f); return r * r; }
  return fmaxf(x, 0.f);
}

// out[t, :d] = act(x[t, :d]) * x[t, d:2d]
template <typename T, int ACT>
__global__ void act_and_mul_kernel(T* __restrict__ out, const T* __restrict__ x, int d, int64_t total_vec) {
  constexpr int N = Vec16<T>::N;
  pdl_trigger();
  pdl_wait();
  const int vec_per_row = d / N;
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total_vec; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / vec_per_row;
    const int c = (int)(i - t * vec_per_row) * N;
    Vec16<T> a = ld16(x + t * 2 * d + c), b = ld16(x + t * 2 * d + d + c), o;
#pragma unroll
    for (int j = 0; j < N; ++j) o.e[j] = from_f32<T>(act_fn<ACT>(to_f32(a.e[j])) * to_f32(b.e[j]));
    st16(out + t * d + c, o);
  }
}

// widths that are no multiple of a vector; IL: gate_i and up_i are neighbours
template <typename T, int ACT, bool IL>
__global__ void act_and_mul_scalar_kernel(T* __restrict__ out, const T* __restrict__ x, int d, int64_t total) {
  pdl_trigger();
  pdl_wait();
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / d;
    const int c = (int)(i - t * d);
    const T* row = x + t * 2 * d;
    out[i] = from_f32<T>(act_fn<ACT>(to_f32(row[IL ? 2 * c : c])) * to_f32(row[IL ? 2 * c + 1 : d + c]));
  }
}

// interleaved variant: x[t, 2i] = gate_i, x[t, 2i+1] = up_i (the weight layout of the fused gate_up GEMM epilogue)
template <typename T>
__global__ void silu_mul_interleaved_kernel(T* __restrict__ out, const T* __restrict__ x, int d, int64_t total_vec) {
  constexpr int N = Vec16<T>::N;
  pdl_trigger();
  pdl_wait();
  const int vec_per_row = d / N;                       // output vectors per row; each consumes two input vectors
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total_vec; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / vec_per_row;
    const int c = (int)(i - t * vec_per_row) * N;
    Vec16<T> a = ld16(x + t * 2 * d + 2 * c), b = ld16(x + t * 2 * d + 2 * c + N), o;
#pragma unroll
    for (int j = 0; j < N / 2; ++j) {
      o.e[j] = from_f32<T>(act_fn<ACT_SILU>(to_f32(a.e[2 * j])) * to_f32(a.e[2 * j + 1]));
      o.e[N / 2 + j] = from_f32<T>(act_fn<ACT_SILU>(to_f32(b.e[2 * j])) * to_f32(b.e[2 * j + 1]));
    }
    st16(out + t * d + c, o);
  }
}

template <typename T, int ACT>
__global__ void act_kernel(T* __restrict__ out, const T* __restrict__ x, int64_t total_vec) {
  constexpr int N = Vec16<T>::N;
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total_vec; i += (int64_t)gridDim.x * blockDim.x) {
    Vec16<T> a = ld16(x + i * N), o;
#pragma unroll
    for (int j = 0; j < N; ++j) o.e[j] = from_f32<T>(act_fn<ACT>(to_f32(a.e[j])));
    st16(out + i * N, o);
  }
}

// y[t, c] = x[t, c] * sigmoid(g[t, c]), row strides free; x may be y
template <typename T, int V>
__global__ void sigmoid_mul_kernel(const T* __restrict__ x, int64_t x_stride, const T* __restrict__ g, int64_t g_stride,
                                   T* __restrict__ y, int64_t y_stride, int n, int64_t total) {
  pdl_trigger();
  pdl_wait();
  const int per_row = n / V;
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / per_row;
    const int c = (int)(i - t * per_row) * V;
    if constexpr (V == 1) {
      y[t * y_stride + c] = from_f32<T>(__fdividef(to_f32(x[t * x_stride + c]), 1.f + __expf(-to_f32(g[t * g_stride + c]))));
    } else {
      const Vec16<T> a = ld16(x + t * x_stride + c), b = ld16(g + t * g_stride + c);
      Vec16<T> o;
#pragma unroll
      for (int j = 0; j < V; ++j) o.e[j] = from_f32<T>(__fdividef(to_f32(a.e[j]), 1.f + __expf(-to_f32(b.e[j]))));
      st16(y + t * y_stride + c, o);
    }
  }
}

// x[t, c] = cap tanh(x[t, c] / cap) in place, rows of n at any stride
template <typename T>
__global__ void soft_cap_kernel(T* __restrict__ x, int64_t stride, int n, int64_t total, float cap) {
  pdl_trigger();
  pdl_wait();
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / n;
    T* p = x + t * stride + (i - t * n);
    *p = from_f32<T>(cap * tanhf(to_f32(*p) / cap));
  }
}

int norm_threads(int H, int vecN) {
  int nvec = H / vecN;
  int t = (nvec + MAXV - 1) / MAXV;
  t = ((t + 31) / 32) * 32;
  if (t < 32) t = 32;
  // prefer more threads (1 vector each) while the row fits
  int t1 = ((nvec + 31) / 32) * 32;
  if (t1 <= 1024) t = t1;
  return t > 1024 ? 1024 : t;
}

}  // namespace

// x: [T, H] (row stride x_stride elements), w: [H]. ADD: residual [T, H] contiguous updated in place, normed → x.
EXPORT int vb_rms_norm(void* out, void* x, void* residual, const void* w, int T, int H, int64_t x_stride, float eps,
                       int gemma, int dtype, cudaStream_t st) {
  if (T == 0) return 0;
  DISPATCH_DTYPE(dtype, TT, {
    constexpr int N = Vec16<TT>::N;
    if (H % N != 0 || H / N > 1024 * MAXV) return -1;
    const int thr = norm_threads(H, N);
    if (residual) {
      if (gemma) vb_launch(rms_norm_kernel<TT, true, true>, T, thr, 0, st, (TT*)x, (TT*)x, (TT*)residual, (const TT*)w, H, eps, x_stride);
      else vb_launch(rms_norm_kernel<TT, true, false>, T, thr, 0, st, (TT*)x, (TT*)x, (TT*)residual, (const TT*)w, H, eps, x_stride);
    } else {
      if (gemma) vb_launch(rms_norm_kernel<TT, false, true>, T, thr, 0, st, (TT*)out, (TT*)x, (TT*)nullptr, (const TT*)w, H, eps, x_stride);
      else vb_launch(rms_norm_kernel<TT, false, false>, T, thr, 0, st, (TT*)out, (TT*)x, (TT*)nullptr, (const TT*)w, H, eps, x_stride);
    }
  });
  return (int)cudaGetLastError();
}

EXPORT int vb_layer_norm(void* out, const void* x, const void* w, const void* b, int T, int H, float eps, int dtype,
                         cudaStream_t st) {
  if (T == 0) return 0;
  DISPATCH_DTYPE(dtype, TT, {
    constexpr int N = Vec16<TT>::N;
    if (H % N != 0 || H / N > 1024 * MAXV) return -1;
    layer_norm_kernel<TT><<<T, norm_threads(H, N), 0, st>>>((TT*)out, (const TT*)x, (const TT*)w, (const TT*)b, H, eps);
  });
  return (int)cudaGetLastError();
}

#define ACT_SWITCH(KERNEL, ...)                                                         \
  switch (act) {                                                                        \
    case ACT_SILU: KERNEL<TT, ACT_SILU> __VA_ARGS__; break;                             \
    case ACT_GELU: KERNEL<TT, ACT_GELU> __VA_ARGS__; break;                             \
    case ACT_GELU_TANH: KERNEL<TT, ACT_GELU_TANH> __VA_ARGS__; break;                   \
    case ACT_RELU: KERNEL<TT, ACT_RELU> __VA_ARGS__; break;                             \
    case ACT_GELU_NEW: KERNEL<TT, ACT_GELU_NEW> __VA_ARGS__; break;                     \
    case ACT_GELU_FAST: KERNEL<TT, ACT_GELU_FAST> __VA_ARGS__; break;                   \
    case ACT_QUICK_GELU: KERNEL<TT, ACT_QUICK_GELU> __VA_ARGS__; break;                 \
    default: KERNEL<TT, ACT_RELU2> __VA_ARGS__; break;                                  \
  }

EXPORT int vb_act_and_mul(void* out, const void* x, int64_t T, int d, int act, int dtype, cudaStream_t st) {
  if (T == 0) return 0;
  DISPATCH_DTYPE(dtype, TT, {
    constexpr int N = Vec16<TT>::N;
    if (d % N != 0) {
      const int64_t n = T * d;
      const int nb = (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
      switch (act) {
        case ACT_SILU: vb_launch(act_and_mul_scalar_kernel<TT, ACT_SILU, false>, nb, 256, 0, st, (TT*)out, (const TT*)x, d, n); break;
        case ACT_GELU: vb_launch(act_and_mul_scalar_kernel<TT, ACT_GELU, false>, nb, 256, 0, st, (TT*)out, (const TT*)x, d, n); break;
        default: vb_launch(act_and_mul_scalar_kernel<TT, ACT_GELU_TANH, false>, nb, 256, 0, st, (TT*)out, (const TT*)x, d, n); break;
      }
      return (int)cudaGetLastError();
    }
    const int64_t total = T * (d / N);
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    switch (act) {
      case ACT_SILU: vb_launch(act_and_mul_kernel<TT, ACT_SILU>, blocks, 256, 0, st, (TT*)out, (const TT*)x, d, total); break;
      case ACT_GELU: vb_launch(act_and_mul_kernel<TT, ACT_GELU>, blocks, 256, 0, st, (TT*)out, (const TT*)x, d, total); break;
      default: vb_launch(act_and_mul_kernel<TT, ACT_GELU_TANH>, blocks, 256, 0, st, (TT*)out, (const TT*)x, d, total); break;
    }
  });
  return (int)cudaGetLastError();
}

EXPORT int vb_silu_mul_interleaved(void* out, const void* x, int64_t T, int d, int dtype, cudaStream_t st) {
  if (T == 0) return 0;
  if (dtype == DT_F32 || d % 8 != 0) {
    const int64_t n = T * d;
    const int nb = (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
    DISPATCH_DTYPE(dtype, TT, {
      vb_launch(act_and_mul_scalar_kernel<TT, ACT_SILU, true>, nb, 256, 0, st, (TT*)out, (const TT*)x, d, n);
    });
    return (int)cudaGetLastError();
  }
  const int64_t total = T * (d / 8);
  const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  DISPATCH_HALF(dtype, TT, {
    vb_launch(silu_mul_interleaved_kernel<TT>, blocks, 256, 0, st, (TT*)out, (const TT*)x, d, total);
  });
  return (int)cudaGetLastError();
}

EXPORT int vb_activation(void* out, const void* x, int64_t n, int act, int dtype, cudaStream_t st) {
  if (n == 0) return 0;
  DISPATCH_DTYPE(dtype, TT, {
    constexpr int N = Vec16<TT>::N;
    if (n % N != 0) return -1;
    const int64_t total = n / N;
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    ACT_SWITCH(act_kernel, <<<blocks, 256, 0, st>>>((TT*)out, (const TT*)x, total));
  });
  return (int)cudaGetLastError();
}

// y = a z^2 + z / 2 above zero, b (e^z - 1 - z) + z / 2 below; y may be x
template <typename T, int V>
__global__ void __launch_bounds__(256) xielu_kernel(const T* __restrict__ x, T* __restrict__ y, const float* __restrict__ coef, int64_t total) {
  pdl_trigger();
  const float a = coef[0], b = coef[1];
  pdl_wait();
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
    if constexpr (V == 1) {
      y[i] = from_f32<T>(sizeof(T) == 4 ? xielu(to_f32(x[i]), a, b) : xielu16(to_f32(x[i]), a, b));
    } else {
      Vec16<T> v = ld16(x + i * V);
#pragma unroll
      for (int j = 0; j < V; ++j) v.e[j] = from_f32<T>(sizeof(T) == 4 ? xielu(to_f32(v.e[j]), a, b) : xielu16(to_f32(v.e[j]), a, b));
      st16(y + i * V, v);
    }
  }
}

EXPORT int vb_xielu(const void* x, void* y, const float* coef, int64_t n, int dtype, cudaStream_t st) {
  if (n == 0) return 0;
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  DISPATCH_DTYPE(dtype, TT, {
    constexpr int N = Vec16<TT>::N;
    const bool vec = n % N == 0 && al(x) && al(y);
    const int64_t total = vec ? n / N : n;
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    if (vec) vb_launch(xielu_kernel<TT, N>, blocks, 256, 0, st, (const TT*)x, (TT*)y, coef, total);
    else vb_launch(xielu_kernel<TT, 1>, blocks, 256, 0, st, (const TT*)x, (TT*)y, coef, total);
  });
  return (int)cudaGetLastError();
}

EXPORT int vb_sigmoid_mul(const void* x, int64_t x_stride, const void* g, int64_t g_stride, void* y, int64_t y_stride, int64_t T, int n,
                          int dtype, cudaStream_t st) {
  if (T == 0) return 0;
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
#define GO(V)                                                                                                       \
  do {                                                                                                              \
    const int64_t total = T * (n / (V));                                                                            \
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);                      \
    vb_launch(sigmoid_mul_kernel<TT, V>, blocks, 256, 0, st, (const TT*)x, x_stride, (const TT*)g, g_stride, (TT*)y, y_stride, n, total); \
  } while (0)
  DISPATCH_DTYPE(dtype, TT, {
    constexpr int N = Vec16<TT>::N;
    if (n % N == 0 && x_stride % N == 0 && g_stride % N == 0 && y_stride % N == 0 && al(x) && al(g) && al(y)) GO(N);
    else GO(1);
  });
#undef GO
  return (int)cudaGetLastError();
}

EXPORT int vb_soft_cap(void* x, int64_t stride, int64_t T, int n, float cap, int dtype, cudaStream_t st) {
  if (T == 0 || n == 0) return 0;
  const int64_t total = T * n;
  const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  DISPATCH_DTYPE(dtype, TT, { vb_launch(soft_cap_kernel<TT>, blocks, 256, 0, st, (TT*)x, stride, n, total, cap); });
  return (int)cudaGetLastError();
}
