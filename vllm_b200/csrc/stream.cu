// fp32 residual stream: embedding entry, and "norm the sublayer's output, then add" (post-norm) steps.
//
// Models that keep the residual sum in 32-bit and normalise the OUTPUT of every sublayer run two kernels of this file
// per layer.  The stream x lives in fp32; beside it every step leaves the 16-bit copy the next GEMM reads (or, in front
// of the LM head, the model's final norm of it), so the conversion never costs a pass of its own:
//   embed_stream      x = table[id] * scale (+ pos_table[position]);   out = T(x)
//   post_norm_add     y = a dense sublayer output row, or the routed sum  sum_j w_j * rows[inv_j]  of an expert layer
//                     x += rmsnorm(y) * w;   out = T(x)  |  T(rmsnorm(x) * w_next)
//   norm_add          the same step for blocks with a norm on either side of a sublayer, layer norms or RMS norms:
//                     x += m norm(y + bias);   out = T(norm_next(x))       (or x = table[id] at the model's entry)
//   add_norm          the same step for pre-norm blocks:  x += y + routed sum;   out = T(norm_next(x)).  The routed sum may have
//                     identity experts: slots whose expert number is past the last one add w_j times the layer's input
//   hyper_step        hyper-connections, S streams per token:  x_t = sum_s mix[s, t] x_s + out[t] y;   out = T(rmsnorm(sum_s in[s] x_s))
//                     (or x_s = rmsnorm(table[id]) for all s at the model's entry); one read and one write of every stream
// The combine of the expert layer is the load of post_norm_add and add_norm: expert outputs are read once, summed in slot order in
// fp32 (deterministic) and never written back.
#include "common.cuh"

namespace stream {

template <typename T, int V> struct Pack { T e[V]; };
template <typename T, int V> VB_DEVICE void load_f32(const T* p, float (&v)[V]) {
  if constexpr (V == 1) {
    v[0] = to_f32(p[0]);
  } else if constexpr (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 f = *reinterpret_cast<const float4*>(p + i);
      v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
    }
  } else {
    const Vec16<T> x = ld16(p);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = to_f32(x.e[i]);
  }
}
template <typename T, int V> VB_DEVICE void store_f32(T* p, const float (&v)[V]) {
  if constexpr (V == 1) {
    p[0] = from_f32<T>(v[0]);
  } else if constexpr (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
    Vec16<T> x;
#pragma unroll
    for (int i = 0; i < V; ++i) x.e[i] = from_f32<T>(v[i]);
    st16(p, x);
  }
}

// one CTA per token; V consecutive elements per access
template <typename T, int V>
__global__ void embed_stream_kernel(const int* __restrict__ ids, const int64_t* __restrict__ positions,
                                    const T* __restrict__ table, const T* __restrict__ pos_table, float scale,
                                    float* __restrict__ x, T* __restrict__ out, int H, int vocab, int max_pos) {
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int id = min(max(ids[row], 0), vocab - 1);
  const T* tr = table + (int64_t)id * H;
  const T* pr = nullptr;
  if (pos_table) {
    int64_t p = positions[row];
    p = p < 0 ? 0 : (p >= max_pos ? max_pos - 1 : p);
    pr = pos_table + p * H;
  }
  for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
    float v[V];
    load_f32<T, V>(tr + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] *= scale;
    if (pr) {
      float q[V];
      load_f32<T, V>(pr + i, q);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] += q[j];
    }
    store_f32<float, V>(x + row * H + i, v);
    if (out) store_f32<T, V>(out + row * H + i, v);
  }
}

// NV vectors of V elements per thread stay in registers between the reductions (H <= 1024 * NV * V)
template <typename T, int V, int NV>
__global__ void __launch_bounds__(1024)
post_norm_add_kernel(const T* __restrict__ y, int64_t y_stride, const int* __restrict__ inv, const float* __restrict__ pair_w,
                     int k, const T* __restrict__ w, int w_off, float* __restrict__ x, const T* __restrict__ w_next,
                     int w_next_off, T* __restrict__ out, int H, float eps) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int step = blockDim.x * V;
  float v[NV][V];
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * step;
    if (i >= H) continue;
    if (inv) {
#pragma unroll
      for (int j = 0; j < V; ++j) v[n][j] = 0.f;
      for (int s = 0; s < k; ++s) {
        const int p = inv[row * k + s];
        if (p < 0) continue;                            // pair computed by another rank
        const float ws = pair_w[row * k + s];
        float r[V];
        load_f32<T, V>(y + (int64_t)p * y_stride + i, r);
#pragma unroll
        for (int j = 0; j < V; ++j) v[n][j] += ws * r[j];
      }
    } else {
      load_f32<T, V>(y + row * y_stride + i, v[n]);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) ss += v[n][j] * v[n][j];
  }
  if (w) {
    const float r1 = rsqrtf(block_sum(ss, red) / (float)H + eps);
    ss = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = threadIdx.x * V + n * step;
      if (i >= H) continue;
      float g[V], xv[V];
      load_f32<T, V>(w + i, g);
      load_f32<float, V>(x + row * H + i, xv);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        v[n][j] = xv[j] + v[n][j] * r1 * (g[j] + (float)w_off);
        ss += v[n][j] * v[n][j];
      }
      store_f32<float, V>(x + row * H + i, v[n]);
    }
  }
  if (!out) return;
  float r2 = 1.f;
  if (w_next) r2 = rsqrtf(block_sum(ss, red) / (float)H + eps);
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * step;
    if (i >= H) continue;
    if (w_next) {
      float g[V];
      load_f32<T, V>(w_next + i, g);
#pragma unroll
      for (int j = 0; j < V; ++j) v[n][j] *= r2 * (g[j] + (float)w_next_off);
    }
    store_f32<T, V>(out + row * H + i, v[n]);
  }
}

// mean and variance (or the mean square) over the row held in v, then (v - mean) * rstd * w + b in place
template <typename T, int V, int NV, bool LN>
VB_DEVICE void normalise(float (&v)[NV][V], const T* w, const T* b, int w_off, int H, float eps, float* red) {
  const int step = blockDim.x * V;
  float mean = 0.f;
  if constexpr (LN) {
    float s = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n)
      if (threadIdx.x * V + n * step < H)
#pragma unroll
        for (int j = 0; j < V; ++j) s += v[n][j];
    mean = block_sum(s, red) / (float)H;
  }
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n)
    if (threadIdx.x * V + n * step < H)
#pragma unroll
      for (int j = 0; j < V; ++j) { v[n][j] -= mean; ss += v[n][j] * v[n][j]; }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)H + eps);
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * step;
    if (i >= H) continue;
    float g[V], o[V];
    load_f32<T, V>(w + i, g);
    if (b) load_f32<T, V>(b + i, o);
#pragma unroll
    for (int j = 0; j < V; ++j) v[n][j] = v[n][j] * r * (g[j] + (float)w_off) + (b ? o[j] : 0.f);
  }
}

// entry (ids): x = table[id];  else x += mult * norm1(y + y_bias).  out = norm2(x), or x where w2 is null
template <typename T, int V, int NV, bool LN>
__global__ void __launch_bounds__(1024)
norm_add_kernel(const int* __restrict__ ids, int vocab, const T* __restrict__ y, int64_t y_stride, const float* __restrict__ y_bias,
                const T* __restrict__ w1, const T* __restrict__ b1, float mult, float* __restrict__ x, const T* __restrict__ w2,
                const T* __restrict__ b2, int w_off, T* __restrict__ out, int H, float eps) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int step = blockDim.x * V;
  const T* src = y + (ids ? (int64_t)min(max(ids[row], 0), vocab - 1) * H : row * y_stride);
  float v[NV][V];
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * step;
    if (i >= H) continue;
    load_f32<T, V>(src + i, v[n]);
    if (y_bias) {
      float b[V];
      load_f32<float, V>(y_bias + i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) v[n][j] += b[j];
    }
  }
  if (!ids) {
    normalise<T, V, NV, LN>(v, w1, b1, w_off, H, eps, red);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = threadIdx.x * V + n * step;
      if (i >= H) continue;
      float xv[V];
      load_f32<float, V>(x + row * H + i, xv);
#pragma unroll
      for (int j = 0; j < V; ++j) v[n][j] = xv[j] + mult * v[n][j];
    }
  }
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * step;
    if (i < H) store_f32<float, V>(x + row * H + i, v[n]);
  }
  if (!out) return;
  if (w2) normalise<T, V, NV, LN>(v, w2, b2, w_off, H, eps, red);
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * step;
    if (i < H) store_f32<T, V>(out + row * H + i, v[n]);
  }
}

// x += y + sum_s w_s (a row of `rows`, or of `h` for identity experts);  out = norm(x), or x where w2 is null.  y, rows, h may be null
struct Routed {
  const void* rows; int64_t stride;
  const int* inv; const float* w; const int* ids;       // [T, k]; inv < 0: no row (identity expert, or another rank's)
  int k, experts;                                       // ids from `experts` on are identities
  const void* h; int64_t h_stride;
};
template <typename T, int V, int NV, bool LN>
__global__ void __launch_bounds__(1024)
add_norm_kernel(const T* __restrict__ y, int64_t y_stride, const Routed r, float* __restrict__ x, const T* __restrict__ w2,
                const T* __restrict__ b2, int w_off, T* __restrict__ out, int H, float eps) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int step = blockDim.x * V;
  float id_w = 0.f;
  if (r.h)
    for (int s = 0; s < r.k; ++s)
      if (r.ids[row * r.k + s] >= r.experts) id_w += r.w[row * r.k + s];
  float v[NV][V];
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * step;
    if (i >= H) continue;
    load_f32<float, V>(x + row * H + i, v[n]);
    auto add = [&](const T* src, float ws) {
      float u[V];
      load_f32<T, V>(src + i, u);
#pragma unroll
      for (int j = 0; j < V; ++j) v[n][j] += ws * u[j];
    };
    if (y) add(y + row * y_stride, 1.f);
    if (r.rows) {
#pragma unroll 4
      for (int s = 0; s < r.k; ++s) {
        const int p = r.inv[row * r.k + s];
        if (p >= 0) add(reinterpret_cast<const T*>(r.rows) + (int64_t)p * r.stride, r.w[row * r.k + s]);
      }
    }
    if (id_w != 0.f) add(reinterpret_cast<const T*>(r.h) + row * r.h_stride, id_w);
    store_f32<float, V>(x + row * H + i, v[n]);
  }
  if (!out) return;
  if (w2) normalise<T, V, NV, LN>(v, w2, b2, w_off, H, eps, red);
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * step;
    if (i < H) store_f32<T, V>(out + row * H + i, v[n]);
  }
}

// S streams per token (x [T, S, H]).  ids: entry, x_s = rmsnorm(y[id]) * w_e;  entry rows (no coef): x_s = y;  coef (out [S], mix [S, S]):
// x_t = sum_s mix[s, t] x_s + out[t] y;  y null: x is read only.  out = rmsnorm(sum_s into[s] x_s) * w.  SM: S, or a bound of it (V = 1).
constexpr int MAX_STREAMS = 16;
template <typename T, int V, int NV, int SM, bool EXACT>
__global__ void __launch_bounds__(512)
hyper_kernel(const int* __restrict__ ids, int vocab, const T* __restrict__ y, int64_t y_stride, const T* __restrict__ w_e,
             const float* __restrict__ coef, const float* __restrict__ into, float* __restrict__ x, int S_, const T* __restrict__ w,
             T* __restrict__ out, int H, float eps) {
  __shared__ float red[32];
  __shared__ float cf[2 * MAX_STREAMS + MAX_STREAMS * MAX_STREAMS];        // into, out, mix
  pdl_trigger();
  const int S = EXACT ? SM : S_;
  const bool step = coef != nullptr;
  // weights are never written by a predecessor: they may be fetched before it ends
  for (int i = threadIdx.x; i < S; i += blockDim.x) cf[i] = into[i];
  if (step)
    for (int i = threadIdx.x; i < S + S * S; i += blockDim.x) cf[S + i] = coef[i];
  __syncthreads();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int stride = blockDim.x * V;
  const float* in_ = cf;
  const float* out_ = cf + S;
  const float* mix = cf + 2 * S;
  float* xr = x + row * S * H;
  float u[NV][V];
  if (y && !step) {
    const T* src = y + (ids ? (int64_t)min(max(ids[row], 0), vocab - 1) * H : row * y_stride);
#pragma unroll
    for (int n = 0; n < NV; ++n)
      if (threadIdx.x * V + n * stride < H) load_f32<T, V>(src + threadIdx.x * V + n * stride, u[n]);
    if (w_e) normalise<T, V, NV, false>(u, w_e, nullptr, 0, H, eps, red);
    float total = 0.f;
    for (int s = 0; s < S; ++s) total += in_[s];
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int i = threadIdx.x * V + n * stride;
      if (i >= H) continue;
      for (int s = 0; s < S; ++s) store_f32<float, V>(xr + (int64_t)s * H + i, u[n]);
#pragma unroll
      for (int j = 0; j < V; ++j) u[n][j] *= total;
    }
  } else {
    constexpr int UN = EXACT ? NV : 1, US = EXACT ? SM : 1;              // many streams: loops, not eight thousand instructions
#pragma unroll UN
    for (int n = 0; n < NV; ++n) {
      const int i = threadIdx.x * V + n * stride;
      if (i >= H) continue;
      float xs[SM][V], yv[V];
#pragma unroll US
      for (int s = 0; s < SM; ++s)
        if (EXACT || s < S) load_f32<float, V>(xr + (int64_t)s * H + i, xs[s]);
      if (step) load_f32<T, V>(y + row * y_stride + i, yv);
#pragma unroll
      for (int j = 0; j < V; ++j) u[n][j] = 0.f;
#pragma unroll US
      for (int t = 0; t < SM; ++t) {
        if (!EXACT && t >= S) break;
        float v[V];
        if (step) {
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] = out_[t] * yv[j];
#pragma unroll US
          for (int s = 0; s < SM; ++s)
            if (EXACT || s < S) {
              const float m = mix[s * S + t];
#pragma unroll
              for (int j = 0; j < V; ++j) v[j] += m * xs[s][j];
            }
          store_f32<float, V>(xr + (int64_t)t * H + i, v);
        } else {
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] = xs[t][j];
        }
#pragma unroll
        for (int j = 0; j < V; ++j) u[n][j] += in_[t] * v[j];
      }
    }
  }
  normalise<T, V, NV, false>(u, w, nullptr, 0, H, eps, red);
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int i = threadIdx.x * V + n * stride;
    if (i < H) store_f32<T, V>(out + row * H + i, u[n]);
  }
}

template <typename T> constexpr int vec_of() { return sizeof(T) == 4 ? 4 : 8; }
static bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace stream

// x [T, H] fp32 and (optional) out [T, H] in the model dtype; pos_table may be null (no learned positions)
EXPORT int vb_embed_stream(const int* ids, const int64_t* positions, const void* table, const void* pos_table, float scale,
                           float* x, void* out, int T_, int H, int vocab, int max_pos, int dtype, cudaStream_t st) {
  using namespace stream;
  if (T_ == 0) return 0;
  DISPATCH_DTYPE(dtype, T, {
    constexpr int V = vec_of<T>();
    const bool vec = H % V == 0 && al16(table) && (!pos_table || al16(pos_table)) && al16(x) && (!out || al16(out));
    const int items = vec ? H / V : H;
    const int thr = items >= 256 ? 256 : ((items + 31) / 32) * 32;
    if (vec) vb_launch(embed_stream_kernel<T, V>, dim3(T_), dim3(thr), 0, st, ids, positions, (const T*)table, (const T*)pos_table, scale, x, (T*)out, H, vocab, max_pos);
    else vb_launch(embed_stream_kernel<T, 1>, dim3(T_), dim3(thr), 0, st, ids, positions, (const T*)table, (const T*)pos_table, scale, x, (T*)out, H, vocab, max_pos);
  });
  return (int)cudaGetLastError();
}

// inv / pair_w null: y is [T, H].  Else y holds expert output rows and inv [T, k] maps (token, slot) to a row (or -1).
// w null: no norm, no residual (x unused): out = T(y or the routed sum).  w_off / w_next_off: 1 where
// the stored weight is the deviation from one.
EXPORT int vb_post_norm_add(const void* y, int64_t y_stride, const int* inv, const float* pair_w, int k, const void* w,
                            int w_off, float* x, const void* w_next, int w_next_off, void* out, int T_, int H, float eps,
                            int dtype, cudaStream_t st) {
  using namespace stream;
  if (T_ == 0) return 0;
  if (w && !x) return -1;
#define GO(VV, NVV) vb_launch(post_norm_add_kernel<T, VV, NVV>, dim3(T_), dim3(thr), 0, st, (const T*)y, y_stride, inv, pair_w, k, (const T*)w, w_off, x, (const T*)w_next, w_next_off, (T*)out, H, eps)
  DISPATCH_DTYPE(dtype, T, {
    constexpr int V = vec_of<T>();
    const bool vec = H % V == 0 && y_stride % V == 0 && al16(y) && (!w || al16(w)) && (!x || al16(x)) &&
                     (!w_next || al16(w_next)) && (!out || al16(out));
    const int items = vec ? H / V : H;
    const int thr = items >= 1024 ? 1024 : ((items + 31) / 32) * 32;
    const int nv = (items + thr - 1) / thr;
    if (vec) { if (nv <= 1) GO(V, 1); else if (nv <= 4) GO(V, 4); else return -1; }
    else { if (nv <= 1) GO(1, 1); else if (nv <= 16) GO(1, 16); else return -1; }
  });
#undef GO
  return (int)cudaGetLastError();
}

// One step of an fp32 stream between sublayers: x += mult * norm1(y + y_bias), out = norm2(x) in the model dtype.  At the
// model's entry ``ids`` pick rows of y = the embedding table [vocab, H] instead and x is written.  ln: layer norms (with b1,
// b2), else RMS norms with weights w + w_off.  w2 null: out = T(x).
EXPORT int vb_norm_add(const int* ids, int vocab, const void* y, int64_t y_stride, const float* y_bias, const void* w1,
                       const void* b1, float mult, float* x, const void* w2, const void* b2, int w_off, int ln, void* out,
                       int T_, int H, float eps, int dtype, cudaStream_t st) {
  using namespace stream;
  if (T_ == 0) return 0;
  if (!ids && !w1) return -1;
#define GO(VV, NVV)                                                                                                          \
  do {                                                                                                                       \
    if (ln) vb_launch(norm_add_kernel<T, VV, NVV, true>, dim3(T_), dim3(thr), 0, st, ids, vocab, (const T*)y, y_stride, y_bias, (const T*)w1, (const T*)b1, mult, x, (const T*)w2, (const T*)b2, w_off, (T*)out, H, eps); \
    else vb_launch(norm_add_kernel<T, VV, NVV, false>, dim3(T_), dim3(thr), 0, st, ids, vocab, (const T*)y, y_stride, y_bias, (const T*)w1, (const T*)b1, mult, x, (const T*)w2, (const T*)b2, w_off, (T*)out, H, eps); \
  } while (0)
  DISPATCH_DTYPE(dtype, T, {
    constexpr int V = vec_of<T>();
    auto ok = [](const void* p) { return !p || al16(p); };
    const bool vec = H % V == 0 && y_stride % V == 0 && ok(y) && ok(y_bias) && ok(w1) && ok(b1) && ok(x) && ok(w2) && ok(b2) && ok(out);
    const int items = vec ? H / V : H;
    const int thr = items >= 1024 ? 1024 : ((items + 31) / 32) * 32;
    const int nv = (items + thr - 1) / thr;
    if (vec) { if (nv <= 1) GO(V, 1); else if (nv <= 4) GO(V, 4); else return -1; }
    else { if (nv <= 1) GO(1, 1); else if (nv <= 16) GO(1, 16); else return -1; }
  });
#undef GO
  return (int)cudaGetLastError();
}

// x += y + routed sum, out = norm2(x) in the model dtype (x where w2 is null).  y [T, H] or null; rows null: nothing routed, else
// inv / pair_w / ids [T, k]; h [T, H]: the input that identity experts (ids >= experts) pass on, or null.  ln, w_off as in vb_norm_add.
EXPORT int vb_add_norm(const void* y, int64_t y_stride, const void* rows, int64_t rows_stride, const int* inv, const float* pair_w,
                       const int* ids, int k, int experts, const void* h, int64_t h_stride, float* x, const void* w2, const void* b2,
                       int w_off, int ln, void* out, int T_, int H, float eps, int dtype, cudaStream_t st) {
  using namespace stream;
  if (T_ == 0) return 0;
  if ((rows && (!inv || !pair_w)) || (h && (!ids || !pair_w))) return -1;
  const Routed r = {rows, rows_stride, inv, pair_w, ids, k, experts, h, h_stride};
#define GO(VV, NVV)                                                                                                          \
  do {                                                                                                                       \
    if (ln) vb_launch(add_norm_kernel<T, VV, NVV, true>, dim3(T_), dim3(thr), 0, st, (const T*)y, y_stride, r, x, (const T*)w2, (const T*)b2, w_off, (T*)out, H, eps); \
    else vb_launch(add_norm_kernel<T, VV, NVV, false>, dim3(T_), dim3(thr), 0, st, (const T*)y, y_stride, r, x, (const T*)w2, (const T*)b2, w_off, (T*)out, H, eps); \
  } while (0)
  DISPATCH_DTYPE(dtype, T, {
    constexpr int V = vec_of<T>();
    auto ok = [](const void* p) { return !p || al16(p); };
    const bool vec = H % V == 0 && (!y || y_stride % V == 0) && (!rows || rows_stride % V == 0) && (!h || h_stride % V == 0) && ok(y) &&
                     ok(rows) && ok(h) && ok(x) && ok(w2) && ok(b2) && ok(out);
    const int items = vec ? H / V : H;
    const int thr = items >= 1024 ? 1024 : ((items + 31) / 32) * 32;
    const int nv = (items + thr - 1) / thr;
    if (vec) { if (nv <= 1) GO(V, 1); else if (nv <= 4) GO(V, 4); else return -1; }
    else { if (nv <= 1) GO(1, 1); else if (nv <= 16) GO(1, 16); else return -1; }
  });
#undef GO
  return (int)cudaGetLastError();
}

// S streams x [T, S, H] (see hyper_kernel).  coef null and y given: the model's entry (ids null: rows of y as they are).
EXPORT int vb_hyper_step(const int* ids, int vocab, const void* y, int64_t y_stride, const void* w_e, const float* coef, const float* into,
                         float* x, int S, const void* w, void* out, int T_, int H, float eps, int dtype, cudaStream_t st) {
  using namespace stream;
  if (T_ == 0) return 0;
  if (S < 1 || S > MAX_STREAMS || !into || !x || !w || !out || (coef && !y) || (ids && !y)) return -1;
#define RUN(VV, NVV, SS, EX) vb_launch(hyper_kernel<T, VV, NVV, SS, EX>, dim3(T_), dim3(thr), 0, st, ids, vocab, (const T*)y, y_stride, (const T*)w_e, coef, into, x, S, (const T*)w, (T*)out, H, eps)
#define GO(VV, NVV)                                                                                                    \
  do {                                                                                                                 \
    if (S == 1) RUN(VV, NVV, 1, true); else if (S == 2) RUN(VV, NVV, 2, true); else if (S == 3) RUN(VV, NVV, 3, true);  \
    else RUN(VV, NVV, 4, true);                                                                                        \
  } while (0)
  DISPATCH_DTYPE(dtype, T, {
    constexpr int V = vec_of<T>();
    auto ok = [](const void* p) { return !p || al16(p); };
    const bool vec = S <= 4 && H % V == 0 && (ids || y_stride % V == 0) && ok(y) && ok(w_e) && ok(x) && ok(w) && ok(out);
    const int items = vec ? H / V : H;
    const int thr = items >= 512 ? 512 : ((items + 31) / 32) * 32;
    const int nv = (items + thr - 1) / thr;
    if (vec && nv <= 8) { if (nv <= 1) GO(V, 1); else if (nv <= 4) GO(V, 4); else GO(V, 8); }
    else if (!vec && nv <= 1) { if (S <= 4) GO(1, 1); else RUN(1, 1, MAX_STREAMS, false); }
    else if (!vec && nv <= 32) RUN(1, 32, MAX_STREAMS, false);
    else return -1;
  });
#undef GO
#undef RUN
  return (int)cudaGetLastError();
}
