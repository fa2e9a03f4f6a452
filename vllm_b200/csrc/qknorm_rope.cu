// Fused per-head RMSNorm(q), RMSNorm(k) + RoPE + paged KV-cache insert (Qwen3 / Gemma-3 / OLMo-2 / Llama-4 style
// attention prologues).
//
// Reference ops: csrc/libtorch_stable/fused_qknorm_rope_kernel.cu:563-686 (q/k norm + rope over the fused qkv
// buffer) and the model-specific q-norm / rope / KV-insert fusions.  Ours goes one step
// further than the generic reference op: the rotated K head is written to its cache page from the registers that
// produced it and the V head is copied by a sibling warp of the same CTA, so a layer's attention prologue is ONE
// launch instead of norm(q), norm(k), rope, reshape_and_cache.
//
// Mapping: one warp per (token, head).  The head lives in registers (E = D / 32 consecutive elements per lane);
// sum of squares by warp shuffle; NeoX partner element (i, i + rot/2) sits in lane ^ (rot / 2 / E) at the same
// register slot, GPT-J pairs (2i, 2i+1) inside the lane.
#include "common.cuh"

namespace {

template <typename T, int E> struct LaneVec {
  alignas(16) T e[E];
  VB_DEVICE void load(const T* p) {
    if constexpr (E * sizeof(T) == 32) {
      reinterpret_cast<uint4*>(e)[0] = reinterpret_cast<const uint4*>(p)[0];
      reinterpret_cast<uint4*>(e)[1] = reinterpret_cast<const uint4*>(p)[1];
    } else if constexpr (E * sizeof(T) == 16) { *reinterpret_cast<uint4*>(e) = *reinterpret_cast<const uint4*>(p); }
    else if constexpr (E * sizeof(T) == 8) { *reinterpret_cast<uint2*>(e) = *reinterpret_cast<const uint2*>(p); }
    else if constexpr (E * sizeof(T) == 4) { *reinterpret_cast<uint32_t*>(e) = *reinterpret_cast<const uint32_t*>(p); }
    else {
#pragma unroll
      for (int j = 0; j < E; ++j) e[j] = p[j];
    }
  }
  VB_DEVICE void store(T* p) const {
    if constexpr (E * sizeof(T) == 32) {
      reinterpret_cast<uint4*>(p)[0] = reinterpret_cast<const uint4*>(e)[0];
      reinterpret_cast<uint4*>(p)[1] = reinterpret_cast<const uint4*>(e)[1];
    } else if constexpr (E * sizeof(T) == 16) { *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(e); }
    else if constexpr (E * sizeof(T) == 8) { *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(e); }
    else if constexpr (E * sizeof(T) == 4) { *reinterpret_cast<uint32_t*>(p) = *reinterpret_cast<const uint32_t*>(e); }
    else {
#pragma unroll
      for (int j = 0; j < E; ++j) p[j] = e[j];
    }
  }
};

struct Params {
  const int64_t* positions;
  void* q; void* k; const void* v;
  const void* q_w; const void* k_w;        // [D] norm weights (null = no norm on that side)
  const float* cos_sin;                    // [max_pos, rot] = cos | sin
  void* kv_cache; const int64_t* slot_mapping;
  int64_t q_stride, k_stride, v_stride;
  int T, Hq, Hkv, D, rot, BS;
  int neox, gemma, kv_fp8, vt;
  const float* v_cos_sin;                  // optional [max_pos, value width]: values are rotated too, in the layout of the keys
  int keep32;                              // the normalised head stays in 32 bits on its way to the rotation
  float eps, k_inv_scale, v_inv_scale;
};

template <typename T, int E>
__global__ void __launch_bounds__(256) qknorm_rope_cache_kernel(const Params p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int wpb = blockDim.x >> 5;
  const int items = p.Hq + 2 * p.Hkv;
  const int64_t w_global = (int64_t)blockIdx.x * wpb + (threadIdx.x >> 5);
  if (w_global >= (int64_t)p.T * items) return;
  const int t = (int)(w_global / items), it = (int)(w_global % items);
  const int D = p.D;
  const int64_t slot = p.slot_mapping ? p.slot_mapping[t] : -1;
  const bool do_cache = p.kv_cache != nullptr && slot >= 0;
  const int64_t blk = do_cache ? slot / p.BS : 0;
  const int off = do_cache ? (int)(slot % p.BS) : 0;

  // NeoX pairs sit in lanes `span` apart (a power of two, checked on the host), GPT-J pairs inside the lane
  auto rotate = [&](float (&f)[E], const float* cs, int rot) {
    const int half = rot / 2;
    if (p.neox) {
      const int span = half / E;                       // lanes per half
      const bool rot_lane = lane < 2 * span;
      const bool first = (lane & span) == 0;
#pragma unroll
      for (int j = 0; j < E; ++j) {
        const float other = __shfl_xor_sync(0xffffffffu, f[j], span);
        if (rot_lane) {
          const int i = (lane & (span - 1)) * E + j;   // index inside the half
          const float co = cs[i], si = cs[half + i];
          f[j] = first ? f[j] * co - other * si : f[j] * co + other * si;
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < E; j += 2) {
        const int e0 = lane * E + j;
        if (e0 < rot) {
          const int i = e0 >> 1;
          const float co = cs[i], si = cs[half + i];
          const float x1 = f[j], x2 = f[j + 1];
          f[j] = x1 * co - x2 * si;
          f[j + 1] = x2 * co + x1 * si;
        }
      }
    }
  };

  if (it >= p.Hq + p.Hkv) {
    // ---- V head → cache page
    if (!do_cache || p.v == nullptr) return;
    const int h = it - p.Hq - p.Hkv;
    LaneVec<T, E> a;
    a.load(reinterpret_cast<const T*>(p.v) + t * p.v_stride + (int64_t)h * D + lane * E);
    if (p.v_cos_sin) {
      float f[E];
#pragma unroll
      for (int j = 0; j < E; ++j) f[j] = to_f32(a.e[j]);
      rotate(f, p.v_cos_sin + p.positions[t] * D, D);
#pragma unroll
      for (int j = 0; j < E; ++j) a.e[j] = from_f32<T>(f[j]);
    }
    const size_t page = (((size_t)blk * 2 + 1) * p.Hkv + h) * p.BS * D;
    if (p.vt) {            // tensor-core layout: V pages transposed [D, BS]
      T* vc = reinterpret_cast<T*>(p.kv_cache) + page + off;
#pragma unroll
      for (int j = 0; j < E; ++j) vc[(size_t)(lane * E + j) * p.BS] = a.e[j];
    } else if (p.kv_fp8) {
      __nv_fp8_storage_t* vc = reinterpret_cast<__nv_fp8_storage_t*>(p.kv_cache) + page + (size_t)off * D + lane * E;
#pragma unroll
      for (int j = 0; j < E; ++j) vc[j] = __nv_cvt_float_to_fp8(to_f32(a.e[j]) * p.v_inv_scale, __NV_SATFINITE, __NV_E4M3);
    } else {
      a.store(reinterpret_cast<T*>(p.kv_cache) + page + (size_t)off * D + lane * E);
    }
    return;
  }
  // ---- q / k head: norm → rope → (k) cache
  const bool is_k = it >= p.Hq;
  const int h = is_k ? it - p.Hq : it;
  T* base = is_k ? reinterpret_cast<T*>(p.k) + t * p.k_stride + (int64_t)h * D
                 : reinterpret_cast<T*>(p.q) + t * p.q_stride + (int64_t)h * D;
  LaneVec<T, E> a;
  a.load(base + lane * E);
  float f[E];
#pragma unroll
  for (int j = 0; j < E; ++j) f[j] = to_f32(a.e[j]);
  const T* w = reinterpret_cast<const T*>(is_k ? p.k_w : p.q_w);
  if (w != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < E; ++j) ss += f[j] * f[j];
    ss = warp_sum(ss);
    const float inv = rsqrtf(ss / (float)D + p.eps);
    LaneVec<T, E> wv;
    wv.load(w + lane * E);
#pragma unroll
    for (int j = 0; j < E; ++j) {
      float g = to_f32(wv.e[j]);
      if (p.gemma) g += 1.f;
      f[j] *= inv * g;
      if (!p.keep32) f[j] = to_f32(from_f32<T>(f[j]));     // round through T like the unfused norm does
    }
  }
  if (p.rot > 0) rotate(f, p.cos_sin + p.positions[t] * p.rot, p.rot);
#pragma unroll
  for (int j = 0; j < E; ++j) a.e[j] = from_f32<T>(f[j]);
  a.store(base + lane * E);
  if (is_k && do_cache) {
    const size_t page = (((size_t)blk * 2 + 0) * p.Hkv + h) * p.BS * D + (size_t)off * D + lane * E;
    if (p.kv_fp8) {
      __nv_fp8_storage_t* kc = reinterpret_cast<__nv_fp8_storage_t*>(p.kv_cache) + page;
#pragma unroll
      for (int j = 0; j < E; ++j) kc[j] = __nv_cvt_float_to_fp8(to_f32(a.e[j]) * p.k_inv_scale, __NV_SATFINITE, __NV_E4M3);
    } else {
      a.store(reinterpret_cast<T*>(p.kv_cache) + page);
    }
  }
}

// The same for every head size, rotated width, value width and dtype: one warp per (token, head), the head in shared memory,
// 32-bit between norm and rotation.  DV: value width; DC: width of a cache row.
constexpr int ANY_MAX_D = 512, ANY_WARPS = 4;
template <typename T>
__global__ void __launch_bounds__(ANY_WARPS * 32) qknorm_rope_any_kernel(const Params p, int DV, int DC) {
  __shared__ float buf[ANY_WARPS][ANY_MAX_D];
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  float* f = buf[threadIdx.x >> 5];
  const int items = p.Hq + 2 * p.Hkv;
  const int64_t wg = (int64_t)blockIdx.x * ANY_WARPS + (threadIdx.x >> 5);
  if (wg >= (int64_t)p.T * items) return;
  const int t = (int)(wg / items), it = (int)(wg % items), D = p.D;
  const int64_t slot = p.slot_mapping ? p.slot_mapping[t] : -1;
  const bool do_cache = p.kv_cache != nullptr && slot >= 0;
  const int64_t blk = do_cache ? slot / p.BS : 0;
  const int off = do_cache ? (int)(slot % p.BS) : 0;
  T* cache = reinterpret_cast<T*>(p.kv_cache);
  if (it >= p.Hq + p.Hkv) {
    if (!do_cache || p.v == nullptr) return;
    const int h = it - p.Hq - p.Hkv;
    const T* v = reinterpret_cast<const T*>(p.v) + t * p.v_stride + (int64_t)h * DV;
    T* dst = cache + ((blk * 2 + 1) * p.Hkv + h) * p.BS * (int64_t)DC + (p.vt ? off : off * DC);
    const float* cs = p.v_cos_sin ? p.v_cos_sin + p.positions[t] * DV : nullptr;
    const int half = DV / 2;
    for (int d = lane; d < DV; d += 32) {
      T y = v[d];
      if (cs) {
        const int i = p.neox ? d % half : d >> 1;
        const bool first = p.neox ? d < half : (d & 1) == 0;
        const float x = to_f32(y), o = to_f32(v[p.neox ? (first ? d + half : d - half) : d ^ 1]), co = cs[i], si = cs[half + i];
        y = from_f32<T>(first ? x * co - o * si : x * co + o * si);
      }
      dst[p.vt ? (int64_t)d * p.BS : d] = y;
    }
    return;
  }
  const bool is_k = it >= p.Hq;
  const int h = is_k ? it - p.Hq : it;
  T* base = is_k ? reinterpret_cast<T*>(p.k) + t * p.k_stride + (int64_t)h * D
                 : reinterpret_cast<T*>(p.q) + t * p.q_stride + (int64_t)h * D;
  const T* w = reinterpret_cast<const T*>(is_k ? p.k_w : p.q_w);
  float ss = 0.f;
  for (int d = lane; d < D; d += 32) { const float x = to_f32(base[d]); f[d] = x; ss += x * x; }
  if (w != nullptr) {
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)D + p.eps);
    for (int d = lane; d < D; d += 32) f[d] *= inv * (to_f32(w[d]) + (p.gemma ? 1.f : 0.f));
  }
  __syncwarp();
  T* dst = is_k && do_cache ? cache + ((blk * 2 * p.Hkv + h) * p.BS + off) * (int64_t)DC : nullptr;
  const int half = p.rot / 2;
  const float* cs = p.rot > 0 ? p.cos_sin + p.positions[t] * p.rot : nullptr;
  for (int d = lane; d < D; d += 32) {
    float x = f[d];
    if (d < p.rot) {
      const int i = p.neox ? d % half : d >> 1;
      const bool first = p.neox ? d < half : (d & 1) == 0;
      const float o = f[p.neox ? (first ? d + half : d - half) : d ^ 1];
      const float co = cs[i], si = cs[half + i];
      x = first ? x * co - o * si : x * co + o * si;
    }
    const T y = from_f32<T>(x);
    base[d] = y;
    if (dst) dst[d] = y;
  }
}

// The norms over the WHOLE projections (all heads of q at once, all of k at once) instead of per head, then rotation and cache write,
// 32-bit in between.  CTA = one token's q, or its k and v; weights [H * D].  V elements per access.  k null: queries alone.
template <typename T, int V> VB_DEVICE void load_v(const T* p, float (&f)[V]) {
  if constexpr (V == 1) f[0] = to_f32(p[0]);
  else {
    const Vec16<T> x = ld16(p);
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = to_f32(x.e[j]);
  }
}
template <typename T, int V> VB_DEVICE void store_v(T* p, const float (&f)[V]) {
  if constexpr (V == 1) p[0] = from_f32<T>(f[0]);
  else {
    Vec16<T> x;
#pragma unroll
    for (int j = 0; j < V; ++j) x.e[j] = from_f32<T>(f[j]);
    st16(p, x);
  }
}
template <typename T, int V>
__global__ void __launch_bounds__(512) qknorm_rope_row_kernel(const Params p, int DV, int DC) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, D = p.D, half = p.rot / 2;
  const bool is_k = blockIdx.y == 1;
  const int heads = is_k ? p.Hkv : p.Hq, n = heads * D;
  T* base = is_k ? reinterpret_cast<T*>(p.k) + t * p.k_stride : reinterpret_cast<T*>(p.q) + t * p.q_stride;
  const T* w = reinterpret_cast<const T*>(is_k ? p.k_w : p.q_w);
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
    float f[V];
    load_v<T, V>(base + i, f);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += f[j] * f[j];
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)n + p.eps);
  const int64_t slot = is_k && p.slot_mapping ? p.slot_mapping[t] : -1;
  const bool do_cache = is_k && p.kv_cache != nullptr && slot >= 0;
  const int64_t blk = do_cache ? slot / p.BS : 0;
  const int off = do_cache ? (int)(slot % p.BS) : 0;
  T* cache = reinterpret_cast<T*>(p.kv_cache);
  const float* cs = p.rot > 0 ? p.cos_sin + p.positions[t] * p.rot : nullptr;
  const int turning = half / V, per_head = turning + (D - p.rot) / V;
  auto normed = [&](int at, float (&f)[V]) {
    float g[V];
    load_v<T, V>(base + at, f);
    load_v<T, V>(w + at, g);
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] *= inv * (g[j] + (p.gemma ? 1.f : 0.f));
  };
  for (int it = threadIdx.x; it < heads * per_head; it += blockDim.x) {
    const int h = it / per_head, c = it - h * per_head;
    T* dst = do_cache ? cache + ((blk * 2 * p.Hkv + h) * p.BS + off) * (int64_t)DC : nullptr;
    float a[V];
    if (c >= turning) {
      const int e = p.rot + (c - turning) * V;
      normed(h * D + e, a);
      store_v<T, V>(base + h * D + e, a);
      if (dst) store_v<T, V>(dst + e, a);
      continue;
    }
    const int e0 = p.neox ? c * V : 2 * c, e1 = p.neox ? half + c * V : 2 * c + 1;      // neighbours turn together: V = 1
    float b[V];
    normed(h * D + e0, a);
    normed(h * D + e1, b);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float co = cs[c * V + j], si = cs[half + c * V + j], x = a[j], y = b[j];
      a[j] = x * co - y * si;
      b[j] = y * co + x * si;
    }
    store_v<T, V>(base + h * D + e0, a);
    store_v<T, V>(base + h * D + e1, b);
    if (dst) { store_v<T, V>(dst + e0, a); store_v<T, V>(dst + e1, b); }
  }
  if (!do_cache || p.v == nullptr) return;
  const T* v = reinterpret_cast<const T*>(p.v) + t * p.v_stride;
  for (int it = threadIdx.x; it < p.Hkv * (DV / V); it += blockDim.x) {
    const int h = it / (DV / V), d = (it - h * (DV / V)) * V;
    T* dst = cache + ((blk * 2 + 1) * p.Hkv + h) * p.BS * (int64_t)DC;
    if constexpr (V == 1) {
      dst[p.vt ? (int64_t)d * p.BS + off : (int64_t)off * DC + d] = v[h * DV + d];
    } else {
      const Vec16<T> x = ld16(v + h * DV + d);
      if (p.vt) {
#pragma unroll
        for (int j = 0; j < V; ++j) dst[(int64_t)(d + j) * p.BS + off] = x.e[j];
      } else {
        st16(dst + (int64_t)off * DC + d, x);
      }
    }
  }
}

}  // namespace

// q, k: [T, H*D] views of the fused qkv buffer (rotated / normalised in place); v may be null (no cache write of V), and is rotated on
// its way into the cache where there is v_cos_sin [positions, value width];
// kv_cache may be null (norm + rope only).  flags: bit0 fp8 cache, bit1 transposed V pages, bit2 no rounding to T between the
// norm and the rotation.
EXPORT int vb_qknorm_rope_cache(const int64_t* positions, void* q, void* k, const void* v, const void* q_w, const void* k_w,
                                const float* cos_sin, const float* v_cos_sin, int rot, int T, int Hq, int Hkv, int D, int64_t q_stride,
                                int64_t k_stride, int64_t v_stride, void* kv_cache, const int64_t* slot_mapping, int BS,
                                int neox, int gemma, int flags, float eps, float k_scale, float v_scale, int dtype,
                                cudaStream_t st) {
  if (T == 0) return 0;
  if (dtype == DT_F32 || D % 32 != 0 || D > 512) return -1;
  const int E = D / 32;
  if (E != 2 && E != 4 && E != 8 && E != 16) return -1;
  if (rot > 0) {
    if (rot > D || rot % 2) return -1;
    if (neox) {
      const int half = rot / 2;
      if (half % E) return -1;
      const int span = half / E;
      if (span & (span - 1)) return -1;            // partner lane = lane ^ span
    } else if (E % 2) return -1;
  }
  Params p;
  p.v_cos_sin = v_cos_sin;
  p.positions = positions; p.q = q; p.k = k; p.v = v; p.q_w = q_w; p.k_w = k_w; p.cos_sin = cos_sin;
  p.kv_cache = kv_cache; p.slot_mapping = slot_mapping; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
  p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.D = D; p.rot = rot; p.BS = BS; p.neox = neox; p.gemma = gemma;
  p.kv_fp8 = flags & 1; p.vt = (flags >> 1) & 1; p.keep32 = (flags >> 2) & 1; p.eps = eps; p.k_inv_scale = 1.f / k_scale; p.v_inv_scale = 1.f / v_scale;
  const int64_t warps = (int64_t)T * (Hq + 2 * Hkv);
  const int wpb = 8;
  const unsigned blocks = (unsigned)((warps + wpb - 1) / wpb);
  DISPATCH_HALF(dtype, TT, {
    switch (E) {
      case 2: vb_launch(qknorm_rope_cache_kernel<TT, 2>, dim3(blocks), dim3(wpb * 32), 0, st, p); break;
      case 4: vb_launch(qknorm_rope_cache_kernel<TT, 4>, dim3(blocks), dim3(wpb * 32), 0, st, p); break;
      case 8: vb_launch(qknorm_rope_cache_kernel<TT, 8>, dim3(blocks), dim3(wpb * 32), 0, st, p); break;
      default: vb_launch(qknorm_rope_cache_kernel<TT, 16>, dim3(blocks), dim3(wpb * 32), 0, st, p); break;
    }
  });
  return (int)cudaGetLastError();
}

// Every other shape and dtype.  The cache holds the model dtype.
EXPORT int vb_qknorm_rope_any(const int64_t* positions, void* q, void* k, const void* v, const void* q_w, const void* k_w,
                              const float* cos_sin, const float* v_cos_sin, int rot, int T, int Hq, int Hkv, int D, int DV, int DC, int64_t q_stride,
                              int64_t k_stride, int64_t v_stride, void* kv_cache, const int64_t* slot_mapping, int BS, int neox,
                              int gemma, int vt, float eps, int dtype, cudaStream_t st) {
  if (T == 0) return 0;
  if (D > ANY_MAX_D || rot > D || rot % 2 || DC < D || DC < DV || (v_cos_sin && DV % 2)) return -1;
  Params p = {};
  p.v_cos_sin = v_cos_sin;
  p.positions = positions; p.q = q; p.k = k; p.v = v; p.q_w = q_w; p.k_w = k_w; p.cos_sin = cos_sin;
  p.kv_cache = kv_cache; p.slot_mapping = slot_mapping; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
  p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.D = D; p.rot = rot; p.BS = BS; p.neox = neox; p.gemma = gemma; p.vt = vt; p.eps = eps;
  const int64_t warps = (int64_t)T * (Hq + 2 * Hkv);
  dim3 grid((unsigned)((warps + ANY_WARPS - 1) / ANY_WARPS));
  DISPATCH_DTYPE(dtype, TT, vb_launch(qknorm_rope_any_kernel<TT>, grid, dim3(ANY_WARPS * 32), 0, st, p, DV, DC));
  return (int)cudaGetLastError();
}

// Norms over whole rows: q_w [Hq * D], k_w [Hkv * D].  Hkv 0: queries alone (a layer that reads another layer's keys).  The cache
// holds the model dtype, rows DC wide.
EXPORT int vb_qknorm_rope_row(const int64_t* positions, void* q, void* k, const void* v, const void* q_w, const void* k_w,
                              const float* cos_sin, int rot, int T, int Hq, int Hkv, int D, int DV, int DC, int64_t q_stride,
                              int64_t k_stride, int64_t v_stride, void* kv_cache, const int64_t* slot_mapping, int BS, int neox,
                              int gemma, int vt, float eps, int dtype, cudaStream_t st) {
  if (T == 0) return 0;
  if (!q_w || (Hkv && !k_w) || rot > D || rot % 2 || (kv_cache && (DC < D || DC < DV))) return -1;
  Params p = {};
  p.positions = positions; p.q = q; p.k = k; p.v = v; p.q_w = q_w; p.k_w = k_w; p.cos_sin = cos_sin;
  p.kv_cache = kv_cache; p.slot_mapping = slot_mapping; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
  p.T = T; p.Hq = Hq; p.Hkv = Hkv; p.D = D; p.rot = rot; p.BS = BS; p.neox = neox; p.gemma = gemma; p.vt = vt; p.eps = eps;
  DISPATCH_DTYPE(dtype, TT, {
    constexpr int N = Vec16<TT>::N;
    auto ok = [](const void* a, int64_t stride) { return !a || ((reinterpret_cast<uintptr_t>(a) & 15) == 0 && stride % N == 0); };
    const bool vec = (neox || rot == 0) && D % N == 0 && rot % (2 * N) == 0 && DV % N == 0 && DC % N == 0 && ok(q, q_stride) &&
                     ok(k, k_stride) && ok(v, v_stride) && ok(q_w, 0) && ok(k_w, 0) && ok(kv_cache, 0);
    const int items = Hq * D / (vec ? N : 1), want = (items + 31) / 32 * 32;
    const dim3 grid(T, Hkv ? 2 : 1), block(want < 64 ? 64 : want > 512 ? 512 : want);
    if (vec) vb_launch(qknorm_rope_row_kernel<TT, N>, grid, block, 0, st, p, DV, DC);
    else vb_launch(qknorm_rope_row_kernel<TT, 1>, grid, block, 0, st, p, DV, DC);
  });
  return (int)cudaGetLastError();
}
