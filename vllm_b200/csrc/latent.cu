// Latent attention (MLA) around the tensor-core kernels: the fused down-projection epilogue, and a variable-length
// attention over the latent cache for every size and dtype the tcgen05 kernels (mla_decode.cu, mla_prefill.cu) do not
// take: fp32, latent widths that are not multiples of 8, wide heads.
//
//   latent_norm_cache   [c_q | c_kv] (one GEMM) → rmsnorm of both halves; c_kv goes straight into its page
//   latent_rope_cache   [q heads | .. | c_kv | k_r] (one GEMM) → rotation of every query head's last part, in place; rmsnorm of c_kv and
//                       rotation of k_r, both straight into their cache row
//   mla_simt            MQA over cache rows [c : R | rope : P], absorbed queries; fp32 arithmetic throughout
#include "common.cuh"

namespace latent {

// one CTA per token
template <typename T, int V>
__global__ void __launch_bounds__(256)
latent_norm_cache_kernel(const T* __restrict__ lat, int64_t lat_stride, int Rq, const T* __restrict__ wq, T* __restrict__ cq,
                         int Rk, const T* __restrict__ wk, T* __restrict__ ckv, T* __restrict__ cache, int64_t cache_row,
                         const int64_t* __restrict__ slots, float eps) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const T* l = lat + row * lat_stride;
  auto sumsq = [&](const T* p, int n) {
    float s = 0.f;
    for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
      if constexpr (V == 1) {
        const float f = to_f32(p[i]);
        s += f * f;
      } else {
        const Vec16<T> v = ld16(p + i);
#pragma unroll
        for (int j = 0; j < V; ++j) { const float f = to_f32(v.e[j]); s += f * f; }
      }
    }
    return block_sum(s, red);
  };
  auto scale_row = [&](const T* p, const T* w, float r, int n, T* o1, T* o2) {
    for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
      if constexpr (V == 1) {
        const T o = from_f32<T>(to_f32(p[i]) * r * to_f32(w[i]));
        if (o1) o1[i] = o;
        if (o2) o2[i] = o;
      } else {
        const Vec16<T> v = ld16(p + i), g = ld16(w + i);
        Vec16<T> o;
#pragma unroll
        for (int j = 0; j < V; ++j) o.e[j] = from_f32<T>(to_f32(v.e[j]) * r * to_f32(g.e[j]));
        if (o1) st16(o1 + i, o);
        if (o2) st16(o2 + i, o);
      }
    }
  };
  if (Rq > 0) {
    const float r = rsqrtf(sumsq(l, Rq) / (float)Rq + eps);
    scale_row(l, wq, r, Rq, cq + row * Rq, (T*)nullptr);
  }
  if (Rk > 0) {
    const float r = rsqrtf(sumsq(l + Rq, Rk) / (float)Rk + eps);
    const int64_t slot = slots ? slots[row] : -1;                     // < 0: padding row, nothing to cache
    scale_row(l + Rq, wk, r, Rk, ckv ? ckv + row * Rk : nullptr, (cache && slot >= 0) ? cache + slot * cache_row : nullptr);
  }
}

// One CTA per token.  Rotated pairs are (i, i + P / 2) (neox) or (2 i, 2 i + 1); V elements per access: pairs of neighbours travel together.
struct RopeParams {
  void* q; const void* kv; const void* w; void* cache;
  const int64_t* positions; const int64_t* slots; const float* cos_sin;
  int64_t st, cache_row;        // row stride of q and kv (columns of one matrix)
  int H, D, P, R;               // query heads of D + P, latent width (0: queries alone)
  int neox;
  float eps;
};
template <typename T, int V> VB_DEVICE void rotate_part(const T* src, T* dst, int item, int P, bool neox, const float* cs) {
  const int half = P / 2;
  if constexpr (V == 1) {
    const int e0 = neox ? item : 2 * item, e1 = neox ? item + half : 2 * item + 1;
    const float a = to_f32(src[e0]), b = to_f32(src[e1]), c = cs[item], s = cs[half + item];
    dst[e0] = from_f32<T>(a * c - b * s);
    dst[e1] = from_f32<T>(b * c + a * s);
  } else if (neox) {
    const int i = item * V;
    Vec16<T> a = ld16(src + i), b = ld16(src + half + i);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float x = to_f32(a.e[j]), y = to_f32(b.e[j]), c = cs[i + j], s = cs[half + i + j];
      a.e[j] = from_f32<T>(x * c - y * s);
      b.e[j] = from_f32<T>(y * c + x * s);
    }
    st16(dst + i, a);
    st16(dst + half + i, b);
  } else {
    Vec16<T> a = ld16(src + item * V);
#pragma unroll
    for (int j = 0; j < V; j += 2) {
      const int i = (item * V + j) / 2;
      const float x = to_f32(a.e[j]), y = to_f32(a.e[j + 1]), c = cs[i], s = cs[half + i];
      a.e[j] = from_f32<T>(x * c - y * s);
      a.e[j + 1] = from_f32<T>(y * c + x * s);
    }
    st16(dst + item * V, a);
  }
}
template <typename T, int V>
__global__ void __launch_bounds__(256) latent_rope_cache_kernel(const RopeParams p) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const float* cs = p.P ? p.cos_sin + p.positions[row] * p.P : nullptr;
  const int per = V == 1 || p.neox ? p.P / 2 / V : p.P / V;                 // accesses of one rotated part
  if (p.R > 0) {
    const int64_t slot = p.cache ? p.slots[row] : -1;                       // < 0: padding row, nothing to cache
    const T* c = reinterpret_cast<const T*>(p.kv) + row * p.st;
    const T* w = reinterpret_cast<const T*>(p.w);
    T* dst = reinterpret_cast<T*>(p.cache) + slot * p.cache_row;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < p.R; i += blockDim.x * V) {
      if constexpr (V == 1) { const float f = to_f32(c[i]); ss += f * f; }
      else {
        const Vec16<T> v = ld16(c + i);
#pragma unroll
        for (int j = 0; j < V; ++j) { const float f = to_f32(v.e[j]); ss += f * f; }
      }
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)p.R + p.eps);
    if (slot >= 0) {
      for (int i = threadIdx.x * V; i < p.R; i += blockDim.x * V) {
        if constexpr (V == 1) dst[i] = from_f32<T>(to_f32(c[i]) * r * to_f32(w[i]));
        else {
          Vec16<T> v = ld16(c + i);
          const Vec16<T> g = ld16(w + i);
#pragma unroll
          for (int j = 0; j < V; ++j) v.e[j] = from_f32<T>(to_f32(v.e[j]) * r * to_f32(g.e[j]));
          st16(dst + i, v);
        }
      }
      for (int i = threadIdx.x; i < per; i += blockDim.x) rotate_part<T, V>(c + p.R, dst + p.R, i, p.P, p.neox, cs);
    }
  }
  T* q = reinterpret_cast<T*>(p.q) + row * p.st;
  for (int i = threadIdx.x; i < p.H * per; i += blockDim.x) {
    const int h = i / per;
    T* part = q + (int64_t)h * (p.D + p.P) + p.D;
    rotate_part<T, V>(part, part, i - h * per, p.P, p.neox, cs);
  }
}

constexpr int KT = 32;        // keys per tile: one per lane
constexpr int HB = 8;         // heads per CTA: one per warp

struct SimtParams {
  const void* q; const void* q_pe; const void* cache; void* out;
  const int* block_table; const int* seq_lens; const int* qsl;      // qsl null: request b owns row b (decode)
  int64_t q_st, q_sh, qp_st, qp_sh, o_st, o_sh, bt_stride;
  int B, T, H, R, P, BS;
  int window;                          // > 0: the last `window` keys only
  float scale;
};

// CTA = (token, HB heads); warp = head.  Lane = key for the scores, lane = latent dims lane + 32 i for the output.
template <typename T, int NI>
__global__ void __launch_bounds__(32 * HB) mla_simt_kernel(const SimtParams p) {
  extern __shared__ float sm[];
  const int D = p.R + p.P, LD = D | 1;                 // odd row pitch: lanes walk different banks
  float* ks = sm;                                      // [KT][LD]
  float* qs = ks + KT * LD;                            // [HB][D]
  float* ps = qs + HB * D;                             // [HB][KT]
  pdl_trigger();
  pdl_wait();
  const int tok = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * HB + warp;
  int b = tok, pos;
  if (p.qsl) {
    int lo = 0, hi = p.B;                              // last request whose start is <= tok
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.qsl[mid] <= tok) lo = mid; else hi = mid;
    }
    b = lo;
    const int s = p.qsl[b], e = p.qsl[b + 1];
    if (tok < s || tok >= e) return;                   // bucket padding
    pos = p.seq_lens[b] - (e - s) + (tok - s);
  } else {
    pos = p.seq_lens[b] - 1;
  }
  const T* q = reinterpret_cast<const T*>(p.q);
  const T* qp = reinterpret_cast<const T*>(p.q_pe);
  const T* cache = reinterpret_cast<const T*>(p.cache);
  if (h < p.H)
    for (int d = lane; d < D; d += 32)
      qs[warp * D + d] = p.scale * to_f32(d < p.R ? q[tok * p.q_st + h * p.q_sh + d] : qp[tok * p.qp_st + h * p.qp_sh + (d - p.R)]);
  float acc[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int k0 = p.window > 0 ? max(0, pos - p.window + 1) : 0; k0 <= pos; k0 += KT) {
    __syncthreads();
    const int n = min(KT, pos + 1 - k0);
    for (int j = warp; j < KT; j += blockDim.x >> 5) {
      if (j < n) {
        const int kp = k0 + j;
        const int64_t r = ((int64_t)p.block_table[b * p.bt_stride + kp / p.BS] * p.BS + kp % p.BS) * D;
        for (int d = lane; d < D; d += 32) ks[j * LD + d] = to_f32(cache[r + d]);
      } else {
        for (int d = lane; d < D; d += 32) ks[j * LD + d] = 0.f;
      }
    }
    __syncthreads();
    if (h < p.H) {
      float s = 0.f;
      for (int d = 0; d < D; ++d) s += qs[warp * D + d] * ks[lane * LD + d];
      if (lane >= n) s = -INFINITY;
      const float mn = fmaxf(m, warp_max(s));
      const float e = lane < n ? expf(s - mn) : 0.f;
      const float a = expf(m - mn);                    // m = -inf on the first tile: 0
      l = l * a + warp_sum(e);
      m = mn;
      ps[warp * KT + lane] = e;
      __syncwarp();
#pragma unroll
      for (int i = 0; i < NI; ++i) acc[i] *= a;
      for (int j = 0; j < n; ++j) {
        const float pj = ps[warp * KT + j];
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const int d = lane + 32 * i;
          if (d < p.R) acc[i] += pj * ks[j * LD + d];
        }
      }
      __syncwarp();
    }
  }
  if (h < p.H) {
    const float inv = 1.f / l;
    T* o = reinterpret_cast<T*>(p.out) + tok * p.o_st + h * p.o_sh;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = lane + 32 * i;
      if (d < p.R) o[d] = from_f32<T>(acc[i] * inv);
    }
  }
}

template <typename T, int NI> static int launch_simt(const SimtParams& p, cudaStream_t st) {
  const int D = p.R + p.P;
  const size_t smem = (size_t)(KT * (D | 1) + HB * D + HB * KT) * sizeof(float);
  if (smem > 220 * 1024) return -3;
  auto k = mla_simt_kernel<T, NI>;
  static size_t have = 48 * 1024;
  if (smem > have) {
    if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess) return -5;
    have = 220 * 1024;
  }
  const int warps = p.H < HB ? p.H : HB;
  vb_launch(k, dim3(p.T, (p.H + HB - 1) / HB), dim3(32 * warps), smem, st, p);
  return (int)cudaGetLastError();
}

static bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace latent

// lat [T, Rq + Rk] (row stride lat_stride); Rk = 0: a layer that reads another layer's latents.  cache may be null
// (no cache bound); a cache row is cache_row elements apart.
EXPORT int vb_latent_norm_cache(const void* lat, int64_t lat_stride, int Rq, const void* wq, void* cq, int Rk, const void* wk,
                                void* ckv, void* cache, int64_t cache_row, const int64_t* slots, int T_, float eps, int dtype,
                                cudaStream_t st) {
  using namespace latent;
  if (T_ == 0) return 0;
  DISPATCH_DTYPE(dtype, T, {
    constexpr int V = Vec16<T>::N;
    const bool vec = Rq % V == 0 && Rk % V == 0 && lat_stride % V == 0 && cache_row % V == 0 && al16(lat) && (!wq || al16(wq)) &&
                     (!wk || al16(wk)) && (!cq || al16(cq)) && (!ckv || al16(ckv)) && (!cache || al16(cache));
    const int big = Rq > Rk ? Rq : Rk;
    const int items = vec ? big / V : big;
    const int thr = items >= 256 ? 256 : ((items + 31) / 32) * 32;
    if (vec) vb_launch(latent_norm_cache_kernel<T, V>, dim3(T_), dim3(thr), 0, st, (const T*)lat, lat_stride, Rq, (const T*)wq, (T*)cq, Rk, (const T*)wk, (T*)ckv, (T*)cache, cache_row, slots, eps);
    else vb_launch(latent_norm_cache_kernel<T, 1>, dim3(T_), dim3(thr), 0, st, (const T*)lat, lat_stride, Rq, (const T*)wq, (T*)cq, Rk, (const T*)wk, (T*)ckv, (T*)cache, cache_row, slots, eps);
  });
  return (int)cudaGetLastError();
}

// q: columns of a matrix with row stride st, H heads of D + P; kv: columns [c : R | k_r : P] of the same matrix (R = 0: none).  cache may be
// null (nothing is cached); cos_sin [positions, P].
EXPORT int vb_latent_rope_cache(void* q, const void* kv, int64_t st, int H, int D, int P, int R, const void* w, float eps,
                                const int64_t* positions, const float* cos_sin, int neox, void* cache, int64_t cache_row,
                                const int64_t* slots, int T_, int dtype, cudaStream_t strm) {
  using namespace latent;
  if (T_ == 0) return 0;
  if (P % 2 || (P && (!positions || !cos_sin)) || (cache && (!slots || R == 0 || cache_row < R + P)) || (R > 0 && (!w || !kv))) return -1;
  RopeParams p;
  p.q = q; p.kv = kv; p.w = w; p.cache = cache; p.positions = positions; p.slots = slots; p.cos_sin = cos_sin; p.st = st;
  p.cache_row = cache_row; p.H = H; p.D = D; p.P = P; p.R = R; p.neox = neox; p.eps = eps;
  DISPATCH_DTYPE(dtype, T, {
    constexpr int V = Vec16<T>::N;
    const bool vec = st % V == 0 && D % V == 0 && P % (neox ? 2 * V : V) == 0 && R % V == 0 && cache_row % V == 0 && al16(q) &&
                     (!kv || al16(kv)) && (!w || al16(w)) && (!cache || al16(cache));
    const int parts = H * P / (vec ? (neox ? 2 * V : V) : 2), lat = vec ? R / V : R, items = parts > lat ? parts : lat;
    const int thr = items >= 256 ? 256 : (items < 32 ? 32 : ((items + 31) / 32) * 32);
    if (vec) vb_launch(latent_rope_cache_kernel<T, V>, dim3(T_), dim3(thr), 0, strm, p);
    else vb_launch(latent_rope_cache_kernel<T, 1>, dim3(T_), dim3(thr), 0, strm, p);
  });
  return (int)cudaGetLastError();
}

// q [T, H, R] (absorbed), q_pe [T, H, P] (P = 0: unused), cache [blocks, BS, R + P], out [T, H, R]; window > 0: a token sees its last
// `window` keys
EXPORT int vb_mla_simt(const void* q, const void* q_pe, const void* cache, void* out, const int* block_table, int64_t bt_stride,
                       const int* seq_lens, const int* qsl, int B, int T_, int H, int R, int P, int BS, int64_t q_st,
                       int64_t q_sh, int64_t qp_st, int64_t qp_sh, int64_t o_st, int64_t o_sh, int window, float scale,
                       int dtype, cudaStream_t st) {
  using namespace latent;
  if (T_ == 0 || B == 0) return 0;
  if (R < 1 || R > 1024) return -2;
  SimtParams p;
  p.q = q; p.q_pe = q_pe; p.cache = cache; p.out = out; p.block_table = block_table; p.seq_lens = seq_lens; p.qsl = qsl;
  p.q_st = q_st; p.q_sh = q_sh; p.qp_st = qp_st; p.qp_sh = qp_sh; p.o_st = o_st; p.o_sh = o_sh; p.bt_stride = bt_stride;
  p.B = B; p.T = T_; p.H = H; p.R = R; p.P = P; p.BS = BS; p.window = window; p.scale = scale;
  const int ni = (R + 31) / 32;
  DISPATCH_DTYPE(dtype, T, {
    if (ni <= 2) return launch_simt<T, 2>(p, st);
    if (ni <= 4) return launch_simt<T, 4>(p, st);
    if (ni <= 8) return launch_simt<T, 8>(p, st);
    if (ni <= 16) return launch_simt<T, 16>(p, st);
    return launch_simt<T, 32>(p, st);
  });
  return -1;
}
