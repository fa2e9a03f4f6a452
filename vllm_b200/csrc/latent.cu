// Latent attention (MLA) around the tensor-core kernels: the fused down-projection epilogue, and a variable-length
// attention over the latent cache for every size and dtype the tcgen05 kernels (mla_decode.cu, mla_prefill.cu) do not
// take: fp32, latent widths that are not multiples of 8, wide heads.
//
//   latent_norm_cache   [c_q | c_kv] (one GEMM) → rmsnorm of both halves; c_kv goes straight into its page
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

constexpr int KT = 32;        // keys per tile: one per lane
constexpr int HB = 8;         // heads per CTA: one per warp

struct SimtParams {
  const void* q; const void* q_pe; const void* cache; void* out;
  const int* block_table; const int* seq_lens; const int* qsl;      // qsl null: request b owns row b (decode)
  int64_t q_st, q_sh, qp_st, qp_sh, o_st, o_sh, bt_stride;
  int B, T, H, R, P, BS;
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
  for (int k0 = 0; k0 <= pos; k0 += KT) {
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

// q [T, H, R] (absorbed), q_pe [T, H, P] (P = 0: unused), cache [blocks, BS, R + P], out [T, H, R]
EXPORT int vb_mla_simt(const void* q, const void* q_pe, const void* cache, void* out, const int* block_table, int64_t bt_stride,
                       const int* seq_lens, const int* qsl, int B, int T_, int H, int R, int P, int BS, int64_t q_st,
                       int64_t q_sh, int64_t qp_st, int64_t qp_sh, int64_t o_st, int64_t o_sh, float scale, int dtype,
                       cudaStream_t st) {
  using namespace latent;
  if (T_ == 0 || B == 0) return 0;
  if (R < 1 || R > 1024) return -2;
  SimtParams p;
  p.q = q; p.q_pe = q_pe; p.cache = cache; p.out = out; p.block_table = block_table; p.seq_lens = seq_lens; p.qsl = qsl;
  p.q_st = q_st; p.q_sh = q_sh; p.qp_st = qp_st; p.qp_sh = qp_sh; p.o_st = o_st; p.o_sh = o_sh; p.bt_stride = bt_stride;
  p.B = B; p.T = T_; p.H = H; p.R = R; p.P = P; p.BS = BS; p.scale = scale;
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
