// Paged variable-length attention for every shape and dtype (CUDA cores, fp32 arithmetic): key and value widths that differ or
// are no power of two, any number of query heads per KV head, 32-bit models; causal, sliding-window and chunk-local masks,
// sinks, soft cap, ALiBi.  The tensor-core kernels (attention_tc*.cu) take head size 128, attention_simt.cu the 16-bit sizes it
// is tuned for; this one takes the rest, prompts and decode steps alike.
//
// FOLD: every query head attends to the values of several KV heads (its scores are with the keys of its own), one result each in
// 32-bit: what a mix of the heads' weights behind the softmax needs (attention_talk.cu).
//
// CTA = 16 query rows (tokens x heads of one KV head) of one request.  Tiles of 32 keys and values are staged in shared
// memory as fp32; in the scores a lane is a key (rows padded to an odd number of 16-byte units: conflict-free), in P.V a lane
// is an output column.  Only the keys that some row of the tile can see are visited.
#include "common.cuh"

namespace anyattn {

constexpr int ROWS = 16, KEYS = 32, WARPS = 4, RPW = ROWS / WARPS;
constexpr int MAX_D = 512;
constexpr float LOG2E = 1.4426950408889634f;

struct Params {
  const void* q; const void* kv_cache; void* out; float* lse_out;
  const int* block_table; const int* seq_lens; const int* qsl;
  int64_t q_stride, out_stride;
  int bt_stride, Hq, Hkv, D, DV, DC, BS;        // DC: width of a cache row (>= D, DV)
  int window, chunk, causal;
  float scale_log2, soft_cap, out_scale;
  const float* alibi; const float* sinks;
  int c0, nc;                                   // FOLD: value heads c0 .. c0 + nc - 1; out fp32 [T, Hq, nc, DV]
};

VB_HOST_DEVICE int padded(int d) {               // floats of a staged row: 16-byte units, an odd number of them
  const int u = (d + 3) / 4;
  return (u | 1) * 4;
}

template <typename T, int NVD, bool FOLD>
__global__ void __launch_bounds__(WARPS * 32) any_attn_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  const int DP = padded(p.D), D4 = (p.D + 3) / 4, DV = p.DV;
  float* qs = sm;                                // ROWS x DP
  float* ks = qs + ROWS * DP;                    // KEYS x DP
  float* vs = ks + KEYS * DP;                    // KEYS x DV
  float* ps = vs + KEYS * DV;                    // WARPS x KEYS x RPW (KEYS * DV is a multiple of four)
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, hk = FOLD ? blockIdx.y / p.nc : blockIdx.y, G = p.Hq / p.Hkv;
  const int hv = FOLD ? p.c0 + blockIdx.y % p.nc : hk;
  const int q0 = p.qsl ? p.qsl[b] : b, q_len = p.qsl ? p.qsl[b + 1] - q0 : 1;
  const int row0 = blockIdx.x * ROWS, n_rows = min(ROWS, q_len * G - row0);
  if (n_rows <= 0) return;
  const int seq = p.seq_lens[b], base = seq - q_len;
  const int pos_lo = base + row0 / G, pos_hi = base + (row0 + n_rows - 1) / G;
  const int kv_end = p.causal ? pos_hi + 1 : seq;
  int kv_begin = p.window > 0 ? max(0, pos_lo - p.window + 1) : 0;
  if (p.chunk > 0) kv_begin = max(kv_begin, pos_lo / p.chunk * p.chunk);
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
  const T* qb = reinterpret_cast<const T*>(p.q);
  for (int i = threadIdx.x; i < ROWS * DP; i += blockDim.x) {
    const int r = i / DP, d = i - r * DP;
    float x = 0.f;
    if (r < n_rows && d < p.D) x = to_f32(qb[(int64_t)(q0 + (row0 + r) / G) * p.q_stride + (int64_t)(hk * G + (row0 + r) % G) * p.D + d]);
    qs[i] = x;
  }
  float m[RPW], l[RPW], acc[RPW][NVD];
  int qpos[RPW], head[RPW];
#pragma unroll
  for (int j = 0; j < RPW; ++j) {
    const int r = w * RPW + j;
    qpos[j] = r < n_rows ? base + (row0 + r) / G : -1;
    head[j] = hk * G + (row0 + r) % G;
    m[j] = -INFINITY; l[j] = 0.f;
#pragma unroll
    for (int i = 0; i < NVD; ++i) acc[j][i] = 0.f;
  }
  const T* cache = reinterpret_cast<const T*>(p.kv_cache);
  const int* bt = p.block_table + (int64_t)b * p.bt_stride;
  for (int t0 = kv_begin; t0 < kv_end; t0 += KEYS) {
    const int nk = min(KEYS, kv_end - t0);
    __syncthreads();
    // warp w stages keys w, w + 4, ...: lanes along the row
    for (int k = w; k < KEYS; k += WARPS) {
      const bool in = k < nk;
      const T* kr = nullptr;
      const T* vr = nullptr;
      if (in) {
        const int pos = t0 + k;
        const int64_t blk = bt[pos / p.BS];
        kr = cache + (((blk * 2) * p.Hkv + hk) * p.BS + pos % p.BS) * (int64_t)p.DC;
        vr = kr + (int64_t)(p.Hkv + hv - hk) * p.BS * p.DC;
      }
      for (int d = lane; d < DP; d += 32) ks[k * DP + d] = in && d < p.D ? to_f32(kr[d]) : 0.f;
      for (int d = lane; d < DV; d += 32) vs[k * DV + d] = in ? to_f32(vr[d]) : 0.f;
    }
    __syncthreads();
    float s[RPW];
#pragma unroll
    for (int j = 0; j < RPW; ++j) s[j] = 0.f;
    const float4* kr = reinterpret_cast<const float4*>(ks + lane * DP);
    for (int d = 0; d < D4; ++d) {
      const float4 kv = kr[d];
#pragma unroll
      for (int j = 0; j < RPW; ++j) {
        const float4 qv = reinterpret_cast<const float4*>(qs + (w * RPW + j) * DP)[d];
        s[j] += qv.x * kv.x + qv.y * kv.y + qv.z * kv.z + qv.w * kv.w;
      }
    }
    const int kpos = t0 + lane;
    float pr[RPW];
#pragma unroll
    for (int j = 0; j < RPW; ++j) {
      float x = s[j] * p.scale_log2;
      if (p.soft_cap > 0.f) x = p.soft_cap * tanhf(x / (LOG2E * p.soft_cap)) * LOG2E;
      if (p.alibi) x += p.alibi[head[j]] * LOG2E * (float)(kpos - qpos[j]);
      bool ok = qpos[j] >= 0 && lane < nk;
      if (p.causal) ok = ok && kpos <= qpos[j];
      if (p.window > 0) ok = ok && kpos > qpos[j] - p.window && (p.causal || kpos < qpos[j] + p.window);
      if (p.chunk > 0) ok = ok && qpos[j] >= 0 && kpos / p.chunk == qpos[j] / p.chunk;
      x = ok ? x : -INFINITY;
      const float mn = fmaxf(m[j], warp_max(x));
      const float mu = mn == -INFINITY ? 0.f : mn;
      const float a = exp2f(m[j] - mu);
      pr[j] = ok ? exp2f(x - mu) : 0.f;
      m[j] = mn;
      l[j] = l[j] * a + pr[j];                   // per lane; summed at the end
#pragma unroll
      for (int i = 0; i < NVD; ++i) acc[j][i] *= a;
    }
    *reinterpret_cast<float4*>(ps + (w * KEYS + lane) * RPW) = make_float4(pr[0], pr[1], pr[2], pr[3]);
    __syncwarp();
    for (int k = 0; k < nk; ++k) {
      const float4 pk = *reinterpret_cast<const float4*>(ps + (w * KEYS + k) * RPW);
#pragma unroll
      for (int i = 0; i < NVD; ++i) {
        const int d = lane + i * 32;
        const float v = d < DV ? vs[k * DV + d] : 0.f;
        acc[0][i] += pk.x * v; acc[1][i] += pk.y * v; acc[2][i] += pk.z * v; acc[3][i] += pk.w * v;
      }
    }
    __syncwarp();
  }
#pragma unroll
  for (int j = 0; j < RPW; ++j) {
    if (qpos[j] < 0) continue;
    float sum = warp_sum(l[j]);
    float top = m[j];
    if (p.sinks) top = fmaxf(top, p.sinks[head[j]] * LOG2E);
    const float tu = top == -INFINITY ? 0.f : top;
    const float f = exp2f(m[j] - tu);
    sum *= f;
    if (p.sinks) sum += exp2f(p.sinks[head[j]] * LOG2E - tu);
    const float inv = sum > 0.f ? f / sum * p.out_scale : 0.f;
    const int64_t tok = q0 + (row0 + w * RPW + j) / G;
    if constexpr (FOLD) {
      float* o = reinterpret_cast<float*>(p.out) + ((tok * p.Hq + head[j]) * p.nc + (hv - p.c0)) * DV;
#pragma unroll
      for (int i = 0; i < NVD; ++i)
        if (lane + i * 32 < DV) o[lane + i * 32] = acc[j][i] * inv;
      continue;
    }
    T* o = reinterpret_cast<T*>(p.out) + tok * p.out_stride + (int64_t)head[j] * DV;
#pragma unroll
    for (int i = 0; i < NVD; ++i) {
      const int d = lane + i * 32;
      if (d < DV) o[d] = from_f32<T>(acc[j][i] * inv);
    }
    if (p.lse_out && lane == 0) p.lse_out[tok * p.Hq + head[j]] = sum > 0.f ? (tu + log2f(sum)) / LOG2E : -INFINITY;
  }
}

}  // namespace anyattn

namespace anyattn {
template <bool FOLD>
static int launch(const Params& p, int B, int max_rows, int dtype, cudaStream_t st) {
  dim3 grid((max_rows + ROWS - 1) / ROWS, FOLD ? p.Hkv * p.nc : p.Hkv, B);
  const size_t smem = ((size_t)(ROWS + KEYS) * padded(p.D) + (size_t)KEYS * p.DV + WARPS * KEYS * RPW) * 4;
#define GO(N)                                                                                                   \
  do {                                                                                                          \
    auto k = any_attn_kernel<T, N, FOLD>;                                                                       \
    static bool set = false;                                                                                    \
    if (!set) { cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); set = true; } \
    vb_launch(k, grid, dim3(WARPS * 32), smem, st, p);                                                          \
  } while (0)
  DISPATCH_DTYPE(dtype, T, {
    if (p.DV <= 64) GO(2); else if (p.DV <= 128) GO(4); else if (p.DV <= 256) GO(8); else GO(16);
  });
#undef GO
  return (int)cudaGetLastError();
}
}  // namespace anyattn

// kv_cache [blocks, 2, Hkv, BS, DC] (not the transposed-value layout); q [T, Hq * D], out [T, Hq * DV] (token strides free).
// qsl null: one token per request.
EXPORT int vb_any_attention(const void* q, const void* kv_cache, const int* block_table, const int* seq_lens, const int* qsl,
                            void* out, float* lse_out, int B, int max_q_len, int Hq, int Hkv, int D, int DV, int DC, int BS,
                            int64_t q_stride, int64_t out_stride, int bt_stride, int window, int chunk, int causal, float scale,
                            float soft_cap, float out_scale, const float* alibi, const float* sinks, int dtype, cudaStream_t st) {
  using namespace anyattn;
  if (B == 0) return 0;
  if (D < 1 || DV < 1 || D > MAX_D || DV > MAX_D || DC < D || DC < DV || Hq % Hkv) return -1;
  Params p;
  p.q = q; p.kv_cache = kv_cache; p.out = out; p.lse_out = lse_out; p.block_table = block_table; p.seq_lens = seq_lens; p.qsl = qsl;
  p.q_stride = q_stride; p.out_stride = out_stride; p.bt_stride = bt_stride; p.Hq = Hq; p.Hkv = Hkv; p.D = D; p.DV = DV; p.DC = DC;
  p.BS = BS; p.window = window; p.chunk = chunk; p.causal = causal; p.scale_log2 = scale * LOG2E; p.soft_cap = soft_cap;
  p.out_scale = out_scale; p.alibi = alibi; p.sinks = sinks; p.c0 = 0; p.nc = 1;
  return launch<false>(p, B, (qsl ? max_q_len : 1) * (Hq / Hkv), dtype, st);
}

// Causal attention of every query head with the values of KV heads c0 .. c0 + nc - 1: out fp32 [T, Hq, nc, DV].
EXPORT int vb_any_attention_fold(const void* q, const void* kv_cache, const int* block_table, const int* seq_lens, const int* qsl,
                                 float* out, int B, int max_q_len, int Hq, int Hkv, int D, int DV, int DC, int BS, int64_t q_stride,
                                 int bt_stride, int window, float scale, float soft_cap, const float* sinks, int c0, int nc, int dtype,
                                 cudaStream_t st) {
  using namespace anyattn;
  if (B == 0) return 0;
  if (D < 1 || DV < 1 || D > MAX_D || DV > MAX_D || DC < D || DC < DV || Hq % Hkv || c0 < 0 || nc < 1 || c0 + nc > Hkv) return -1;
  Params p;
  p.q = q; p.kv_cache = kv_cache; p.out = out; p.lse_out = nullptr; p.block_table = block_table; p.seq_lens = seq_lens; p.qsl = qsl;
  p.q_stride = q_stride; p.out_stride = 0; p.bt_stride = bt_stride; p.Hq = Hq; p.Hkv = Hkv; p.D = D; p.DV = DV; p.DC = DC; p.BS = BS;
  p.window = window; p.chunk = 0; p.causal = 1; p.scale_log2 = scale * LOG2E; p.soft_cap = soft_cap; p.out_scale = 1.f;
  p.alibi = nullptr; p.sinks = sinks; p.c0 = c0; p.nc = nc;
  return launch<true>(p, B, (qsl ? max_q_len : 1) * (Hq / Hkv), dtype, st);
}
