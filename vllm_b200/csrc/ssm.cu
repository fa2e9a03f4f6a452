// State-space / linear-attention kernels over the paged recurrent-state cache (sm_100a):
//   causal depthwise conv1d with cached window     (Mamba-1/2, gated delta net; prefill, chunked prefill, decode)
//   Mamba-1 selective scan                          (per-channel A, state N <= 32)
//   gated delta rule scan                           (Qwen3-Next GDN: rank-1 corrected state [dk, dv] per head)
//
// Reference ops: csrc/libtorch_stable/mamba/selective_scan_fwd.cu, vllm/model_executor/layers/mamba/ops/
// causal_conv1d.py, fla ops/fused_recurrent (GDN decode).  One design replaces that family here: every op is a varlen kernel driven
// by device-resident `query_start_loc` / `seq_lens` / cache-row ids, reads and writes the request's state row in
// the cache pool in place, and walks the request's tokens in order with the state held in registers — decode is
// the q = 1 case of the same kernel, so there is one code path, no host loop, no `.tolist()`, and every batch shape
// is CUDA-graph capturable.  A linear-time scan keeps all 148 SMs busy because the independent (request, head,
// state-row) warps number in the thousands even for one sequence.
//
// State row of request r (fp32): [ conv window (C x (k-1)) | recurrent state ... ]; `state_stride` floats per row.
#include "common.cuh"

namespace {

VB_DEVICE float silu_f(float x) { return x / (1.f + __expf(-x)); }

// ------------------------------------------------------------------ causal conv1d (+ SiLU), window cached per request
// Thread = V channels x TT consecutive tokens of the batch: the grid depends on the token count alone, and a long prompt is
// spread over all SMs.  A token's request is found from query_start_loc.  The cached window of a request (the last K - 1
// inputs) is read and rewritten by one thread only, the one that has the request's first token; it also takes the tokens
// behind its tile that still look into the old window.  KT: compile-time tap count, 0: any up to MAX_TAPS.
constexpr int MAX_TAPS = 16;
template <typename T, int V> VB_DEVICE void ld_ch(const T* p, float (&v)[V]) {
  if constexpr (V == 2 && sizeof(T) == 2) {
    const float2 f = unpack2<T>(*reinterpret_cast<const uint32_t*>(p));
    v[0] = f.x; v[1] = f.y;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = to_f32(p[i]);
  }
}
template <typename T, int KT, int V>
__global__ void __launch_bounds__(128) causal_conv1d_kernel(const T* __restrict__ x, int64_t x_stride, float* __restrict__ out,
                                                             int64_t out_stride, const T* __restrict__ w,
                                                             const T* __restrict__ bias, float* __restrict__ state,
                                                             int64_t state_stride, const int* __restrict__ qsl,
                                                             const int* __restrict__ seq_lens,
                                                             const int* __restrict__ rows, int64_t rows_stride, int num_reqs,
                                                             int n_tok, int C, int taps, int act, int TT) {
  constexpr int KM = KT ? KT : MAX_TAPS;
  pdl_trigger();
  pdl_wait();
  const int K = KT ? KT : taps;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  const int tile0 = blockIdx.x * TT, tile1 = min(tile0 + TT, n_tok);
  const int total = qsl[num_reqs];
  // last request that starts at or before the tile
  int r = 0;
  for (int lo = 0, hi = num_reqs - 1; lo <= hi;) {
    const int mid = (lo + hi) >> 1;
    if (qsl[mid] <= tile0) { r = mid; lo = mid + 1; } else hi = mid - 1;
  }
  float wr[KM][V], b[V];
#pragma unroll
  for (int j = 0; j < KM; ++j)
#pragma unroll
    for (int v = 0; v < V; ++v) wr[j][v] = j < K ? to_f32(w[(int64_t)(c + v) * K + j]) : 0.f;
#pragma unroll
  for (int v = 0; v < V; ++v) b[v] = bias ? to_f32(bias[c + v]) : 0.f;
  int t = tile0;
  while (t < tile1) {
    if (t >= total) {                                   // padding of a graph bucket
#pragma unroll
      for (int v = 0; v < V; ++v) out[t * out_stride + c + v] = 0.f;
      ++t;
      continue;
    }
    while (t >= qsl[r + 1]) ++r;
    const int t0 = qsl[r], t1 = qsl[r + 1];
    const bool first = t == t0;
    if (!first && t < t0 + K - 1) { t = min(t0 + K - 1, t1); continue; }      // an earlier thread's tokens
    const int end = first ? min(t1, max(tile1, t0 + K - 1)) : min(t1, tile1);
    float win[KM][V];                                   // inputs t - K + 1 .. t - 1
    if (first) {
      const bool has_init = seq_lens[r] - (t1 - t0) > 0;
      const int q = t1 - t0;
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float* st = state + (int64_t)rows[r * rows_stride] * state_stride + (int64_t)(c + v) * (K - 1);
#pragma unroll
        for (int j = 0; j < KM; ++j) win[j][v] = j < K - 1 && has_init ? st[j] : 0.f;
#pragma unroll
        for (int j = 0; j < KM; ++j) {
          if (j >= K - 1) continue;
          const int p = q - (K - 1) + j;                // token of this step, or place j + q of the old window
          float nv = 0.f;
          if (p >= 0) nv = to_f32(x[(int64_t)(t0 + p) * x_stride + c + v]);
          else {
#pragma unroll
            for (int i = 0; i < KM; ++i) if (i == j + q) nv = win[i][v];
          }
          st[j] = nv;
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < KM; ++j) {
        if (j < K - 1) ld_ch<T, V>(x + (int64_t)(t - (K - 1) + j) * x_stride + c, win[j]);
        else {
#pragma unroll
          for (int v = 0; v < V; ++v) win[j][v] = 0.f;
        }
      }
    }
#pragma unroll 4
    for (; t < end; ++t) {
      float in[V], acc[V];
      ld_ch<T, V>(x + (int64_t)t * x_stride + c, in);
#pragma unroll
      for (int v = 0; v < V; ++v) {
        acc[v] = b[v];
#pragma unroll
        for (int j = 0; j < KM; ++j) acc[v] += wr[j][v] * (j == K - 1 ? in[v] : win[j][v]);
        if (act) acc[v] = silu_f(acc[v]);
#pragma unroll
        for (int j = 0; j < KM - 1; ++j) win[j][v] = j == K - 2 ? in[v] : win[j + 1][v];
      }
      float* o = out + (int64_t)t * out_stride + c;
      if constexpr (V == 2) *reinterpret_cast<float2*>(o) = make_float2(acc[0], acc[1]);
      else o[0] = acc[0];
    }
  }
}

// ------------------------------------------------------------------ Mamba-1 selective scan
// thread = (request, channel); h[N] in registers.  x, dt: [T, di] fp32 (dt already softplus'ed); B, C: [T, N] fp32;
// A: [di, N] (negative); D: [di]; z: optional [T, 2*di]-strided gate (silu) — y = (scan + D x) * silu(z).
template <int N>
__global__ void __launch_bounds__(128) selective_scan_kernel(const float* __restrict__ x, const float* __restrict__ dt,
                                                              const float* __restrict__ Bm, const float* __restrict__ Cm,
                                                              const float* __restrict__ A, const float* __restrict__ D,
                                                              float* __restrict__ y, float* __restrict__ state,
                                                              int64_t state_stride, int64_t state_off,
                                                              const int* __restrict__ qsl, const int* __restrict__ seq_lens,
                                                              const int* __restrict__ rows, int64_t rows_stride, int di) {
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x;
  const int d = blockIdx.y * blockDim.x + threadIdx.x;
  const int t0 = qsl[r], t1 = qsl[r + 1];
  if (d >= di || t1 <= t0) return;
  const bool has_init = seq_lens[r] - (t1 - t0) > 0;
  float* st = state + (int64_t)rows[r * rows_stride] * state_stride + state_off + (int64_t)d * N;
  float h[N], a[N];
#pragma unroll
  for (int n = 0; n < N; ++n) { h[n] = has_init ? st[n] : 0.f; a[n] = A[(int64_t)d * N + n]; }
  const float dd = D[d];
  for (int t = t0; t < t1; ++t) {
    const float dtv = dt[(int64_t)t * di + d], xv = x[(int64_t)t * di + d];
    const float dx = dtv * xv;
    float acc = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      h[n] = __expf(dtv * a[n]) * h[n] + dx * Bm[(int64_t)t * N + n];
      acc += h[n] * Cm[(int64_t)t * N + n];
    }
    y[(int64_t)t * di + d] = acc + dd * xv;
  }
#pragma unroll
  for (int n = 0; n < N; ++n) st[n] = h[n];
}

// ------------------------------------------------------------------ gated delta rule scan (GDN)
// warp = (request, value head, column j of the [dk, dv] state); lane holds KPL = dk / 32 rows of that column.
//   S *= exp(g);  delta_j = (v_j - Σ_i S[i,j] k_i) β;  S[i,j] += k_i delta_j;  o_j = Σ_i S[i,j] q_i
// q, k: [T, nv, dk] fp32 (already l2-normalised / scaled / repeated to value heads); v: [T, nv, dv]; g, beta: [T, nv].
template <int KPL>
__global__ void __launch_bounds__(256) gdn_scan_kernel(const float* __restrict__ q, const float* __restrict__ k,
                                                        const float* __restrict__ v, const float* __restrict__ g,
                                                        const float* __restrict__ beta, float* __restrict__ o,
                                                        float* __restrict__ state, int64_t state_stride, int64_t state_off,
                                                        const int* __restrict__ qsl, const int* __restrict__ seq_lens,
                                                        const int* __restrict__ rows, int64_t rows_stride, int nv, int dv) {
  pdl_trigger();
  pdl_wait();
  constexpr int DK = KPL * 32;
  const int lane = threadIdx.x & 31;
  const int r = blockIdx.y;
  const int wid = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);      // (head, j)
  const int t0 = qsl[r], t1 = qsl[r + 1];
  if (wid >= nv * dv || t1 <= t0) return;
  const int hh = wid / dv, j = wid % dv;
  const bool has_init = seq_lens[r] - (t1 - t0) > 0;
  // state layout [nv, dk, dv]: element (i, j) at ((hh * DK + i) * dv + j); lane owns rows i = lane + 32 * u
  float* st = state + (int64_t)rows[r * rows_stride] * state_stride + state_off + (int64_t)hh * DK * dv + j;
  float S[KPL];
#pragma unroll
  for (int u = 0; u < KPL; ++u) S[u] = has_init ? st[(int64_t)(lane + 32 * u) * dv] : 0.f;
  for (int t = t0; t < t1; ++t) {
    const float* kp = k + ((int64_t)t * nv + hh) * DK;
    const float* qp = q + ((int64_t)t * nv + hh) * DK;
    const float decay = __expf(g[(int64_t)t * nv + hh]);
    float kk[KPL], mem = 0.f;
#pragma unroll
    for (int u = 0; u < KPL; ++u) {
      kk[u] = kp[lane + 32 * u];
      S[u] *= decay;
      mem += S[u] * kk[u];
    }
    mem = warp_sum(mem);
    const float delta = (v[((int64_t)t * nv + hh) * dv + j] - mem) * beta[(int64_t)t * nv + hh];
    float acc = 0.f;
#pragma unroll
    for (int u = 0; u < KPL; ++u) {
      S[u] += kk[u] * delta;
      acc += S[u] * qp[lane + 32 * u];
    }
    acc = warp_sum(acc);
    if (lane == 0) o[((int64_t)t * nv + hh) * dv + j] = acc;
  }
#pragma unroll
  for (int u = 0; u < KPL; ++u) st[(int64_t)(lane + 32 * u) * dv] = S[u];
}

}  // namespace

// x: [T, C], out: [T, C] fp32 (rows behind the last request are zeroed); state rows hold the (k-1)-window at offset 0 ([C, k-1] fp32).
// rows: cache-row id of each request (block_table[:, 0], int32, stride rows_stride).
EXPORT int vb_causal_conv1d(const void* x, int64_t x_stride, float* out, int64_t out_stride, const void* w, const void* bias,
                            float* state, int64_t state_stride, const int* qsl, const int* seq_lens, const int* rows,
                            int64_t rows_stride, int num_reqs, int n_tok, int C, int K, int act, int dtype, cudaStream_t st) {
  if (num_reqs == 0 || n_tok == 0) return 0;
  if (K < 1 || K > MAX_TAPS) return -1;
  // tokens per thread: one where most requests bring one (each is a walk through the state of its own), more in prompts
  const int tile = n_tok <= 2 * num_reqs ? 1 : n_tok <= 16 * num_reqs ? 4 : 16;
  const bool two = dtype != DT_F32 && C % 2 == 0 && x_stride % 2 == 0 && out_stride % 2 == 0 &&
                   (reinterpret_cast<uintptr_t>(x) & 3) == 0 && (reinterpret_cast<uintptr_t>(out) & 7) == 0;
  dim3 grid((n_tok + tile - 1) / tile, (C + (two ? 255 : 127)) / (two ? 256 : 128));
#define GO(KK)                                                                                                                  \
  do {                                                                                                                          \
    if (two) GO2(KK, 2); else GO2(KK, 1);                                                                                       \
  } while (0)
#define GO2(KK, VV) vb_launch(causal_conv1d_kernel<TT, KK, VV>, grid, dim3(128), 0, st, reinterpret_cast<const TT*>(x), x_stride, out, \
                         out_stride, reinterpret_cast<const TT*>(w), reinterpret_cast<const TT*>(bias), state, state_stride,   \
                         qsl, seq_lens, rows, rows_stride, num_reqs, n_tok, C, K, act, tile)
  DISPATCH_DTYPE(dtype, TT, {
    if (K == 2) GO(2); else if (K == 3) GO(3); else if (K == 4) GO(4); else GO(0);
  });
#undef GO
#undef GO2
  return (int)cudaGetLastError();
}

EXPORT int vb_selective_scan(const float* x, const float* dt, const float* B, const float* C, const float* A, const float* D,
                             float* y, float* state, int64_t state_stride, int64_t state_off, const int* qsl,
                             const int* seq_lens, const int* rows, int64_t rows_stride, int num_reqs, int di, int N,
                             cudaStream_t st) {
  if (num_reqs == 0) return 0;
  dim3 grid(num_reqs, (di + 127) / 128);
#define GO(NN) vb_launch(selective_scan_kernel<NN>, grid, dim3(128), 0, st, x, dt, B, C, A, D, y, state, state_stride, \
                         state_off, qsl, seq_lens, rows, rows_stride, di)
  if (N == 16) GO(16); else if (N == 8) GO(8); else if (N == 32) GO(32); else return -1;
#undef GO
  return (int)cudaGetLastError();
}

EXPORT int vb_gdn_scan(const float* q, const float* k, const float* v, const float* g, const float* beta, float* o,
                       float* state, int64_t state_stride, int64_t state_off, const int* qsl, const int* seq_lens,
                       const int* rows, int64_t rows_stride, int num_reqs, int nv, int dk, int dv, cudaStream_t st) {
  if (num_reqs == 0) return 0;
  if (dk % 32 || dk > 256) return -1;
  const int wpb = 8;
  dim3 grid((nv * dv + wpb - 1) / wpb, num_reqs);
#define GO(P) vb_launch(gdn_scan_kernel<P>, grid, dim3(wpb * 32), 0, st, q, k, v, g, beta, o, state, state_stride, state_off, \
                        qsl, seq_lens, rows, rows_stride, nv, dv)
  switch (dk / 32) {
    case 1: GO(1); break;
    case 2: GO(2); break;
    case 4: GO(4); break;
    case 8: GO(8); break;
    default: return -1;
  }
#undef GO
  return (int)cudaGetLastError();
}
