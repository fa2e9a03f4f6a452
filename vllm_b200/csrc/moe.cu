// Mixture-of-experts routing / dispatch / combine kernels (decode-sized batches stay entirely on the device:
// no host sync, CUDA-graph capturable).  The expert GEMMs themselves are the grouped mode of gemm_tc.cu.
//
// Reference counterparts: csrc/moe/topk_softmax_kernels.cu, moe_align_sum_kernels.cu, moe_permute_unpermute_op.cu
// (here: routing probabilities + top-k in one warp per token; counting sort of (token, slot) pairs by expert with
// an inverse map; weighted un-permute that sums a token's k expert outputs in a fixed order → deterministic).
#include "common.cuh"

namespace moe {

constexpr int MAX_E_PER_LANE = 16;   // experts <= 512

// one warp per token: softmax over E logits, pick the k largest, optionally renormalise
template <typename T>
__global__ void topk_softmax_kernel(const T* __restrict__ logits, float* __restrict__ out_w, int* __restrict__ out_ids,
                                    int n_tokens, int E, int k, int renorm, float scale) {
  pdl_trigger();
  pdl_wait();
  const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (warp >= n_tokens) return;
  const T* row = logits + (size_t)warp * E;
  float v[MAX_E_PER_LANE];
  float mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < MAX_E_PER_LANE; ++i) {
    const int e = lane + i * 32;
    v[i] = e < E ? to_f32(row[e]) : -INFINITY;
    mx = fmaxf(mx, v[i]);
  }
  mx = warp_max(mx);
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < MAX_E_PER_LANE; ++i) {
    const int e = lane + i * 32;
    v[i] = e < E ? __expf(v[i] - mx) : 0.f;
    sum += v[i];
  }
  sum = warp_sum(sum);
  const float inv = 1.f / sum;
  float picked_sum = 0.f;
  float my_w = 0.f; int my_id = 0;
  for (int j = 0; j < k; ++j) {
    float best = -1.f; int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < MAX_E_PER_LANE; ++i) {
      const int e = lane + i * 32;
      if (e < E && (v[i] > best)) { best = v[i]; bi = e; }     // lowest index wins ties inside a lane
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
    }
    if ((bi & 31) == lane) v[bi >> 5] = -1.f;                   // remove the winner
    if (lane == j) { my_w = best * inv; my_id = bi; }
    picked_sum += best * inv;
  }
  if (lane < k) {
    out_w[(size_t)warp * k + lane] = (renorm ? my_w / picked_sum : my_w) * scale;
    out_ids[(size_t)warp * k + lane] = my_id;
  }
}

// Router with sigmoid or softmax scores, a selection bias and group-limited choice; one CTA per token, fp32 throughout.
//   logits: given ([T, E] fp32), or computed here from x [T, H] and w [E, H] (one warp per expert, decode batches)
//   choice score = score + bias;  a group (one of n_group contiguous runs) is ranked by the sum of its two best choice
//   scores (group_top2) or by its best;  the k best experts of the `keep` best groups are taken, the lowest
//   index winning ties;  weight = score WITHOUT the bias (optionally renormalised) * scale
template <typename TX, typename TW>
__global__ void __launch_bounds__(512)
grouped_topk_kernel(const float* __restrict__ logits, const TX* __restrict__ x, const TW* __restrict__ w, int H,
                    const float* __restrict__ bias, float* __restrict__ out_w, int* __restrict__ out_ids, int E, int k,
                    int n_group, int keep, int group_top2, int softmax, int renorm, float scale) {
  extern __shared__ float smf[];
  float* score = smf;               // [E]
  float* choice = score + E;        // [E]
  float* gs = choice + E;           // [n_group]
  float* xs = gs + n_group;         // [H] when the logits are computed here
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  if (logits) {
    for (int e = threadIdx.x; e < E; e += blockDim.x) score[e] = logits[(int64_t)t * E + e];
  } else {
    const TX* xr = x + (int64_t)t * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) xs[i] = to_f32(xr[i]);
    __syncthreads();
    constexpr int V = Vec16<TW>::N;
    const bool vec = H % V == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0;
    constexpr int EB = 4;                       // experts of a warp in flight together
    for (int e0 = warp * EB; e0 < E; e0 += n_warps * EB) {
      float a[EB] = {};
      if (vec) {
        for (int i = lane * V; i < H; i += 32 * V) {
          Vec16<TW> wv[EB];
#pragma unroll
          for (int u = 0; u < EB; ++u) wv[u] = ld16(w + (int64_t)min(e0 + u, E - 1) * H + i);
#pragma unroll
          for (int j = 0; j < V; ++j) {
            const float xv = xs[i + j];
#pragma unroll
            for (int u = 0; u < EB; ++u) a[u] += xv * to_f32(wv[u].e[j]);
          }
        }
      } else {
        for (int i = lane; i < H; i += 32)
#pragma unroll
          for (int u = 0; u < EB; ++u) a[u] += xs[i] * to_f32(w[(int64_t)min(e0 + u, E - 1) * H + i]);
      }
#pragma unroll
      for (int u = 0; u < EB; ++u) {
        a[u] = warp_sum(a[u]);
        if (lane == 0 && e0 + u < E) score[e0 + u] = a[u];
      }
    }
  }
  __syncthreads();
  if (softmax) {
    float mx = -INFINITY;
    for (int e = threadIdx.x; e < E; e += blockDim.x) mx = fmaxf(mx, score[e]);
    mx = warp_max(mx);
    if (lane == 0) red[warp] = mx;
    __syncthreads();
    mx = warp_max(lane < n_warps ? red[lane] : -INFINITY);
    __syncthreads();
    float sum = 0.f;
    for (int e = threadIdx.x; e < E; e += blockDim.x) { score[e] = expf(score[e] - mx); sum += score[e]; }
    const float inv = 1.f / block_sum(sum, red);
    for (int e = threadIdx.x; e < E; e += blockDim.x) score[e] *= inv;
  } else {
    for (int e = threadIdx.x; e < E; e += blockDim.x) score[e] = 1.f / (1.f + expf(-score[e]));
  }
  for (int e = threadIdx.x; e < E; e += blockDim.x) choice[e] = score[e] + (bias ? bias[e] : 0.f);
  __syncthreads();
  if (warp) return;                 // the choice is one warp's work
  auto argmax = [&](const float* v, int n) -> int {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int i = lane; i < n; i += 32)
      if (v[i] > best) { best = v[i]; bi = i; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
    }
    return bi;                      // 0x7fffffff: nothing above -inf is left
  };
  if (n_group > 1) {
    const int gsz = E / n_group;
    for (int g = lane; g < n_group; g += 32) {
      float a = -INFINITY, b = -INFINITY;
      for (int i = 0; i < gsz; ++i) {
        const float c = choice[g * gsz + i];
        if (c > a) { b = a; a = c; } else if (c > b) { b = c; }
      }
      gs[g] = group_top2 && gsz > 1 ? a + b : a;
    }
    __syncwarp();
    // drop the worst groups: what the keep-th best leaves behind.  A taken group is marked by -inf.
    for (int n = 0; n < keep; ++n) {
      const int g = argmax(gs, n_group);
      __syncwarp();
      if (lane == 0 && g < n_group) gs[g] = -INFINITY;
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (gs[e / gsz] != -INFINITY) choice[e] = -INFINITY;
    __syncwarp();
  }
  float wsum = 0.f, mine = 0.f;
  for (int j = 0; j < k; ++j) {
    int e = argmax(choice, E);
    if (e >= E) e = 0;              // fewer than k candidates: cannot happen for a valid configuration
    const float s = score[e];
    wsum += s;
    __syncwarp();
    if (lane == 0) {
      choice[e] = -INFINITY;
      out_ids[(int64_t)t * k + j] = e;
      if (!renorm) out_w[(int64_t)t * k + j] = s * scale;
    }
    if (lane == (j & 31)) mine = s;
    if (renorm && ((j & 31) == 31 || j == k - 1) && lane <= (j & 31)) out_w[(int64_t)t * k + (j & ~31) + lane] = mine;
    __syncwarp();
  }
  if (renorm)
    for (int j = lane; j < k; j += 32) out_w[(int64_t)t * k + j] *= scale / (wsum + 1e-20f);
}

// Grouped GEMM on the CUDA cores for what the tcgen05 kernel (gemm_tc.cu) does not take — fp32, or rows that are not
// 16-byte multiples:  y[r, n] = act(sum_k x[tok(r), k] * w[e(r), n, k]), rows sorted by expert.  64 x 64 tiles; grid.y
// enumerates (expert, row tile) pairs, found from `offs` on the device.
constexpr int GT = 64, GK = 16;
template <typename T>
__global__ void __launch_bounds__(256)
grouped_simt_kernel(const T* __restrict__ x, const T* __restrict__ w, T* __restrict__ y, const int* __restrict__ offs,
                    const int* __restrict__ row_tok, int N, int K, int E, int act) {
  __shared__ float as[GK][GT + 4], bs[GK][GT + 4];
  pdl_trigger();
  pdl_wait();
  int tile = blockIdx.y, e = 0, lo = 0, hi = 0;
  for (; e < E; ++e) {
    lo = offs[e]; hi = offs[e + 1];
    const int nt = (hi - lo + GT - 1) / GT;
    if (tile < nt) break;
    tile -= nt;
  }
  if (e == E) return;
  const int r0 = lo + tile * GT, n0 = blockIdx.x * GT;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += GK) {
    for (int i = threadIdx.x; i < GT * GK; i += 256) {
      const int r = i / GK, kk = i % GK, row = r0 + r, n = n0 + r, kc = k0 + kk;
      as[kk][r] = (row < hi && kc < K) ? to_f32(x[(int64_t)(row_tok ? row_tok[row] : row) * K + kc]) : 0.f;
      bs[kk][r] = (n < N && kc < K) ? to_f32(w[((int64_t)e * N + n) * K + kc]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < GK; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = as[kk][ty * 4 + i]; b[i] = bs[kk][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * b[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = r0 + ty * 4 + i, n = n0 + tx * 4 + j;
      float v = acc[i][j];
      if (act == 2) { v = fmaxf(v, 0.f); v *= v; }
      if (row < hi && n < N) y[(int64_t)row * N + n] = from_f32<T>(v);
    }
}

// counting sort of R = T*k (token, slot) pairs by (mapped) expert id.  One CTA.
//   ids[i]  : global expert of pair i;  emap (optional): global → local expert or -1 (not on this rank)
//   sorted_tok[p] : token of the pair placed at sorted position p;  inv[i] : sorted position of pair i (or -1)
//   offs[e] : first sorted position of local expert e;  offs[E] = number of valid pairs
__global__ void align_kernel(const int* __restrict__ ids, const int* __restrict__ emap, int* __restrict__ sorted_tok,
                             int* __restrict__ inv, int* __restrict__ offs, int R, int k, int E,
                             int* __restrict__ sorted_pair) {
  extern __shared__ int sm[];
  int* cnt = sm;            // [E]
  int* start = sm + E;      // [E + 1]
  pdl_trigger();
  pdl_wait();
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < R; i += blockDim.x) {
    int e = ids[i];
    if (emap) e = emap[e];
    if (e >= 0) atomicAdd(&cnt[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int acc = 0;
    for (int e = 0; e < E; ++e) { start[e] = acc; offs[e] = acc; acc += cnt[e]; cnt[e] = 0; }
    start[E] = acc; offs[E] = acc;
  }
  __syncthreads();
  // placement: the order of pairs inside one expert's segment is arbitrary (atomic cursor) — every row of the
  // grouped GEMM is computed independently and the combine step goes through `inv`, so results do not depend on it
  for (int i = threadIdx.x; i < R; i += blockDim.x) {
    int e = ids[i];
    if (emap) e = emap[e];
    if (e < 0) { inv[i] = -1; continue; }
    const int p = start[e] + atomicAdd(&cnt[e], 1);
    sorted_tok[p] = i / k;
    if (sorted_pair) sorted_pair[p] = i;
    inv[i] = p;
  }
  // sorted positions past the valid pairs (padding rows of the activation buffer) point at token 0
  for (int p = start[E] + threadIdx.x; p < R; p += blockDim.x) { sorted_tok[p] = 0; if (sorted_pair) sorted_pair[p] = 0; }
}

// Tail of the fused MoE combine: acc (fp32, every rank holds the complete sum after the multimem.red epilogue of the
// w2 grouped GEMM) + residual → new residual, RMSNorm → out; acc is zeroed for its next use.  One CTA per token.
template <typename T, bool GEMMA>
__global__ void __launch_bounds__(1024) moe_finish_kernel(float* __restrict__ acc, T* __restrict__ residual,
                                                           const T* __restrict__ w, T* __restrict__ out, int H, float eps) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t row = blockIdx.x;
  float* a = acc + row * H;
  T* r = residual ? residual + row * H : nullptr;
  constexpr int MAXV4 = 8;                     // float4 per thread kept in registers (H <= 1024 * 8 * 4)
  float4 v[MAXV4];
  float ss = 0.f;
  const int nv = H / 4;
#pragma unroll
  for (int i = 0; i < MAXV4; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nv) {
      v[i] = *reinterpret_cast<const float4*>(a + vi * 4);
      *reinterpret_cast<float4*>(a + vi * 4) = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r) {
        const uint2 rv = *reinterpret_cast<const uint2*>(r + vi * 4);
        const float2 r0 = unpack2<T>(rv.x), r1 = unpack2<T>(rv.y);
        // the stream is kept in T: round the sum through T like the unfused path
        v[i].x = to_f32(from_f32<T>(v[i].x)) + r0.x; v[i].y = to_f32(from_f32<T>(v[i].y)) + r0.y;
        v[i].z = to_f32(from_f32<T>(v[i].z)) + r1.x; v[i].w = to_f32(from_f32<T>(v[i].w)) + r1.y;
        uint2 o;
        o.x = pack2<T>(v[i].x, v[i].y); o.y = pack2<T>(v[i].z, v[i].w);
        *reinterpret_cast<uint2*>(r + vi * 4) = o;
        const float2 q0 = unpack2<T>(o.x), q1 = unpack2<T>(o.y);
        v[i] = make_float4(q0.x, q0.y, q1.x, q1.y);
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
  }
  if (w == nullptr) {                          // no norm: out = combined (+ residual) in T
#pragma unroll
    for (int i = 0; i < MAXV4; ++i) {
      const int vi = threadIdx.x + i * blockDim.x;
      if (vi < nv) {
        uint2 o;
        o.x = pack2<T>(v[i].x, v[i].y); o.y = pack2<T>(v[i].z, v[i].w);
        *reinterpret_cast<uint2*>(out + row * H + vi * 4) = o;
      }
    }
    return;
  }
  ss = block_sum(ss, red);
  const float inv = rsqrtf(ss / (float)H + eps);
#pragma unroll
  for (int i = 0; i < MAXV4; ++i) {
    const int vi = threadIdx.x + i * blockDim.x;
    if (vi < nv) {
      const uint2 wv = *reinterpret_cast<const uint2*>(w + vi * 4);
      float2 w0 = unpack2<T>(wv.x), w1 = unpack2<T>(wv.y);
      if (GEMMA) { w0.x += 1.f; w0.y += 1.f; w1.x += 1.f; w1.y += 1.f; }
      uint2 o;
      o.x = pack2<T>(v[i].x * inv * w0.x, v[i].y * inv * w0.y);
      o.y = pack2<T>(v[i].z * inv * w1.x, v[i].w * inv * w1.y);
      *reinterpret_cast<uint2*>(out + row * H + vi * 4) = o;
    }
  }
}

// out[t, :] = sum_j w[t, j] * y[inv[t*k + j], :]   (pairs not computed on this rank contribute 0)
template <typename T>
__global__ void combine_kernel(const T* __restrict__ y, const int* __restrict__ inv, const float* __restrict__ w,
                               T* __restrict__ out, int H, int k) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  for (int g = threadIdx.x; g < H / 8; g += blockDim.x) {
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
    for (int j = 0; j < k; ++j) {
      const int p = inv[t * k + j];
      if (p < 0) continue;
      const float wj = w[t * k + j];
      const Vec16<T> v = ld16(y + (size_t)p * H + g * 8);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] += wj * to_f32(v.e[e]);
    }
    Vec16<T> o;
#pragma unroll
    for (int e = 0; e < 8; ++e) o.e[e] = from_f32<T>(acc[e]);
    st16(out + (size_t)t * H + g * 8, o);
  }
}

// xs[p, :] = x[sorted_tok[p], :]
template <typename T>
__global__ void gather_kernel(const T* __restrict__ x, const int* __restrict__ sorted_tok, T* __restrict__ xs, int H) {
  pdl_trigger();
  pdl_wait();
  const int p = blockIdx.x;
  const T* src = x + (size_t)sorted_tok[p] * H;
  for (int g = threadIdx.x; g < H / 8; g += blockDim.x) st16(xs + (size_t)p * H + g * 8, ld16(src + g * 8));
}

}  // namespace moe

EXPORT int vb_moe_topk_softmax(const void* logits, float* out_w, int* out_ids, int n_tokens, int E, int k, int renorm,
                               float scale, int dtype, cudaStream_t st) {
  if (E > 32 * moe::MAX_E_PER_LANE || k > 32) return -1;
  const int threads = 128, warps_per_block = threads / 32;
  dim3 grid((n_tokens + warps_per_block - 1) / warps_per_block);
  DISPATCH_DTYPE(dtype, T, {
    vb_launch(moe::topk_softmax_kernel<T>, grid, dim3(threads), 0, st, (const T*)logits, out_w, out_ids, n_tokens, E, k,
              renorm, scale);
  });
  return (int)cudaGetLastError();
}

// x / w null: `logits` are given.  dtypes: x fp32 or the model dtype (x_f32), w the model dtype.
EXPORT int vb_moe_grouped_topk(const float* logits, const void* x, int x_f32, const void* w, int H, const float* bias,
                               float* out_w, int* out_ids, int n_tokens, int E, int k, int n_group, int keep, int group_top2,
                               int softmax, int renorm, float scale, int dtype, cudaStream_t st) {
  if (n_tokens == 0) return 0;
  if (E < 1 || E > 4096 || k < 1 || k > E || n_group < 1 || E % n_group || keep < 1 || keep > n_group) return -1;
  if (!logits && (!x || !w)) return -1;
  const size_t smem = (size_t)(2 * E + n_group + (logits ? 0 : H)) * sizeof(float);
  if (smem > 48 * 1024) return -3;
  const int thr = logits ? (E > 128 ? 256 : 64) : (E > 32 ? 512 : 256);
#define GO(TX, TW) vb_launch(moe::grouped_topk_kernel<TX, TW>, dim3(n_tokens), dim3(thr), smem, st, logits, (const TX*)x, (const TW*)w, H, bias, out_w, out_ids, E, k, n_group, keep, group_top2, softmax, renorm, scale)
  DISPATCH_DTYPE(dtype, T, {
    if (x_f32) GO(float, T); else GO(T, T);
  });
#undef GO
  return (int)cudaGetLastError();
}

// x [*, K] read through row_tok (null: x is already in sorted order), w [E, N, K], y [R, N]; act: 0 none, 2 squared ReLU
EXPORT int vb_moe_grouped_simt(const void* x, const void* w, void* y, const int* offs, const int* row_tok, int R, int N, int K,
                               int E, int act, int dtype, cudaStream_t st) {
  if (R == 0) return 0;
  if (act != 0 && act != 2) return -1;
  const dim3 grid((N + moe::GT - 1) / moe::GT, R / moe::GT + (E < R ? E : R));
  DISPATCH_DTYPE(dtype, T, {
    vb_launch(moe::grouped_simt_kernel<T>, grid, dim3(256), 0, st, (const T*)x, (const T*)w, (T*)y, offs, row_tok, N, K, E, act);
  });
  return (int)cudaGetLastError();
}

EXPORT int vb_moe_align2(const int* ids, const int* emap, int* sorted_tok, int* inv, int* offs, int R, int k, int E,
                         int* sorted_pair, cudaStream_t st) {
  if (E > 4096) return -1;
  vb_launch(moe::align_kernel, dim3(1), dim3(R > 4096 ? 1024 : 256), (size_t)(2 * E + 1) * sizeof(int), st, ids, emap, sorted_tok, inv, offs,
            R, k, E, sorted_pair);
  return (int)cudaGetLastError();
}
EXPORT int vb_moe_align(const int* ids, const int* emap, int* sorted_tok, int* inv, int* offs, int R, int k, int E,
                        cudaStream_t st) {
  return vb_moe_align2(ids, emap, sorted_tok, inv, offs, R, k, E, nullptr, st);
}

// out = RMSNorm(acc + residual) (norm_w may be null: out = acc (+ residual)); residual updated in place; acc zeroed
EXPORT int vb_moe_finish(float* acc, void* residual, const void* norm_w, void* out, int T_, int H, float eps, int gemma,
                         int dtype, cudaStream_t st) {
  if (T_ == 0) return 0;
  if (dtype == DT_F32 || H % 4 || H > 1024 * 8 * 4) return -1;
  int thr = ((H / 4 + 7) / 8 + 31) / 32 * 32;
  thr = thr < 64 ? 64 : (thr > 1024 ? 1024 : thr);
  DISPATCH_HALF(dtype, T, {
    if (gemma) vb_launch(moe::moe_finish_kernel<T, true>, dim3(T_), dim3(thr), 0, st, acc, (T*)residual, (const T*)norm_w, (T*)out, H, eps);
    else vb_launch(moe::moe_finish_kernel<T, false>, dim3(T_), dim3(thr), 0, st, acc, (T*)residual, (const T*)norm_w, (T*)out, H, eps);
  });
  return (int)cudaGetLastError();
}

EXPORT int vb_moe_combine(const void* y, const int* inv, const float* w, void* out, int T_, int H, int k, int dtype,
                          cudaStream_t st) {
  if (H % 8) return -1;
  DISPATCH_HALF(dtype, T, {
    vb_launch(moe::combine_kernel<T>, dim3(T_), dim3(128), 0, st, (const T*)y, inv, w, (T*)out, H, k);
  });
  return (int)cudaGetLastError();
}

EXPORT int vb_moe_gather(const void* x, const int* sorted_tok, void* xs, int R, int H, int dtype, cudaStream_t st) {
  if (H % 8) return -1;
  DISPATCH_HALF(dtype, T, {
    vb_launch(moe::gather_kernel<T>, dim3(R), dim3(128), 0, st, (const T*)x, sorted_tok, (T*)xs, H);
  });
  return (int)cudaGetLastError();
}
