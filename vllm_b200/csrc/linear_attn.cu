// Recurrences with a decayed outer-product state over the per-request state slots (sm_100a):
//
//   S_t = diag(a_t) S_{t-1} + k_t v_t^T,    o_t = S_t^T q_t        S [R, C] fp32 per (request, head)
//
// covers gated linear attention (a decay per key channel: R = key width, C = value width) and the Mamba-2 state-space scan
// (one decay exp(-exp(A_log) dt) per head; k = dt B, q = C, v = x: R = state size, C = head width, plus the D x skip).
//
//   state_scan    variable-length: a request's tokens in order, decode is the one-token case of the same kernel
//   gla_decay     a = sigmoid(W2 y + b)^(1/tau) for whole prompts (decode steps evaluate it inside state_scan)
//   gated_norm    RMS norm over equal groups of channels with the silu gate before or behind it
//
// state_scan: a CTA owns a column tile of one head of one request.  Producer warps stage a block of tokens (decays, keys,
// queries, values, in fp32) into one half of shared memory while consumer warps run the recurrence over the other; one
// barrier per block of TB tokens.  A consumer lane holds 2 NP rows x 4 columns of S in registers as packed pairs of rows, so
// that the three products per element are fma.rn.f32x2; the sum over the rows ends in a few shuffles.  In memory a head's
// state is stored in the order the lanes hold it ([column quad][row in lane][lane][4]): every access is a full 16-byte
// vector per lane and consecutive across the warp.
#include "common.cuh"

namespace lattn {

VB_DEVICE float silu_f(float x) { return x / (1.f + __expf(-x)); }
VB_DEVICE float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
// sigmoid(z)^(1/tau), through the logarithm so that z of either sign keeps its digits
VB_DEVICE float decay_of(float z, float inv_tau) {
  return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau);
}
VB_DEVICE float ld_any(const void* p, int64_t i, int dt) {
  if (dt == DT_F32) return reinterpret_cast<const float*>(p)[i];
  if (dt == DT_BF16) return to_f32(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
  return to_f32(reinterpret_cast<const __half*>(p)[i]);
}
VB_DEVICE float4 ld_any4(const void* p, int64_t i, int dt) {      // i and p aligned to four elements
  if (dt == DT_F32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
  const uint2 u = *reinterpret_cast<const uint2*>(reinterpret_cast<const uint16_t*>(p) + i);
  float2 a, b;
  if (dt == DT_BF16) { a = unpack2<__nv_bfloat16>(u.x); b = unpack2<__nv_bfloat16>(u.y); }
  else { a = unpack2<__half>(u.x); b = unpack2<__half>(u.y); }
  return make_float4(a.x, a.y, b.x, b.y);
}

using pair_t = unsigned long long;      // two fp32
VB_DEVICE pair_t fma2(pair_t a, pair_t b, pair_t c) {
  pair_t d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d;
}
VB_DEVICE pair_t mul2(pair_t a, pair_t b) {
  pair_t d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d;
}
VB_DEVICE pair_t pack(float x, float y) {
  pair_t d; asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y)); return d;
}
VB_DEVICE float2 unpack(pair_t a) {
  float2 v; asm("mov.b64 {%0, %1}, %2;" : "=f"(v.x), "=f"(v.y) : "l"(a)); return v;
}

// barrier over the whole CTA, reached from the producers' and the consumers' code
VB_DEVICE void bar_all() { asm volatile("bar.sync 0;" ::: "memory"); }

enum : int { DECAY_GIVEN = 0, DECAY_LOWRANK = 1, DECAY_HEAD = 2 };
constexpr int PRODUCERS = 4;            // warps

struct ScanParams {
  const void* q; const void* k; const void* v;
  int64_t q_stride, k_stride, v_stride;      // elements between tokens
  int q_dt, k_dt, v_dt;
  float q_scale;
  const float* alpha;                        // DECAY_GIVEN: [T, H * R]
  const void* a1; int64_t a1_stride; int a_dt; const void* a2; const void* a2_b; int rank; float inv_tau;   // DECAY_LOWRANK
  const void* dt; int64_t dt_stride; int dt_dt;                                                            // DECAY_HEAD
  const float* dt_bias; const float* A_log; const float* D; float dt_min, dt_max;
  float* out;                                // [T, H * C]
  float* state; int64_t state_stride, state_off, head_elems;
  const int* qsl; const int* seq_lens; const int* rows; int64_t rows_stride;
  int H, groups, R, C, TB, vec;
};

// NP row pairs per lane, L lanes share the rows: capacity 2 NP L rows; a warp covers 32 / L quads of columns
template <int NP, int L, int MODE>
__global__ void __launch_bounds__(384) state_scan_kernel(const ScanParams p) {
  constexpr int RL = 2 * NP;                 // rows per lane
  constexpr int RP = RL * L;                 // padded rows
  constexpr int CW = 32 / L * 4;             // columns per warp
  extern __shared__ __align__(16) float sm[];
  const int warps = (blockDim.x >> 5) - PRODUCERS;        // consumers
  const int CT = warps * CW, TB = p.TB;
  const int per_tok = (MODE == DECAY_HEAD ? 2 : 3) * RP + 2 * CT + 4;
  float* bufs = sm;                                       // 2 x TB x per_tok
  float* obuf = sm + 2 * TB * per_tok;                    // 2 x TB x CT
  pdl_trigger();
  pdl_wait();
  const int req = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * CT;
  const int t0 = p.qsl[req], t1 = p.qsl[req + 1], n = t1 - t0;
  if (n <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool has_init = p.seq_lens[req] > n;
  const int R = p.R, C = p.C;
  const int g = h / (p.H / p.groups);
  const int nblk = (n + TB - 1) / TB;

  if (warp >= warps) {
    // ================= producers
    const int tid = threadIdx.x - warps * 32;
    constexpr int NT = PRODUCERS * 32;
    auto stage = [&](int blk) {
      float* b = bufs + (blk & 1) * TB * per_tok;
      const int tb = min(TB, n - blk * TB);
      const int64_t tok0 = t0 + (int64_t)blk * TB;
      if constexpr (MODE == DECAY_HEAD) {
        // [k | q] rows, then values, then (decay, dt); the decay goes first: keys are scaled by dt
        const float A = -expf(p.A_log[h]), db = p.dt_bias[h];
        for (int i = tid; i < tb; i += NT) {
          const float dt = fminf(fmaxf(softplus_f(ld_any(p.dt, (tok0 + i) * p.dt_stride + h, p.dt_dt) + db), p.dt_min), p.dt_max);
          float* s = b + i * per_tok + 2 * RP + 2 * CT;
          s[0] = s[1] = expf(A * dt);
          s[2] = dt;
        }
        asm volatile("bar.sync 1, %0;" ::"n"(NT) : "memory");
      }
      if (p.vec) {
        const int rq = RP / 4;
        for (int i = tid; i < tb * rq; i += NT) {
          const int t = i / rq, r = (i - t * rq) * 4;
          float* row = b + t * per_tok;
          float4 kk = make_float4(0.f, 0.f, 0.f, 0.f), qq = kk;
          if (r < R) {
            kk = ld_any4(p.k, (tok0 + t) * p.k_stride + (int64_t)g * R + r, p.k_dt);
            qq = ld_any4(p.q, (tok0 + t) * p.q_stride + (int64_t)g * R + r, p.q_dt);
          }
          const float ks = MODE == DECAY_HEAD ? row[2 * RP + 2 * CT + 2] : 1.f;
          *reinterpret_cast<float4*>(row + r) = make_float4(kk.x * ks, kk.y * ks, kk.z * ks, kk.w * ks);
          *reinterpret_cast<float4*>(row + RP + r) = make_float4(qq.x * p.q_scale, qq.y * p.q_scale, qq.z * p.q_scale, qq.w * p.q_scale);
          if constexpr (MODE == DECAY_GIVEN) {
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < R) a = *reinterpret_cast<const float4*>(p.alpha + ((tok0 + t) * p.H + h) * (int64_t)R + r);
            *reinterpret_cast<float4*>(row + 2 * RP + 2 * CT + 4 + r) = a;
          }
        }
      } else {
        for (int i = tid; i < tb * RP; i += NT) {
          const int t = i / RP, r = i - t * RP;
          float* row = b + t * per_tok;
          float kk = 0.f, qq = 0.f;
          if (r < R) {
            kk = ld_any(p.k, (tok0 + t) * p.k_stride + (int64_t)g * R + r, p.k_dt);
            qq = ld_any(p.q, (tok0 + t) * p.q_stride + (int64_t)g * R + r, p.q_dt);
          }
          row[r] = MODE == DECAY_HEAD ? kk * row[2 * RP + 2 * CT + 2] : kk;
          row[RP + r] = qq * p.q_scale;
          if constexpr (MODE == DECAY_GIVEN)
            row[2 * RP + 2 * CT + 4 + r] = r < R ? p.alpha[((tok0 + t) * p.H + h) * (int64_t)R + r] : 0.f;
        }
      }
      if constexpr (MODE == DECAY_LOWRANK) {
        for (int r = tid; r < RP; r += NT) {
          if (r >= R) { for (int t = 0; t < tb; ++t) b[t * per_tok + 2 * RP + 2 * CT + 4 + r] = 0.f; continue; }
          const int64_t w0 = ((int64_t)h * R + r) * p.rank;
          const float bias = ld_any(p.a2_b, (int64_t)h * R + r, p.a_dt);
          for (int t = 0; t < tb; ++t) {
            float z = bias;
            for (int j = 0; j < p.rank; ++j) z += ld_any(p.a2, w0 + j, p.a_dt) * ld_any(p.a1, (tok0 + t) * p.a1_stride + j, p.a_dt);
            b[t * per_tok + 2 * RP + 2 * CT + 4 + r] = decay_of(z, p.inv_tau);
          }
        }
      }
      for (int i = tid; i < tb * CT; i += NT) {
        const int t = i / CT, c = i - t * CT;
        const float v = c0 + c < C ? ld_any(p.v, (tok0 + t) * p.v_stride + (int64_t)h * C + c0 + c, p.v_dt) : 0.f;
        *reinterpret_cast<float2*>(b + t * per_tok + 2 * RP + 2 * c) = make_float2(v, v);
      }
    };
    auto flush = [&](int blk) {
      const float* o = obuf + (blk & 1) * TB * CT;
      const int tb = min(TB, n - blk * TB);
      for (int i = tid; i < tb * CT; i += NT) {
        const int t = i / CT, c = i - t * CT;
        if (c0 + c < C) p.out[(t0 + (int64_t)blk * TB + t) * p.H * C + (int64_t)h * C + c0 + c] = o[i];
      }
    };
    stage(0);
    bar_all();
    for (int blk = 0; blk < nblk; ++blk) {
      if (blk + 1 < nblk) stage(blk + 1);
      if (blk > 0) flush(blk - 1);
      bar_all();
    }
    flush(nblk - 1);
    return;
  }

  // ================= consumers
  const int lr = lane % L, quad = warp * (32 / L) + lane / L;         // quad of columns inside the tile
  const int cq = c0 / 4 + quad;                                       // ... of the head
  const bool live = cq * 4 < C;
  float* st = p.state + (int64_t)p.rows[req * p.rows_stride] * p.state_stride + p.state_off + (int64_t)h * p.head_elems +
              (int64_t)cq * RP * 4 + lr * 4;
  pair_t S[4][NP];
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
    if (has_init && live) {
      x = *reinterpret_cast<const float4*>(st + (2 * i) * L * 4);
      y = *reinterpret_cast<const float4*>(st + (2 * i + 1) * L * 4);
    }
    S[0][i] = pack(x.x, y.x); S[1][i] = pack(x.y, y.y); S[2][i] = pack(x.z, y.z); S[3][i] = pack(x.w, y.w);
  }
  const float dskip = MODE == DECAY_HEAD ? p.D[h] : 0.f;
  bar_all();
  for (int blk = 0; blk < nblk; ++blk) {
    const float* b = bufs + (blk & 1) * TB * per_tok;
    float* o = obuf + (blk & 1) * TB * CT;
    const int tb = min(TB, n - blk * TB);
#pragma unroll 2
    for (int t = 0; t < tb; ++t) {
      const float* row = b + t * per_tok;
      pair_t kk[NP], qq[NP], aa[NP], vv[4];
      auto ld_rows = [&](const float* src, pair_t (&dst)[NP]) {
        if constexpr (NP == 1) dst[0] = *reinterpret_cast<const pair_t*>(src + lr * RL);
        else {
#pragma unroll
          for (int i = 0; i < NP; i += 2) {
            const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(src + lr * RL + 2 * i);
            dst[i] = u.x; dst[i + 1] = u.y;
          }
        }
      };
      ld_rows(row, kk);
      ld_rows(row + RP, qq);
      if constexpr (MODE == DECAY_HEAD) {
        const pair_t a = *reinterpret_cast<const pair_t*>(row + 2 * RP + 2 * CT);
#pragma unroll
        for (int i = 0; i < NP; ++i) aa[i] = a;
      } else {
        ld_rows(row + 2 * RP + 2 * CT + 4, aa);
      }
      const ulonglong2 v01 = *reinterpret_cast<const ulonglong2*>(row + 2 * RP + quad * 8);
      const ulonglong2 v23 = *reinterpret_cast<const ulonglong2*>(row + 2 * RP + quad * 8 + 4);
      vv[0] = v01.x; vv[1] = v01.y; vv[2] = v23.x; vv[3] = v23.y;
      float s[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        pair_t acc;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          S[c][i] = fma2(aa[i], S[c][i], mul2(kk[i], vv[c]));
          acc = i == 0 ? mul2(S[c][i], qq[i]) : fma2(S[c][i], qq[i], acc);
        }
        const float2 f = unpack(acc);
        s[c] = f.x + f.y;
      }
      // four sums over L lanes: halve the columns twice, then add the rest up
      constexpr int H1 = L / 2, H2 = L / 4;
      const bool up1 = (lr & H1) != 0, up2 = (lr & H2) != 0;
      float x0 = up1 ? s[2] : s[0], x1 = up1 ? s[3] : s[1];
      x0 += __shfl_xor_sync(0xffffffffu, up1 ? s[0] : s[2], H1);
      x1 += __shfl_xor_sync(0xffffffffu, up1 ? s[1] : s[3], H1);
      float x = up2 ? x1 : x0;
      x += __shfl_xor_sync(0xffffffffu, up2 ? x0 : x1, H2);
#pragma unroll
      for (int d = H2 / 2; d > 0; d >>= 1) x += __shfl_xor_sync(0xffffffffu, x, d);
      if ((lr & (H2 - 1)) == 0) {
        const int c = quad * 4 + (up1 ? 2 : 0) + (up2 ? 1 : 0);
        o[t * CT + c] = MODE == DECAY_HEAD ? x + dskip * row[2 * RP + 2 * c] : x;
      }
    }
    bar_all();
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const float2 a = unpack(S[0][i]), b = unpack(S[1][i]), c = unpack(S[2][i]), d = unpack(S[3][i]);
      *reinterpret_cast<float4*>(st + (2 * i) * L * 4) = make_float4(a.x, b.x, c.x, d.x);
      *reinterpret_cast<float4*>(st + (2 * i + 1) * L * 4) = make_float4(a.y, b.y, c.y, d.y);
    }
  }
}

// a[t, ch] = sigmoid(sum_j a1[t, j] a2[ch, j] + b[ch])^(1/tau); thread = channel, DT tokens per CTA
constexpr int DT = 16;
template <typename T>
__global__ void __launch_bounds__(256) gla_decay_kernel(const T* __restrict__ a1, int64_t a1_stride, const T* __restrict__ a2,
                                                         const T* __restrict__ b, float* __restrict__ out, int n, int CH,
                                                         int rank, float inv_tau) {
  extern __shared__ float y[];           // [DT][rank]
  pdl_trigger();
  pdl_wait();
  const int t0 = blockIdx.x * DT, nt = min(DT, n - t0);
  for (int i = threadIdx.x; i < nt * rank; i += blockDim.x) y[i] = to_f32(a1[(int64_t)(t0 + i / rank) * a1_stride + i % rank]);
  __syncthreads();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= CH) return;
  float z[DT];
  const float bias = to_f32(b[c]);
#pragma unroll
  for (int t = 0; t < DT; ++t) z[t] = bias;
  for (int j = 0; j < rank; ++j) {
    const float w = to_f32(a2[(int64_t)c * rank + j]);
#pragma unroll
    for (int t = 0; t < DT; ++t)
      if (t < nt) z[t] += w * y[t * rank + j];
  }
#pragma unroll
  for (int t = 0; t < DT; ++t)
    if (t < nt) out[(int64_t)(t0 + t) * CH + c] = decay_of(z[t], inv_tau);
}

// (token, group of W channels) per group of WPG warps: rms over the group of y (gate first: of y silu(z)), times w, (gate
// last: times silu(z)), times a constant; w repeats after w_len channels
template <typename T, int V>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, int64_t z_stride,
                                                          const T* __restrict__ w, int w_len, T* __restrict__ out,
                                                          int64_t out_stride, int64_t n_rows, int groups, int W, int gate_first,
                                                          float eps, float scale, int wpg) {
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per_cta = 8 / wpg, sub = warp / wpg;
  const int64_t row = (int64_t)blockIdx.x * per_cta + sub;
  const bool ok = row < n_rows;
  const int64_t tok = ok ? row / groups : 0;
  const int g = ok ? (int)(row % groups) : 0;
  const float* yr = y + (tok * groups + g) * (int64_t)W;
  const T* zr = z + tok * z_stride + (int64_t)g * W;
  const int i0 = ((warp % wpg) * 32 + lane) * V, step = wpg * 32 * V;
  constexpr int dt = DTypeOf<T>::v;
  float ss = 0.f;
  if (ok)
    for (int i = i0; i < W; i += step) {
      if constexpr (V == 4) {
        float4 a = *reinterpret_cast<const float4*>(yr + i);
        if (gate_first) {
          const float4 b = ld_any4(zr, i, dt);
          a.x *= silu_f(b.x); a.y *= silu_f(b.y); a.z *= silu_f(b.z); a.w *= silu_f(b.w);
        }
        ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
      } else {
        float a = yr[i];
        if (gate_first) a *= silu_f(to_f32(zr[i]));
        ss += a * a;
      }
    }
  ss = warp_sum(ss);
  if (wpg > 1) {
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int i = 0; i < wpg; ++i) ss += red[sub * wpg + i];
  }
  if (!ok) return;
  const float r = scale / sqrtf(ss / (float)W + eps);
  T* orow = out + tok * out_stride + (int64_t)g * W;
  for (int i = i0; i < W; i += step) {
    const int wi = (int)(((int64_t)g * W + i) % w_len);
    if constexpr (V == 4) {
      const float4 a = *reinterpret_cast<const float4*>(yr + i), b = ld_any4(zr, i, dt), ww = ld_any4(w, wi, dt);
      const float o0 = a.x * silu_f(b.x) * ww.x * r, o1 = a.y * silu_f(b.y) * ww.y * r;
      const float o2 = a.z * silu_f(b.z) * ww.z * r, o3 = a.w * silu_f(b.w) * ww.w * r;
      if constexpr (dt == DT_F32) *reinterpret_cast<float4*>(orow + i) = make_float4(o0, o1, o2, o3);
      else *reinterpret_cast<uint2*>(orow + i) = make_uint2(pack2<T>(o0, o1), pack2<T>(o2, o3));
    } else {
      orow[i] = from_f32<T>(yr[i] * silu_f(to_f32(zr[i])) * to_f32(w[wi]) * r);
    }
  }
}

template <int NP, int L>
int scan_shape(ScanParams& p, int mode, int num_reqs, int max_len, cudaStream_t st) {
  constexpr int RP = 2 * NP * L, CW = 32 / L * 4;
  // narrow tiles while they are needed to fill the SMs, wide ones (fewer copies of the staged rows) otherwise
  int warps = 8;
  while (warps > 1 && ((warps / 2) * CW >= p.C || (int64_t)num_reqs * p.H * ((p.C + warps * CW - 1) / (warps * CW)) < 148)) warps /= 2;
  const int CT = warps * CW;
  const int per_tok = (mode == DECAY_HEAD ? 2 : 3) * RP + 2 * CT + 4;
  int TB = 16;
  while (TB > 1 && (TB / 2 >= max_len || (size_t)(2 * TB * (per_tok + CT)) * 4 > 100 * 1024)) TB /= 2;
  p.TB = TB;
  const size_t smem = (size_t)(2 * TB * (per_tok + CT)) * 4;
  dim3 grid((p.C + CT - 1) / CT, p.H, num_reqs), block(32 * (warps + PRODUCERS));
#define GO(M)                                                                                             \
  do {                                                                                                    \
    auto kern = state_scan_kernel<NP, L, M>;                                                              \
    static bool set = false;                                                                              \
    if (!set) { cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 101 * 1024); set = true; } \
    vb_launch(kern, grid, block, smem, st, p);                                                            \
  } while (0)
  if (mode == DECAY_GIVEN) GO(DECAY_GIVEN);
  else if (mode == DECAY_LOWRANK) GO(DECAY_LOWRANK);
  else GO(DECAY_HEAD);
#undef GO
  return (int)cudaGetLastError();
}

inline bool al(const void* p, int64_t n) { return p == nullptr || (reinterpret_cast<uintptr_t>(p) % (size_t)n) == 0; }
inline int esz(int dt) { return dt == DT_F32 ? 4 : 2; }

int scan(ScanParams& p, int mode, int num_reqs, int max_len, cudaStream_t st) {
  if (num_reqs == 0) return 0;
  if (p.R < 1 || p.C < 1 || p.groups < 1 || p.H % p.groups || (mode != DECAY_HEAD && p.groups != p.H)) return -1;
  if (p.state_stride % 4 || p.state_off % 4 || !al(p.state, 16)) return -2;
  p.vec = p.R % 4 == 0 && p.q_stride % 4 == 0 && p.k_stride % 4 == 0 && al(p.q, 4 * esz(p.q_dt)) && al(p.k, 4 * esz(p.k_dt)) &&
          al(p.alpha, 16);
  const int rp = p.R <= 16 ? 16 : p.R <= 32 ? 32 : p.R <= 64 ? 64 : p.R <= 128 ? 128 : p.R <= 256 ? 256 : 512;
  if (p.R > 512) return -3;
  p.head_elems = (int64_t)((p.C + 3) / 4) * 4 * rp;
  switch (rp) {
    case 16: return scan_shape<1, 8>(p, mode, num_reqs, max_len, st);
    case 32: return scan_shape<1, 16>(p, mode, num_reqs, max_len, st);
    case 64: return scan_shape<2, 16>(p, mode, num_reqs, max_len, st);
    case 128: return scan_shape<2, 32>(p, mode, num_reqs, max_len, st);
    case 256: return scan_shape<4, 32>(p, mode, num_reqs, max_len, st);
    default: return scan_shape<8, 32>(p, mode, num_reqs, max_len, st);
  }
}

}  // namespace lattn

// Floats that a head's [R, C] state takes in a slot (multiples of the lane layout); < 0: not covered.
EXPORT int vb_state_scan_elems(int R, int C) {
  if (R < 1 || R > 512 || C < 1) return -1;
  const int rp = R <= 16 ? 16 : R <= 32 ? 32 : R <= 64 ? 64 : R <= 128 ? 128 : R <= 256 ? 256 : 512;
  return (C + 3) / 4 * 4 * rp;
}

// Gated linear attention.  q, k [T, H * R], v [T, H * C] (token strides free); alpha [T, H * R] fp32, or null and the decay
// is evaluated from a1 [T, rank], a2 [H * R, rank], a2_b [H * R].  out [T, H * C] fp32.
EXPORT int vb_gla_scan(const void* q, const void* k, const void* v, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                       float q_scale, const float* alpha, const void* a1, int64_t a1_stride, const void* a2, const void* a2_b,
                       int rank, float inv_tau, float* out, float* state, int64_t state_stride, int64_t state_off,
                       const int* qsl, const int* seq_lens, const int* rows, int64_t rows_stride, int num_reqs, int max_len,
                       int H, int R, int C, int dtype, cudaStream_t st) {
  lattn::ScanParams p = {};
  p.q = q; p.k = k; p.v = v; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
  p.q_dt = p.k_dt = p.v_dt = p.a_dt = dtype; p.q_scale = q_scale; p.alpha = alpha;
  p.a1 = a1; p.a1_stride = a1_stride; p.a2 = a2; p.a2_b = a2_b; p.rank = rank; p.inv_tau = inv_tau;
  p.out = out; p.state = state; p.state_stride = state_stride; p.state_off = state_off;
  p.qsl = qsl; p.seq_lens = seq_lens; p.rows = rows; p.rows_stride = rows_stride;
  p.H = H; p.groups = H; p.R = R; p.C = C;
  return lattn::scan(p, alpha ? lattn::DECAY_GIVEN : lattn::DECAY_LOWRANK, num_reqs, max_len, st);
}

// Mamba-2.  xbc [T, H * C + 2 groups * R] fp32 = x | B | C behind the convolution; dt [T, H] raw (bias, softplus and clamp
// here).  out [T, H * C] fp32, D x included.
EXPORT int vb_ssd_scan(const float* xbc, int64_t xbc_stride, const void* dt, int64_t dt_stride, const float* dt_bias,
                       const float* A_log, const float* D, float* out, float* state, int64_t state_stride, int64_t state_off,
                       const int* qsl, const int* seq_lens, const int* rows, int64_t rows_stride, int num_reqs, int max_len,
                       int H, int C, int groups, int R, float dt_min, float dt_max, int dt_dtype, cudaStream_t st) {
  lattn::ScanParams p = {};
  p.v = xbc; p.k = xbc + (int64_t)H * C; p.q = xbc + (int64_t)H * C + (int64_t)groups * R;
  p.q_stride = p.k_stride = p.v_stride = xbc_stride; p.q_dt = p.k_dt = p.v_dt = DT_F32; p.q_scale = 1.f;
  p.dt = dt; p.dt_stride = dt_stride; p.dt_dt = dt_dtype; p.dt_bias = dt_bias; p.A_log = A_log; p.D = D;
  p.dt_min = dt_min; p.dt_max = dt_max; p.out = out; p.state = state; p.state_stride = state_stride; p.state_off = state_off;
  p.qsl = qsl; p.seq_lens = seq_lens; p.rows = rows; p.rows_stride = rows_stride;
  p.H = H; p.groups = groups; p.R = R; p.C = C;
  return lattn::scan(p, lattn::DECAY_HEAD, num_reqs, max_len, st);
}

EXPORT int vb_gla_decay(const void* a1, int64_t a1_stride, const void* a2, const void* b, float* out, int T_, int CH, int rank,
                        float inv_tau, int dtype, cudaStream_t st) {
  using namespace lattn;
  if (T_ == 0) return 0;
  const size_t smem = (size_t)DT * rank * 4;
  if (smem > 48 * 1024) return -1;
  dim3 grid((T_ + DT - 1) / DT, (CH + 255) / 256);
  DISPATCH_DTYPE(dtype, T, vb_launch(gla_decay_kernel<T>, grid, dim3(256), smem, st, (const T*)a1, a1_stride, (const T*)a2,
                                     (const T*)b, out, T_, CH, rank, inv_tau));
  return (int)cudaGetLastError();
}

// y [T, groups * W] fp32, z [T, groups * W] (token stride free), w [w_len] repeated along the channels (w_len a multiple or
// a divisor of W); out [T, groups * W] in the model dtype (token stride free)
EXPORT int vb_gated_norm(const float* y, const void* z, int64_t z_stride, const void* w, int w_len, void* out,
                         int64_t out_stride, int T_, int groups, int W, int gate_first, float eps, float scale, int dtype,
                         cudaStream_t st) {
  using namespace lattn;
  if (T_ == 0) return 0;
  const int64_t rows = (int64_t)T_ * groups;
  const int e = esz(dtype);
  const bool vec = W % 4 == 0 && w_len % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0 && al(y, 16) && al(z, 4 * e) &&
                   al(w, 4 * e) && al(out, 4 * e);
  const int wpg = W <= 512 ? 1 : W <= 1024 ? 2 : W <= 2048 ? 4 : 8;
  dim3 grid((unsigned)((rows + 8 / wpg - 1) / (8 / wpg)));
  DISPATCH_DTYPE(dtype, T, {
    if (vec) vb_launch(gated_norm_kernel<T, 4>, grid, dim3(256), 0, st, y, (const T*)z, z_stride, (const T*)w, w_len, (T*)out, out_stride, rows, groups, W, gate_first, eps, scale, wpg);
    else vb_launch(gated_norm_kernel<T, 1>, grid, dim3(256), 0, st, y, (const T*)z, z_stride, (const T*)w, w_len, (T*)out, out_stride, rows, groups, W, gate_first, eps, scale, wpg);
  });
  return (int)cudaGetLastError();
}
