// Recurrences with a decayed outer-product state over the per-request state slots (sm_100a):
//
//   S_t = diag(a_t) S_{t-1} + k_t v_t^T,    o_t = S_t^T q_t        S [R, C] fp32 per (request, head)
//
// covers gated linear attention (a decay per key channel: R = key width, C = value width), the Mamba-2 state-space scan
// (one decay exp(-exp(A_log) dt) per head; k = dt B, q = C, v = x: R = state size, C = head width, plus the D x skip) and the
// matrix memory of xLSTM (a decay and an input factor per head, exp(f + m' - m) and exp(i - m) with a running maximum m; one more
// column of S, whose value is always 1, is the normaliser n).
//
//   state_scan    variable-length: a request's tokens in order, decode is the one-token case of the same kernel
//   gla_decay     a = sigmoid(W2 y + b)^(1/tau) for whole prompts (decode steps evaluate it inside state_scan)
//   memory_gates  log gates -> (decay, input factor, exp(-m)) per token and head; m is carried in the slot
//   gated_norm    RMS norm over equal groups of channels with a silu or sigmoid gate before or behind it; of a matrix memory, the
//                 division by max(|n . q|, exp(-m)) in front of it
//
// state_scan: a CTA owns a column tile of one head of one request.  Producer warps stage a block of tokens (decays, keys,
// queries, values, in fp32) into one half of shared memory while consumer warps run the recurrence over the other; one
// barrier per block of TB tokens, and the loads of the block after next are in flight meanwhile.  A consumer lane holds 2 NP
// rows x 4 Q columns of S in registers as packed pairs of rows, so that the three products per element are fma.rn.f32x2; the
// sum over the rows ends in a few shuffles.  In memory a head's
// state is stored in the order the lanes of decode steps hold it: every access of theirs is a full 16-byte vector per lane and
// consecutive across the warp.
#include "common.cuh"

namespace lattn {

VB_DEVICE float silu_f(float x) { return __fdividef(x, 1.f + __expf(-x)); }
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

// values of four elements as they lie in memory
VB_DEVICE float4 values4(uint4 u, int dt) {
  if (dt == DT_F32) return make_float4(__uint_as_float(u.x), __uint_as_float(u.y), __uint_as_float(u.z), __uint_as_float(u.w));
  const float2 a = dt == DT_BF16 ? unpack2<__nv_bfloat16>(u.x) : unpack2<__half>(u.x);
  const float2 b = dt == DT_BF16 ? unpack2<__nv_bfloat16>(u.y) : unpack2<__half>(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
VB_DEVICE uint4 bits4(float4 v) {
  return make_uint4(__float_as_uint(v.x), __float_as_uint(v.y), __float_as_uint(v.z), __float_as_uint(v.w));
}

// up to four elements, zeros behind the n-th; not inlined: the path of odd sizes and addresses
__device__ __noinline__ float4 ld_some(const void* p, int64_t i, int dt, int n) {
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (n > 0) v.x = ld_any(p, i, dt);
  if (n > 1) v.y = ld_any(p, i + 1, dt);
  if (n > 2) v.z = ld_any(p, i + 2, dt);
  if (n > 3) v.w = ld_any(p, i + 3, dt);
  return v;
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

enum : int { DECAY_GIVEN = 0, DECAY_LOWRANK = 1, DECAY_HEAD = 2, DECAY_GATES = 3 };
constexpr bool head_decay(int mode) { return mode == DECAY_HEAD || mode == DECAY_GATES; }      // one decay and key factor per head

struct ScanParams {
  const void* q; const void* k; const void* v;
  int64_t q_stride, k_stride, v_stride;      // elements between tokens
  int q_dt, k_dt, v_dt;
  float q_scale;
  const float* alpha;                        // DECAY_GIVEN: [T, H * R]
  const void* a1; int64_t a1_stride; int a_dt; const void* a2; const void* a2_b; int rank; float inv_tau;   // DECAY_LOWRANK
  const void* dt; int64_t dt_stride; int dt_dt;                                                            // DECAY_HEAD
  const float* dt_bias; const float* A_log; const float* D; float dt_min, dt_max;
  const float4* gates;                       // DECAY_GATES: [T, H] (decay, key factor, ...)
  float* out;                                // [T, H * CO]
  float* state; int64_t state_stride, state_off, head_elems;
  const int* qsl; const int* seq_lens; const int* rows; int64_t rows_stride;
  int H, groups, R, C;
  int CV, CO;                                // columns that v has and columns of an output row; C but for DECAY_GATES
  int vec, vec_v, vec_o, vec_a;              // accesses in units of four elements
};

// N sums per lane over the lanes lr, lr ^ D, ...: each step hands half of the columns to the other lane; ``at``: first column left
template <int N, int D>
VB_DEVICE void reduce_columns(float* s, int lr, int& at) {
  if constexpr (D > 0) {
    const bool up = (lr & D) != 0;
    if constexpr (N > 1) {
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        const float keep = up ? s[i + N / 2] : s[i], send = up ? s[i] : s[i + N / 2];
        s[i] = keep + __shfl_xor_sync(0xffffffffu, send, D);
      }
      at += up ? N / 2 : 0;
      reduce_columns<N / 2, D / 2>(s, lr, at);
    } else {
      s[0] += __shfl_xor_sync(0xffffffffu, s[0], D);
      reduce_columns<1, D / 2>(s, lr, at);
    }
  }
}

// Place of row r in a column quad's [RP][4] block: the order in which the lanes of the decode form (SL lanes, SNP pairs) hold them.
template <int SNP, int SL> VB_DEVICE int row_place(int r) {
  if constexpr (SNP == 1) return (r & 1) * SL + (r >> 1);
  else return ((r >> 2) / SL * 4 + (r & 3)) * SL + (r >> 2) % SL;
}

// NP row pairs per lane, L lanes share the rows (capacity 2 NP L rows); a lane holds Q quads of columns.  Decode steps want many
// warps and whole vectors of state (SNP, SL: the form whose order the state has in memory).  Prompts want many rows per lane:
// a staged row is then read by few lanes for many columns, and the sum over the lanes is short.
template <int NP, int L, int SNP, int SL, int MODE, int Q, int TB, int PRODUCERS>
__global__ void __launch_bounds__(384, TB == 1 && NP <= 2 ? 2 : 1) state_scan_kernel(const ScanParams p) {
  constexpr int RL = 2 * NP;                 // rows per lane
  constexpr int RP = RL * L;                 // padded rows
  constexpr int LG = 32 / L;
  constexpr int CW = LG * 4 * Q;             // columns per warp
  constexpr int U = TB >= 4 ? 4 : TB;        // tokens whose sums are reduced together
  constexpr int NT = PRODUCERS * 32;
  extern __shared__ __align__(16) float sm[];
  const int warps = (blockDim.x >> 5) - PRODUCERS;        // consumers
  const int CT = warps * CW;
  // a staged token: keys RP | queries RP | values 2 CT (each twice) | decay, decay, key factor, - | decays RP (per channel)
  const int per_tok = (head_decay(MODE) ? 2 : 3) * RP + 2 * CT + 4;
  float* bufs = sm;                                       // 2 x TB x per_tok
  float* obuf = sm + 2 * TB * per_tok;                    // 2 x TB x CT
  pdl_trigger();
  pdl_wait();
  const int req = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * CT;
  const int t0 = p.qsl[req], t1 = p.qsl[req + 1], n = t1 - t0;
  if (n <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int R = p.R, C = p.C;
  const int nblk = (n + TB - 1) / TB;

  if (warp >= warps) {
    // ================= producers: the loads of a block are in flight while the block before it is computed
    const int tid = threadIdx.x - warps * 32;
    const int g = h / (p.H / p.groups);
    constexpr int NI = (TB * (RP / 4) + NT - 1) / NT;     // row vectors per thread and operand
    constexpr int NVI = (TB * 32 + NT - 1) / NT;          // value vectors per thread held ahead (of wider tiles the rest is late)
    uint4 rk[NI], rq[NI], rv[NVI];
    float4 ra[NI];
    uint32_t rdt = 0;
    float2 rgate = make_float2(0.f, 0.f);
    // what the registers hold: operands as they lie in memory (one branch per block, no conversion and no predicate between
    // the loads, or each of them would be waited for), or fp32 bits where sizes or addresses are odd
    const bool fast16 = p.vec && p.vec_v && p.k_dt != DT_F32, fast32 = p.vec && p.vec_v && p.k_dt == DT_F32;
    const int dt = fast16 ? p.k_dt : DT_F32;
    const int cv = CT / 4;
    int vt[NVI], vc[NVI];                                 // token and column of the value vectors
#pragma unroll
    for (int i = 0; i < NVI; ++i) { vt[i] = (tid + i * NT) / cv; vc[i] = (tid + i * NT - vt[i] * cv) * 4; }
    const float neg_a = MODE == DECAY_HEAD ? -expf(p.A_log[h]) : 0.f, db = MODE == DECAY_HEAD ? p.dt_bias[h] : 0.f;
    auto slow_value = [&](int64_t tok, int c) { return bits4(ld_some(p.v, tok * p.v_stride + (int64_t)h * p.CV + c, p.v_dt, p.CV - c)); };
    auto fetch = [&](int blk) {
      const int tb = min(TB, n - blk * TB);
      const int64_t tok0 = t0 + (int64_t)blk * TB;
      auto token = [&](int t) { return tok0 + min(t, tb - 1); };       // the rest reads the last token again
      if constexpr (MODE == DECAY_HEAD) {
        const int64_t i = token(tid) * p.dt_stride + h;
        if (p.dt_dt == DT_F32) rdt = reinterpret_cast<const uint32_t*>(p.dt)[i];
        else rdt = reinterpret_cast<const uint16_t*>(p.dt)[i];
      }
      if constexpr (MODE == DECAY_GATES) rgate = *reinterpret_cast<const float2*>(p.gates + token(tid) * p.H + h);
      auto load = [&](auto vec_type) {
        using V = decltype(vec_type);
        constexpr int ES = sizeof(V) / 4;
        auto get = [&](uint4& d, const void* base, int64_t i) {
          const V u = *reinterpret_cast<const V*>(reinterpret_cast<const char*>(base) + i * ES);
          d.x = u.x; d.y = u.y;
          if constexpr (ES == 4) { d.z = u.z; d.w = u.w; }
        };
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const int it = tid + i * NT, r = min((it % (RP / 4)) * 4, R - 4);
          const int64_t tok = token(it / (RP / 4));
          get(rk[i], p.k, tok * p.k_stride + (int64_t)g * R + r);
          get(rq[i], p.q, tok * p.q_stride + (int64_t)g * R + r);
          if constexpr (MODE == DECAY_GIVEN) ra[i] = *reinterpret_cast<const float4*>(p.alpha + (tok * p.H + h) * (int64_t)R + r);
        }
#pragma unroll
        for (int i = 0; i < NVI; ++i) get(rv[i], p.v, token(vt[i]) * p.v_stride + (int64_t)h * p.CV + min(c0 + vc[i], p.CV - 4));
      };
      if (fast16) load(uint2{});
      else if (fast32) load(uint4{});
      else {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const int it = tid + i * NT, r = (it % (RP / 4)) * 4;
          const int64_t tok = token(it / (RP / 4));
          rk[i] = bits4(ld_some(p.k, tok * p.k_stride + (int64_t)g * R + r, p.k_dt, R - r));
          rq[i] = bits4(ld_some(p.q, tok * p.q_stride + (int64_t)g * R + r, p.q_dt, R - r));
          if constexpr (MODE == DECAY_GIVEN) ra[i] = ld_some(p.alpha, (tok * p.H + h) * (int64_t)R + r, DT_F32, R - r);
        }
#pragma unroll
        for (int i = 0; i < NVI; ++i) rv[i] = slow_value(token(vt[i]), c0 + vc[i]);
      }
    };
    auto store = [&](int blk) {
      float* b = bufs + (blk & 1) * TB * per_tok;
      const int tb = min(TB, n - blk * TB);
      const int64_t tok0 = t0 + (int64_t)blk * TB;
      if constexpr (MODE == DECAY_HEAD) {
        if (tid < tb) {
          const float raw = p.dt_dt == DT_F32 ? __uint_as_float(rdt) : p.dt_dt == DT_BF16 ? unpack2<__nv_bfloat16>(rdt).x : unpack2<__half>(rdt).x;
          const float step = fminf(fmaxf(softplus_f(raw + db), p.dt_min), p.dt_max);
          float* d = b + tid * per_tok + 2 * RP + 2 * CT;
          d[0] = d[1] = expf(neg_a * step);
          d[2] = step;
        }
        asm volatile("bar.sync 1, %0;" ::"n"(NT) : "memory");
      }
      if constexpr (MODE == DECAY_GATES) {
        if (tid < tb) {
          float* d = b + tid * per_tok + 2 * RP + 2 * CT;
          d[0] = d[1] = rgate.x;
          d[2] = rgate.y;
        }
        asm volatile("bar.sync 1, %0;" ::"n"(NT) : "memory");
      }
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int it = tid + i * NT, t = it / (RP / 4), r = (it % (RP / 4)) * 4;
        if (t >= tb) continue;
        float* row = b + t * per_tok;
        const float ks = head_decay(MODE) ? row[2 * RP + 2 * CT + 2] : 1.f;
        const bool in = r < R;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), kv = in ? values4(rk[i], dt) : zero, qv = in ? values4(rq[i], dt) : zero;
        *reinterpret_cast<float4*>(row + r) = make_float4(kv.x * ks, kv.y * ks, kv.z * ks, kv.w * ks);
        *reinterpret_cast<float4*>(row + RP + r) = make_float4(qv.x * p.q_scale, qv.y * p.q_scale, qv.z * p.q_scale, qv.w * p.q_scale);
        if constexpr (MODE == DECAY_GIVEN) *reinterpret_cast<float4*>(row + 2 * RP + 2 * CT + 4 + r) = in ? ra[i] : zero;
      }
      if constexpr (MODE == DECAY_LOWRANK) {
        for (int r = tid; r < RP; r += NT) {
          const int64_t w0 = ((int64_t)h * R + r) * p.rank;
          const float bias = r < R ? ld_any(p.a2_b, (int64_t)h * R + r, p.a_dt) : 0.f;
          for (int t = 0; t < tb; ++t) {
            float z = bias;
            const int64_t y0 = (tok0 + t) * p.a1_stride;
            if (r < R) {
              if (p.vec_a) {
#pragma unroll 4
                for (int j = 0; j < p.rank; j += 4) {
                  const float4 w = ld_any4(p.a2, w0 + j, p.a_dt), y = ld_any4(p.a1, y0 + j, p.a_dt);
                  z += w.x * y.x; z += w.y * y.y; z += w.z * y.z; z += w.w * y.w;
                }
              } else {
                for (int j = 0; j < p.rank; ++j) z += ld_any(p.a2, w0 + j, p.a_dt) * ld_any(p.a1, y0 + j, p.a_dt);
              }
            }
            b[t * per_tok + 2 * RP + 2 * CT + 4 + r] = r < R ? decay_of(z, p.inv_tau) : 0.f;
          }
        }
      }
      auto put = [&](int t, int c, float4 v) {
        if constexpr (MODE == DECAY_GATES) {                 // behind the values: zeros up to a quad's end, the one, zeros
          const int past = c0 + c - p.CV;
          if (past > -4) {
            const int one = p.CO - 4 - p.CV;
            if (past >= 0) v.x = past == one ? 1.f : 0.f;
            if (past >= -1) v.y = past + 1 == one ? 1.f : 0.f;
            if (past >= -2) v.z = past + 2 == one ? 1.f : 0.f;
            v.w = past + 3 == one ? 1.f : 0.f;
          }
        }
        float4* d = reinterpret_cast<float4*>(b + t * per_tok + 2 * RP + 2 * c);
        d[0] = make_float4(v.x, v.x, v.y, v.y);
        d[1] = make_float4(v.z, v.z, v.w, v.w);
      };
#pragma unroll
      for (int i = 0; i < NVI; ++i) {
        if (vt[i] < tb) put(vt[i], vc[i], values4(rv[i], dt));
      }
      for (int it = tid + NVI * NT; it < tb * cv; it += NT) {
        const int t = it / cv, c = (it - t * cv) * 4;
        put(t, c, values4(slow_value(tok0 + t, c0 + c), DT_F32));
      }
    };
    auto flush = [&](int blk) {
      const float* o = obuf + (blk & 1) * TB * CT;
      const int tb = min(TB, n - blk * TB);
      if (p.vec_o) {
        for (int i = tid; i < tb * cv; i += NT) {
          const int t = i / cv, c = (i - t * cv) * 4;
          if (c0 + c < p.CO)
            *reinterpret_cast<float4*>(p.out + (t0 + (int64_t)blk * TB + t) * p.H * p.CO + (int64_t)h * p.CO + c0 + c) =
                *reinterpret_cast<const float4*>(o + t * CT + c);
        }
        return;
      }
      for (int i = tid; i < tb * CT; i += NT) {
        const int t = i / CT, c = i - t * CT;
        if (c0 + c < p.CO) p.out[(t0 + (int64_t)blk * TB + t) * p.H * p.CO + (int64_t)h * p.CO + c0 + c] = o[i];
      }
    };
    fetch(0);
    store(0);
    if (nblk > 1) fetch(1);
    bar_all();
    for (int blk = 0; blk < nblk; ++blk) {
      if (blk + 1 < nblk) {
        store(blk + 1);
        if (blk + 2 < nblk) fetch(blk + 2);
      }
      if (blk > 0) flush(blk - 1);
      bar_all();
    }
    flush(nblk - 1);
    return;
  }

  // ================= consumers
  const int lr = lane % L, lg = lane / L;
  auto quad_of = [&](int j) { return (warp * Q + j) * LG + lg; };     // quad of columns inside the tile
  auto row_of = [&](int i) { return NP == 1 ? lr * 2 : ((i >> 1) * L + lr) * 4 + (i & 1) * 2; };      // first row of pair i
  const bool has_init = p.seq_lens[req] > n;
  float* st = p.state + (int64_t)p.rows[req * p.rows_stride] * p.state_stride + p.state_off + (int64_t)h * p.head_elems;
  auto at_row = [&](int64_t cq, int r) { return st + (cq * RP + row_place<SNP, SL>(r)) * 4; };
  pair_t S[Q][4][NP];
#pragma unroll
  for (int j = 0; j < Q; ++j) {
    const int64_t cq = c0 / 4 + quad_of(j);
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
      if (has_init && cq * 4 < C) {
        x = *reinterpret_cast<const float4*>(at_row(cq, row_of(i)));
        y = *reinterpret_cast<const float4*>(at_row(cq, row_of(i) + 1));
      }
      S[j][0][i] = pack(x.x, y.x); S[j][1][i] = pack(x.y, y.y); S[j][2][i] = pack(x.z, y.z); S[j][3][i] = pack(x.w, y.w);
    }
  }
  const float dskip = MODE == DECAY_HEAD ? p.D[h] : 0.f;
  bar_all();
  for (int blk = 0; blk < nblk; ++blk) {
    const float* b = bufs + (blk & 1) * TB * per_tok;
    float* o = obuf + (blk & 1) * TB * CT;
    const int tb = min(TB, n - blk * TB);
    // U tokens at a time: their sums are reduced together (fewer shuffles, and none of them waits for the one before)
    for (int tg = 0; tg < tb; tg += U) {
      float s[U * 4 * Q];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (tg + u >= tb) {                      // behind the last token: nothing may touch the state
#pragma unroll
          for (int i = 0; i < 4 * Q; ++i) s[u * 4 * Q + i] = 0.f;
          continue;
        }
        const float* row = b + (tg + u) * per_tok;
        constexpr int M = NP == 1 ? 1 : NP / 2, P = NP == 1 ? 1 : 2;      // vectors of rows, pairs in one
        auto ld_rows = [&](const float* src, pair_t (&dst)[P]) {
          if constexpr (NP == 1) dst[0] = *reinterpret_cast<const pair_t*>(src);
          else {
            const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(src);
            dst[0] = w.x; dst[P - 1] = w.y;
          }
        };
        pair_t vv[Q][4], acc[Q][4];
#pragma unroll
        for (int j = 0; j < Q; ++j) {
          const float* vp = row + 2 * RP + quad_of(j) * 8;
          const ulonglong2 v01 = *reinterpret_cast<const ulonglong2*>(vp), v23 = *reinterpret_cast<const ulonglong2*>(vp + 4);
          vv[j][0] = v01.x; vv[j][1] = v01.y; vv[j][2] = v23.x; vv[j][3] = v23.y;
        }
        pair_t ah = 0;
        if constexpr (head_decay(MODE)) ah = *reinterpret_cast<const pair_t*>(row + 2 * RP + 2 * CT);
#pragma unroll
        for (int m = 0; m < M; ++m) {
          pair_t kk[P], qq[P], aa[P];
          const int r = row_of(2 * m);
          ld_rows(row + r, kk);
          ld_rows(row + RP + r, qq);
          if constexpr (head_decay(MODE)) {
#pragma unroll
            for (int i = 0; i < P; ++i) aa[i] = ah;
          } else {
            ld_rows(row + 2 * RP + 2 * CT + 4 + r, aa);
          }
#pragma unroll
          for (int j = 0; j < Q; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
              for (int i = 0; i < P; ++i) {
                pair_t& S1 = S[j][c][P * m + i];
                S1 = fma2(aa[i], S1, mul2(kk[i], vv[j][c]));
                acc[j][c] = m + i == 0 ? mul2(S1, qq[i]) : fma2(S1, qq[i], acc[j][c]);
              }
        }
#pragma unroll
        for (int j = 0; j < Q; ++j)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float2 f = unpack(acc[j][c]);
            s[(u * Q + j) * 4 + c] = f.x + f.y;
          }
      }
      // the sums over L lanes: halve their number while there are two or more, then add the rest up
      constexpr int N = 4 * Q * U;
      int at = 0;
      reduce_columns<N, L / 2>(s, lr, at);
      constexpr int LEFT = N > L ? N / L : 1, SAME = L > N ? L / N : 1;      // sums per lane, lanes with the same
      if ((lr & (SAME - 1)) == 0) {
#pragma unroll
        for (int i = 0; i < LEFT; ++i) {
          const int x = at + i, t = tg + x / (4 * Q), c = quad_of(x / 4 % Q) * 4 + (x & 3);
          if (t < tb) o[t * CT + c] = MODE == DECAY_HEAD ? s[i] + dskip * b[t * per_tok + 2 * RP + 2 * c] : s[i];
        }
      }
    }
    bar_all();
  }
#pragma unroll
  for (int j = 0; j < Q; ++j) {
    const int64_t cq = c0 / 4 + quad_of(j);
    if (cq * 4 >= C) continue;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const float2 a = unpack(S[j][0][i]), bb = unpack(S[j][1][i]), c = unpack(S[j][2][i]), d = unpack(S[j][3][i]);
      *reinterpret_cast<float4*>(at_row(cq, row_of(i))) = make_float4(a.x, bb.x, c.x, d.x);
      *reinterpret_cast<float4*>(at_row(cq, row_of(i) + 1)) = make_float4(a.y, bb.y, c.y, d.y);
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

// Gates of a matrix memory, one CTA per request and head.  z = W h + b, capped: z' = cap tanh(z / cap); log input gate i = z'_i, log
// forget gate f = log sigmoid(z'_f);  m_t = max(m_{t-1} + f_t, i_t), m before the first token 0;  out = (exp(f + m_{t-1} - m_t),
// exp(i - m_t), exp(-m_t), 0).  A token maps m to max(m + F, M) with (F, M) = (f, i), and so does a run of tokens: blocks of
// blockDim tokens are scanned in parallel.  logits null: one token per request, and the two products are computed here.
constexpr int GATE_T = 256, GATE_MAX_T = 1024;
struct GateParams {
  const void* h; int64_t h_stride; const void* w; int W;
  const float* logits;                       // [T, 2 H], before the bias
  const float* bias; float cap;              // [2 H]: input gates, forget gates
  float4* out;
  float* state; int64_t state_stride, m_off;
  const int* qsl; const int* seq_lens; const int* rows; int64_t rows_stride;
  int H;
};
VB_DEVICE float2 compose(float2 a, float2 b) { return make_float2(a.x + b.x, fmaxf(a.y + b.x, b.y)); }      // a, then b

template <typename T, int V>
__global__ void __launch_bounds__(GATE_MAX_T) memory_gates_kernel(const GateParams p) {
  __shared__ float red[32];
  __shared__ float2 runs[32];
  __shared__ float ms[GATE_MAX_T];
  pdl_trigger();
  pdl_wait();
  const int req = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, width = blockDim.x;
  const int t0 = p.qsl[req], n = p.qsl[req + 1] - t0;
  if (n <= 0) return;
  float* slot = p.state + (int64_t)p.rows[req * p.rows_stride] * p.state_stride + p.m_off + hd;
  float m = p.seq_lens[req] > n ? *slot : 0.f;
  const float bi = p.bias[hd], bf = p.bias[p.H + hd];
  auto capped = [&](float z) { return p.cap * tanhf(z / p.cap); };
  auto log_sigmoid = [](float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); };
  auto gates = [&](float f, float i, float before, float after) {
    return make_float4(expf(f + before - after), expf(i - after), expf(-after), 0.f);
  };
  if (p.logits == nullptr) {
    const T* h = reinterpret_cast<const T*>(p.h) + (int64_t)t0 * p.h_stride;
    const T* wi = reinterpret_cast<const T*>(p.w) + (int64_t)hd * p.W;
    const T* wf = wi + (int64_t)p.H * p.W;
    float zi = 0.f, zf = 0.f;
    for (int c = tid * V; c < p.W; c += width * V) {
      if constexpr (V == 4) {
        constexpr int dt = DTypeOf<T>::v;
        const float4 x = ld_any4(h, c, dt), a = ld_any4(wi, c, dt), b = ld_any4(wf, c, dt);
        zi += x.x * a.x; zi += x.y * a.y; zi += x.z * a.z; zi += x.w * a.w;
        zf += x.x * b.x; zf += x.y * b.y; zf += x.z * b.z; zf += x.w * b.w;
      } else {
        const float x = to_f32(h[c]);
        zi += x * to_f32(wi[c]); zf += x * to_f32(wf[c]);
      }
    }
    zi = block_sum(zi, red);
    zf = block_sum(zf, red);
    if (tid == 0) {
      const float i = capped(zi + bi), f = log_sigmoid(capped(zf + bf)), after = fmaxf(f + m, i);
      p.out[(int64_t)t0 * p.H + hd] = gates(f, i, m, after);
      *slot = after;
    }
    return;
  }
  auto scan = [&](float2 run) {                                 // of the warp's lanes, each with those before it
#pragma unroll
    for (int d = 1; d < 32; d *= 2) {
      const float2 o = make_float2(__shfl_up_sync(0xffffffffu, run.x, d), __shfl_up_sync(0xffffffffu, run.y, d));
      if (lane >= d) run = compose(o, run);
    }
    return run;
  };
  for (int b0 = 0; b0 < n; b0 += width) {
    const int t = b0 + tid;
    float i = -INFINITY, f = 0.f;                               // behind the last token: m stays
    if (t < n) {
      const float* z = p.logits + (int64_t)(t0 + t) * 2 * p.H + hd;
      i = capped(z[0] + bi);
      f = log_sigmoid(capped(z[p.H] + bf));
    }
    const float2 run = scan(make_float2(f, i));
    if (lane == 31) runs[warp] = run;
    __syncthreads();
    if (warp == 0) {
      const float2 all = scan(lane < width / 32 ? runs[lane] : make_float2(0.f, -INFINITY));
      runs[lane] = all;
    }
    __syncthreads();
    const float before = warp ? fmaxf(m + runs[warp - 1].x, runs[warp - 1].y) : m;
    const float after = fmaxf(before + run.x, run.y);
    ms[tid] = after;
    __syncthreads();
    if (t < n) p.out[(int64_t)(t0 + t) * p.H + hd] = gates(f, i, tid ? ms[tid - 1] : m, after);
    m = ms[width - 1];
    __syncthreads();
  }
  if (tid == 0) *slot = m;
}

// (token, group of W channels) per group of wpg warps: rms over the group of y (gate first: of y g(z)), times w, (gate last:
// times g(z)), times a constant; w repeats after w_len channels.  NV vectors of V elements per lane stay in registers.
// gates not null (a matrix memory's rows of y, y_row wide): y is first divided by max(|y[n_col]|, gates.z) + 1e-6.
constexpr int GN_NV = 4;
struct RowDivisor { const float4* gates; int n_col; };
template <typename T, int V>
__global__ void __launch_bounds__(1024) gated_norm_kernel(const float* __restrict__ y, int y_row, const T* __restrict__ z,
                                                           int64_t z_stride, const T* __restrict__ w, int w_len, T* __restrict__ out,
                                                           int64_t out_stride, int64_t n_rows, int groups, int W, int gate_first,
                                                           int sigmoid_gate, RowDivisor by, float eps, float scale, int wpg) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per_cta = (blockDim.x >> 5) / wpg, sub = warp / wpg;
  const int64_t row = (int64_t)blockIdx.x * per_cta + sub;
  const bool ok = row < n_rows;
  const int64_t tok = ok ? row / groups : 0;
  const int g = ok ? (int)(row - tok * groups) : 0;
  const float* yr = y + (tok * groups + g) * (int64_t)y_row;
  const T* zr = z + tok * z_stride + (int64_t)g * W;
  const int i0 = ((warp % wpg) * 32 + lane) * V, step = wpg * 32 * V;
  constexpr int dt = DTypeOf<T>::v;
  const float f = by.gates && ok ? 1.f / (fmaxf(fabsf(yr[by.n_col]), by.gates[row].z) + 1e-6f) : 1.f;
  auto gate = [&](float u) { return sigmoid_gate ? __fdividef(1.f, 1.f + __expf(-u)) : silu_f(u); };
  auto load = [&](int i, float (&a)[V], float (&b)[V]) {
    if constexpr (V == 4) {
      const float4 x = *reinterpret_cast<const float4*>(yr + i), u = ld_any4(zr, i, dt);
      a[0] = x.x * f; a[1] = x.y * f; a[2] = x.z * f; a[3] = x.w * f;
      b[0] = gate(u.x); b[1] = gate(u.y); b[2] = gate(u.z); b[3] = gate(u.w);
    } else {
      a[0] = yr[i] * f;
      b[0] = gate(to_f32(zr[i]));
    }
  };
  float a[GN_NV][V], b[GN_NV][V], ss = 0.f;
  auto square = [&](const float (&u)[V], const float (&v)[V]) {
#pragma unroll
    for (int j = 0; j < V; ++j) { const float x = gate_first ? u[j] * v[j] : u[j]; ss += x * x; }
  };
#pragma unroll
  for (int k = 0; k < GN_NV; ++k)
    if (ok && i0 + k * step < W) { load(i0 + k * step, a[k], b[k]); square(a[k], b[k]); }
  for (int i = i0 + GN_NV * step; ok && i < W; i += step) {            // rows too long for the registers
    float u[V], v[V];
    load(i, u, v);
    square(u, v);
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
  const int w0 = w_len > W ? g * W : 0;                                // (w_len is W, a multiple or a divisor of it)
  auto emit = [&](int i, const float (&u)[V], const float (&v)[V]) {
    const int wi = w_len < W ? i % w_len : w0 + i;
    if constexpr (V == 4) {
      const float4 ww = ld_any4(w, wi, dt);
      const float o0 = u[0] * v[0] * ww.x * r, o1 = u[1] * v[1] * ww.y * r, o2 = u[2] * v[2] * ww.z * r, o3 = u[3] * v[3] * ww.w * r;
      if constexpr (dt == DT_F32) *reinterpret_cast<float4*>(orow + i) = make_float4(o0, o1, o2, o3);
      else *reinterpret_cast<uint2*>(orow + i) = make_uint2(pack2<T>(o0, o1), pack2<T>(o2, o3));
    } else {
      orow[i] = from_f32<T>(u[0] * v[0] * to_f32(w[wi]) * r);
    }
  };
#pragma unroll
  for (int k = 0; k < GN_NV; ++k)
    if (i0 + k * step < W) emit(i0 + k * step, a[k], b[k]);
  for (int i = i0 + GN_NV * step; i < W; i += step) {
    float u[V], v[V];
    load(i, u, v);
    emit(i, u, v);
  }
}

template <int NP, int L, int SNP, int SL, int MODE, int Q, int TB, int PRODUCERS>
int scan_launch(ScanParams& p, int num_reqs, int warps, cudaStream_t st) {
  static_assert(NP * L == SNP * SL, "one state layout");
  constexpr int RP = 2 * NP * L, CW = 32 / L * 4 * Q;
  const int CT = warps * CW, per_tok = (head_decay(MODE) ? 2 : 3) * RP + 2 * CT + 4;
  const size_t smem = (size_t)(2 * TB * (per_tok + CT)) * 4;
  if (smem > 200 * 1024) return -4;
  auto kern = state_scan_kernel<NP, L, SNP, SL, MODE, Q, TB, PRODUCERS>;
  static bool set = false;
  if (!set) { cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); set = true; }
  vb_launch(kern, dim3((p.C + CT - 1) / CT, p.H, num_reqs), dim3(32 * (warps + PRODUCERS)), smem, st, p);
  return (int)cudaGetLastError();
}

constexpr int SMS = 148;
// SNP, SL: decode form; NP1, L1 and NP2, L2: prompt forms, few and many rows per lane
template <int SNP, int SL, int NP1, int L1, int NP2, int L2>
int scan_shape(ScanParams& p, int mode, int num_reqs, int max_len, cudaStream_t st) {
  const int head_quads = (p.C + 3) / 4;
  const int64_t quads = (int64_t)num_reqs * p.H * head_quads;           // of the whole launch
  // warps per CTA: at most 8, no more than one head's columns need (``per``: quads of a warp), fewer while SMs would stay empty
  auto cta_warps = [&](int per, int64_t ctas) {
    int w = 1;
    while (w < 8 && w * per < head_quads) w *= 2;
    while (w > 1 && quads / (w * per) < ctas) w /= 2;
    return w;
  };
  if (max_len == 1) {
    // the state's bytes count; two quads per lane keep more of them in flight where there are many states
    constexpr int Q2 = SNP <= 4 ? 2 : 1;
    const bool many = quads / (2 * (32 / SL)) >= 8 * SMS * 3;
    const int w = many ? cta_warps(Q2 * (32 / SL), 1) : cta_warps(32 / SL, SMS);
#define DECODE(M) (many ? scan_launch<SNP, SL, SNP, SL, M, Q2, 1, 4>(p, num_reqs, w, st) : scan_launch<SNP, SL, SNP, SL, M, 1, 1, 4>(p, num_reqs, w, st))
    if (mode == DECAY_HEAD) return DECODE(DECAY_HEAD);
    if (mode == DECAY_GATES) return DECODE(DECAY_GATES);
    if (mode == DECAY_GIVEN) return DECODE(DECAY_GIVEN);
    return DECODE(DECAY_LOWRANK);
#undef DECODE
  }
  if (mode == DECAY_LOWRANK) return -5;                                 // prompts bring their decays
  constexpr int TB = 8;
  constexpr int64_t CTAS = SMS * 3 / 4, WARPS = SMS * 3;                // measured: where the next form begins to win
  // PH: producer warps of the forms with one decay per head; the widest rows of those let two CTAs share an SM
#define PROMPT(NP, L, PH)                                                                                \
  (mode == DECAY_HEAD    ? scan_launch<NP, L, SNP, SL, DECAY_HEAD, 1, TB, PH>(p, num_reqs, w, st)        \
   : mode == DECAY_GATES ? scan_launch<NP, L, SNP, SL, DECAY_GATES, 1, TB, PH>(p, num_reqs, w, st)       \
                         : scan_launch<NP, L, SNP, SL, DECAY_GIVEN, 1, TB, 4>(p, num_reqs, w, st))
  if (quads / (32 / L2) >= WARPS) {
    constexpr int per = 32 / L2;
    int w = cta_warps(per, CTAS);
    if (mode == DECAY_GATES && w >= 4) {                                // the normaliser's quad: one more warp, not one more CTA
      const int tiles = (head_quads - 1 + w * per - 1) / (w * per), need = (head_quads + tiles * per - 1) / (tiles * per);
      if (need == w + 1) w = need;
    }
    return PROMPT(NP2, L2, 2);
  }
  if (quads / (32 / L1) >= WARPS) {
    const int w = cta_warps(32 / L1, CTAS);
    return PROMPT(NP1, L1, 4);
  }
  const int w = cta_warps(32 / SL, CTAS);
  return PROMPT(SNP, SL, 4);
#undef PROMPT
}

inline bool al(const void* p, int64_t n) { return p == nullptr || (reinterpret_cast<uintptr_t>(p) % (size_t)n) == 0; }
inline int esz(int dt) { return dt == DT_F32 ? 4 : 2; }

int scan(ScanParams& p, int mode, int num_reqs, int max_len, cudaStream_t st) {
  if (num_reqs == 0) return 0;
  if (p.R < 1 || p.C < 1 || p.groups < 1 || p.H % p.groups || (mode != DECAY_HEAD && p.groups != p.H)) return -1;
  if (mode != DECAY_GATES) p.CV = p.CO = p.C;
  if (p.state_stride % 4 || p.state_off % 4 || !al(p.state, 16)) return -2;
  p.vec = p.R % 4 == 0 && p.q_stride % 4 == 0 && p.k_stride % 4 == 0 && al(p.q, 4 * esz(p.q_dt)) && al(p.k, 4 * esz(p.k_dt)) &&
          al(p.alpha, 16);
  p.vec_v = p.CV % 4 == 0 && p.v_stride % 4 == 0 && al(p.v, 4 * esz(p.v_dt));
  p.vec_o = p.CO % 4 == 0 && al(p.out, 16);
  p.vec_a = p.rank % 4 == 0 && p.a1_stride % 4 == 0 && al(p.a1, 4 * esz(p.a_dt)) && al(p.a2, 4 * esz(p.a_dt));
  const int rp = p.R <= 16 ? 16 : p.R <= 32 ? 32 : p.R <= 64 ? 64 : p.R <= 128 ? 128 : p.R <= 256 ? 256 : 512;
  if (p.R > 512) return -3;
  p.head_elems = (int64_t)((p.C + 3) / 4) * 4 * rp;
  switch (rp) {
    case 16: return scan_shape<1, 8, 2, 4, 4, 2>(p, mode, num_reqs, max_len, st);
    case 32: return scan_shape<1, 16, 2, 8, 4, 4>(p, mode, num_reqs, max_len, st);
    case 64: return scan_shape<2, 16, 4, 8, 8, 4>(p, mode, num_reqs, max_len, st);
    case 128: return scan_shape<2, 32, 4, 16, 8, 8>(p, mode, num_reqs, max_len, st);
    case 256: return scan_shape<4, 32, 8, 16, 8, 16>(p, mode, num_reqs, max_len, st);
    default: return scan_shape<8, 32, 8, 32, 8, 32>(p, mode, num_reqs, max_len, st);
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

// Matrix memory.  q, k [T, H * R], v [T, H * C] (token strides free); gates [T, H] float4 of vb_memory_gates.  out [T, H, CO] fp32,
// CO = C rounded up to four, plus four: column CO - 4 is n . q.  A head's state has CO columns (vb_state_scan_elems(R, CO)).
EXPORT int vb_memory_scan(const void* q, const void* k, const void* v, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                          float q_scale, const float* gates, float* out, float* state, int64_t state_stride, int64_t state_off,
                          const int* qsl, const int* seq_lens, const int* rows, int64_t rows_stride, int num_reqs, int max_len,
                          int H, int R, int C, int dtype, cudaStream_t st) {
  lattn::ScanParams p = {};
  if (!lattn::al(gates, 16)) return -2;
  p.q = q; p.k = k; p.v = v; p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
  p.q_dt = p.k_dt = p.v_dt = dtype; p.q_scale = q_scale; p.gates = reinterpret_cast<const float4*>(gates);
  p.out = out; p.state = state; p.state_stride = state_stride; p.state_off = state_off;
  p.qsl = qsl; p.seq_lens = seq_lens; p.rows = rows; p.rows_stride = rows_stride;
  p.H = H; p.groups = H; p.R = R; p.CV = C; p.C = p.CO = (C + 3) / 4 * 4 + 4;
  return lattn::scan(p, lattn::DECAY_GATES, num_reqs, max_len, st);
}

// h [T, W] (token stride free), w [2 H, W] (input gates, then forget gates), bias [2 H]; logits [T, 2 H] fp32 without the bias, or
// null where every request has one token.  gates [T, H] float4; the maxima at m_off of the slots advance in place.
EXPORT int vb_memory_gates(const void* h, int64_t h_stride, const void* w, int W, const float* logits, const float* bias, float cap,
                           float* gates, float* state, int64_t state_stride, int64_t m_off, const int* qsl, const int* seq_lens,
                           const int* rows, int64_t rows_stride, int num_reqs, int max_len, int H, int dtype, cudaStream_t st) {
  using namespace lattn;
  if (num_reqs == 0) return 0;
  if (!al(gates, 16) || (!logits && max_len != 1)) return -1;
  GateParams p = {h, h_stride, w, W, logits, bias, cap, reinterpret_cast<float4*>(gates), state, state_stride, m_off, qsl, seq_lens,
                  rows, rows_stride, H};
  const bool vec = W % 4 == 0 && h_stride % 4 == 0 && al(h, 4 * esz(dtype)) && al(w, 4 * esz(dtype));
  const dim3 block(max_len > 2 * GATE_T ? GATE_MAX_T : GATE_T);
  DISPATCH_DTYPE(dtype, T, {
    if (vec) vb_launch(memory_gates_kernel<T, 4>, dim3(num_reqs, H), block, 0, st, p);
    else vb_launch(memory_gates_kernel<T, 1>, dim3(num_reqs, H), block, 0, st, p);
  });
  return (int)cudaGetLastError();
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
// a divisor of W); out [T, groups * W] in the model dtype (token stride free).  flags: bit0 gate first, bit1 sigmoid gate (else
// silu).  gates not null: y holds the rows [T, groups, CO] of vb_memory_scan and gates its gates.
EXPORT int vb_gated_norm(const float* y, const float* gates, const void* z, int64_t z_stride, const void* w, int w_len, void* out,
                         int64_t out_stride, int T_, int groups, int W, int flags, float eps, float scale, int dtype,
                         cudaStream_t st) {
  using namespace lattn;
  if (T_ == 0) return 0;
  const int64_t rows = (int64_t)T_ * groups;
  const int e = esz(dtype);
  const int n_col = (W + 3) / 4 * 4, y_row = gates ? n_col + 4 : W;
  const RowDivisor by = {reinterpret_cast<const float4*>(gates), n_col};
  const bool vec = W % 4 == 0 && w_len % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0 && al(y, 16) && al(z, 4 * e) &&
                   al(w, 4 * e) && al(out, 4 * e);
  const int per_warp = vec ? 32 * 4 * GN_NV : 32 * GN_NV;
  int wpg = 1;
  while (wpg < 32 && wpg * per_warp < W) wpg *= 2;
  const int warps = wpg > 8 ? wpg : 8, per_cta = warps / wpg;
  dim3 grid((unsigned)((rows + per_cta - 1) / per_cta)), block(warps * 32);
#define GO(V) vb_launch(gated_norm_kernel<T, V>, grid, block, 0, st, y, y_row, (const T*)z, z_stride, (const T*)w, w_len, (T*)out, out_stride, rows, groups, W, flags & 1, flags >> 1 & 1, by, eps, scale, wpg)
  DISPATCH_DTYPE(dtype, T, { if (vec) GO(4); else GO(1); });
#undef GO
  return (int)cudaGetLastError();
}
