// Attention whose heads talk to one another: the weights of all heads are mixed behind the softmax,
//
//   out_h(i) = sum_j ( sum_g T[h, g] w_g(i, j) ) V_c(h)(j)  =  sum_g T[h, g]  O_{g, c(h)}(i),      O_{g, c}(i) = sum_j w_g(i, j) V_c(j)
//
// (c(h): the KV head of h).  The mix is linear, so it can wait until the keys are summed up: the attention kernels produce O_{g, c}, every
// query head with the values of every KV head ("fold"), in one pass over the keys, and talk_mix applies T to H x vdim numbers per token
// instead of H x H numbers per key.  (Mixing the weights themselves needs the denominators first, hence a second pass over the scores, and
// H multiplications per weight on the CUDA cores: more time than the tensor cores take for the additional values.)
//
//   talk_fold   prompts: tcgen05 on pairs of CTAs (cta_group::2), 256 rows (tokens x heads of one KV head), two value heads
//   talk_mix    T, split-KV sums and denominators, the turn back of rotated values, 16-bit output
// Decode steps: attention_talk_decode.cu; other head shapes and dtypes: attention_any.cu.
//
// Scores are capped, cap tanh(s / cap), with cap <= 60: e^s then fits into fp32 (and bf16) whatever the score is, and the softmax needs no
// running maximum: one pass over S, no rescaling, and partial sums of different key ranges simply add up.
#include "common.cuh"
#include "talk.cuh"

namespace talk {

constexpr int D = 128, BS = 64, TM = 128, TN = 128;
constexpr int SOFTMAX_WARPS = 16, NUM_THREADS = 64 + SOFTMAX_WARPS * 32;
constexpr int K_STAGES = 4, V_STAGES = 3;
constexpr int Q_BYTES = TM * D * 2;             // 32 KB: 2 k-blocks of [128 rows x 64]
constexpr int K_BYTES = BS * D * 2;             // 16 KB: this CTA's page of a key tile, 2 k-blocks of [64 tokens x 64]
constexpr int V_BYTES = 2 * 128 * 128;          // 32 KB: this CTA's value rows of a tile, 2 pages of [up to 128 rows x 64 tokens]

struct Params {
  const int* block_table; const int* seq_lens; const int* qsl;
  void* out;                    // [T, Hq, nc, D], normalised
  const float* sinks;           // optional [Hq]
  int bt_stride, Hq, Hkv, G, TQ, window, c0, nc;
  int per_cta;                  // pairs of value heads that a pair of CTAs does one after the other
  Cap cap;
  int* error;
};

VB_DEVICE void tmem_st_32x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
VB_DEVICE void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// ---- pairs of CTAs: one MMA over the rows of both, issued by the leader (rank 0).  Each CTA holds its own rows of A and D, and half of
// the N rows of B.
// D[tmem] (+)= A * B; A from shared memory, or from TMEM (row = lane, two 16-bit values per column).  The whole warp calls these and one
// lane is elected inside: descriptors stay in uniform registers, an MMA behind a lane test takes a hundred cycles to issue.
VB_DEVICE void umma2_f16(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
  asm volatile("{\n\t.reg .pred p, q;\n\telect.sync _|q, 0xffffffff;\n\tsetp.ne.b32 p, %4, 0;\n\t"
               "@q tcgen05.mma.cta_group::2.kind::f16 [%0], %1, %2, %3, p;\n\t}"
               ::"r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate) : "memory");
}
VB_DEVICE void umma2_f16_ta(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
  asm volatile("{\n\t.reg .pred p, q;\n\telect.sync _|q, 0xffffffff;\n\tsetp.ne.b32 p, %4, 0;\n\t"
               "@q tcgen05.mma.cta_group::2.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
               ::"r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate) : "memory");
}
// arrives on the barrier at this offset in both CTAs once the MMAs issued before have completed
VB_DEVICE void umma2_commit(uint64_t* bar) {
  asm volatile("{\n\t.reg .pred q;\n\telect.sync _|q, 0xffffffff;\n\t"
               "@q tcgen05.commit.cta_group::2.mbarrier::arrive::one.shared::cluster.multicast::cluster.b64 [%0], %1;\n\t}"
               ::"r"(smem_u32(bar)), "h"((uint16_t)3) : "memory");
}
// loads into this CTA's shared memory and counts the bytes on a barrier of the pair (a shared::cluster address)
VB_DEVICE void tma2_load_2d(void* dst, const void* tmap, int c0, int c1, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.2d.cta_group::2.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
               ::"r"(smem_u32(dst)), "l"(tmap), "r"(bar), "r"(c0), "r"(c1) : "memory");
}
VB_DEVICE void tma2_load_3d(void* dst, const void* tmap, int c0, int c1, int c2, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.3d.cta_group::2.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
               ::"r"(smem_u32(dst)), "l"(tmap), "r"(bar), "r"(c0), "r"(c1), "r"(c2) : "memory");
}
VB_DEVICE void tmem2_alloc(uint32_t* smem_dst, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::2.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(smem_dst)), "r"(ncols) : "memory");
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::2.sync.aligned;" ::: "memory");
}
VB_DEVICE void tmem2_dealloc(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::2.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}
VB_DEVICE void arrive_cluster(uint32_t bar) {
  asm volatile("mbarrier.arrive.shared::cluster.b64 _, [%0];" ::"r"(bar) : "memory");
}
VB_DEVICE void wait_cluster_lim(uint64_t* bar, uint32_t parity, int& budget) {      // what threads of the other CTA have arrived on
  for (;;) {
    uint32_t ok;
    asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                 : "=r"(ok) : "r"(smem_u32(bar)), "r"(parity) : "memory");
    if (ok || --budget < 0) break;
  }
}

// Pair of CTAs = two query tiles in a row x KV head of the scores x some pairs of value heads (one after the other), one request.  Both
// tiles read the same keys and values; each CTA fetches half of them (a page of the key tile; one value head, or half of a single one).
// Warp roles: 0 TMA producer, 1 MMA issuer (leader) + TMEM owner, 2..17 softmax / epilogue (thread = query row = TMEM lane, a quarter of
// the columns: four warps per scheduler, since one alone waits for its own results most of the time).  TMEM: S double-buffered (2 x 128
// columns), two accumulators (2 x 128).  P overwrites the S it came from (bf16, 16 of each 32 columns) and is the PV product's A operand
// there, so it is double-buffered too: the softmax of tile n runs under the PV products of tile n - 1.  Tiles are numbered through over
// the pairs of value heads: the first scores of the next pair are computed while the last results of this one are stored.
__global__ void __launch_bounds__(NUM_THREADS, 1)
talk_fold_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                 const __grid_constant__ CUtensorMap tmap_v, const Params p) {
  using T = __nv_bfloat16;
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* q_smem = smem;
  unsigned char* k_smem = q_smem + Q_BYTES;
  unsigned char* v_smem = k_smem + K_STAGES * K_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_smem + V_STAGES * V_BYTES);
  uint64_t* q_full = bars;                     // the leader's count the bytes of both CTAs
  uint64_t* k_full = bars + 1;                 // [K_STAGES] (leader's)
  uint64_t* k_empty = k_full + K_STAGES;
  uint64_t* v_full = k_empty + K_STAGES;       // [V_STAGES] (leader's)
  uint64_t* v_empty = v_full + V_STAGES;
  uint64_t* s_full = v_empty + V_STAGES;       // [2]
  uint64_t* p_full = s_full + 2;               // [2] (leader's: the warps of both CTAs)
  uint64_t* o_full = p_full + 2;
  uint64_t* o_empty = o_full + 1;              // (leader's: the warps of both CTAs)
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_empty + 1);
  float* sums = reinterpret_cast<float*>(tmem_slot + 2);        // 2 x [4][128] sums of the column quarters

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int budget = MBAR_BUDGET;
  const int rank = (int)cluster_ctarank(), b = blockIdx.z, groups = (p.nc + 1) / 2;
  const int parts = (groups + p.per_cta - 1) / p.per_cta;
  const int h = blockIdx.y / parts, g0 = blockIdx.y % parts * p.per_cta; // KV head of the scores, first pair of value heads
  const int ng = min(p.per_cta, groups - g0);
  auto heads_of = [&](int ci) { return min(2, p.nc - (g0 + ci) * 2); };  // value heads of pair ci: two, or one at the end
  pdl_trigger();
  pdl_wait();
  const int q0 = p.qsl[b], q_len = p.qsl[b + 1] - q0;
  const int pair0 = ((int)blockIdx.x & ~1) * p.TQ, tok0 = blockIdx.x * p.TQ;
  if (pair0 >= q_len) return;                                            // uniform across the pair
  const int n_tok = min(p.TQ, q_len - tok0);                             // <= 0: the pair's second tile is empty
  const int ctx = p.seq_lens[b] - q_len, pos0 = ctx + tok0;
  const int kv_end = ctx + min(q_len, pair0 + 2 * p.TQ), kv_begin = p.window > 0 ? max(0, ctx + pair0 - p.window + 1) : 0;
  const int tile_lo = kv_begin / TN, n_tiles = (kv_end + TN - 1) / TN - tile_lo;
  const int n_pages = (kv_end + BS - 1) / BS;

  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tmap_q); tma_prefetch_desc(&tmap_k); tma_prefetch_desc(&tmap_v);
    mbar_init(q_full, 1);
    for (int s = 0; s < K_STAGES; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); }
    for (int s = 0; s < V_STAGES; ++s) { mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
    for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&p_full[s], 2 * SOFTMAX_WARPS); }
    mbar_init(o_full, 1);
    mbar_init(o_empty, 2 * SOFTMAX_WARPS);
    mbar_fence_init();
  }
  if (warp == 1) tmem2_alloc(tmem_slot, 512);
  tc_fence_before();
  __syncthreads();
  cluster_sync();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot, tmem_o = tmem_base + 256;

  if (warp == 0) {
    if (lane == 0) {
      // ===== TMA producer of this CTA's halves.  Tiles are always whole: pages past the sequence are read from the null page (finite,
      // masked)
      const uint32_t bar_q = dsmem_addr(smem_u32(q_full), 0);
      if (rank == 0) mbar_expect_tx(q_full, 2 * Q_BYTES);
      tma2_load_3d(q_smem, &tmap_q, 0, h * p.G, q0 + tok0, bar_q);
      tma2_load_3d(q_smem + TM * 128, &tmap_q, 64, h * p.G, q0 + tok0, bar_q);
      const int* bt = p.block_table + (int64_t)b * p.bt_stride;
      const int total = ng * n_tiles;
      for (int n = 0, j = 0, ci = 0; n < total; ++n) {
        const int cv = (g0 + ci) * 2, nv = heads_of(ci), v_rows = nv * 64;      // rows of a value tile's B operand in this CTA
        int blk[2];
        for (int u = 0; u < 2; ++u) {
          const int page = (tile_lo + j) * 2 + u;
          blk[u] = page < n_pages ? bt[page] : 0;
        }
        const int s = n % K_STAGES, vs = n % V_STAGES;
        mbar_wait_lim(&k_empty[s], ((n / K_STAGES) & 1) ^ 1, budget);
        if (budget < 0) break;
        const uint32_t bar_k = dsmem_addr(smem_u32(&k_full[s]), 0);
        if (rank == 0) mbar_expect_tx(&k_full[s], 2 * K_BYTES);
        for (int kb = 0; kb < 2; ++kb)
          tma2_load_2d(k_smem + s * K_BYTES + kb * (BS * 128), &tmap_k, kb * 64, ((rank ? blk[1] : blk[0]) * 2 * p.Hkv + h) * BS, bar_k);
        mbar_wait_lim(&v_empty[vs], ((n / V_STAGES) & 1) ^ 1, budget);
        if (budget < 0) break;
        const uint32_t bar_v = dsmem_addr(smem_u32(&v_full[vs]), 0);
        if (rank == 0) mbar_expect_tx(&v_full[vs], 2 * 2 * v_rows * 128);
        for (int u = 0; u < 2; ++u) {
          // two value heads: the CTA's own, 128 rows; one: half of its rows
          const int row = ((blk[u] * 2 + 1) * p.Hkv + p.c0 + cv + (nv == 2 ? rank : 0)) * D + (nv == 2 ? 0 : rank * 64);
          for (int r = 0; r < v_rows; r += 64) tma2_load_2d(v_smem + vs * V_BYTES + (u * v_rows + r) * 128, &tmap_v, 0, row + r, bar_v);
        }
        if (++j == n_tiles) { j = 0; ++ci; }
      }
      if (budget < 0 && rank == 0) {            // let the copies in flight land before the pair gives up its memory
        for (int s = 0; s < K_STAGES; ++s)
          for (int n = 0; n < 4096 && !(mbar_try_wait(&k_full[s], 0) || mbar_try_wait(&k_full[s], 1)); ++n) {}
        for (int s = 0; s < V_STAGES; ++s)
          for (int n = 0; n < 4096 && !(mbar_try_wait(&v_full[s], 0) || mbar_try_wait(&v_full[s], 1)); ++n) {}
      }
    }
  } else if (warp == 1) {
    if (rank == 0) {
      // ===== MMA issuer.  MMAs of one thread execute in order, so QK of tile j may follow PV of tile j - 2, whose P it overwrites, at once:
      // the tensor cores always have the next product queued while this thread waits
      const uint32_t idesc_s = umma_idesc_f16(2 * TM, TN, true);
      const uint64_t d_q = umma_desc_sw128(q_smem), d_k = umma_desc_sw128(k_smem), d_v = umma_desc_sw128(v_smem);
      mbar_wait_lim(q_full, 0, budget);
      const int nt = __shfl_sync(0xffffffffu, n_tiles, 0), total = ng * nt;        // (uniform)
      for (int n = 0, jj = 0, ci = 0; n <= total; ++n) {
        if (n < total) {
          const int s = n % K_STAGES;
          mbar_wait_lim(&k_full[s], (n / K_STAGES) & 1, budget);
          __syncwarp();
          tc_fence_after();
#pragma unroll
          for (int kb = 0; kb < 2; ++kb)
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma2_f16(tmem_base + (n & 1) * 128, d_q + (uint64_t)(((kb * TM * 128) >> 4) + k * 2),
                        d_k + (uint64_t)(((s * K_BYTES + kb * BS * 128) >> 4) + k * 2), idesc_s, (kb | k) != 0);
          umma2_commit(&s_full[n & 1]);
          umma2_commit(&k_empty[s]);
        }
        if (n > 0) {
          const int m = n - 1, vs = m % V_STAGES, nv = heads_of(ci);     // tile jj of pair ci
          const uint32_t idesc_o = umma_idesc_f16(2 * TM, nv * 128, true);
          if (jj == 0 && ci > 0) wait_cluster_lim(o_empty, (ci - 1) & 1, budget);
          mbar_wait_lim(&v_full[vs], (m / V_STAGES) & 1, budget);
          wait_cluster_lim(&p_full[m & 1], (m >> 1) & 1, budget);
          __syncwarp();
          tc_fence_after();
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            umma2_f16_ta(tmem_o, tmem_base + (m & 1) * 128 + (kk / 2) * 32 + (kk & 1) * 8,
                         d_v + (uint64_t)((vs * V_BYTES + (kk / 4) * nv * 64 * 128) >> 4) + (uint64_t)((kk & 3) * 2), idesc_o, (jj | kk) != 0);
          umma2_commit(&v_empty[vs]);
          if (++jj == nt) { umma2_commit(o_full); jj = 0; ++ci; }
        }
      }
    }
  } else {
    // ===== softmax / epilogue
    const int qd = warp & 3, r = qd * 32 + lane, quarter = (warp - 2) >> 2, c0 = quarter * 32;
    const uint32_t t_lane = (uint32_t)(qd * 32) << 16;
    const uint32_t bar_p = dsmem_addr(smem_u32(p_full), 0), bar_o = dsmem_addr(smem_u32(o_empty), 0);
    const int tq = r / p.G, g = r % p.G, hq = h * p.G + g;
    const bool row_valid = tq < n_tok;
    const int qpos = pos0 + tq;
    const float sink = p.sinks && row_valid ? ex2(p.sinks[hq] * 1.4426950408889634f) : 0.f;
    int n = 0;
    for (int ci = 0; ci < ng; ++ci) {
      float l_run = 0.f;
      for (int j = 0; j < n_tiles; ++j, ++n) {
        const uint32_t t_s = tmem_base + (n & 1) * 128 + c0 + t_lane;
        const int first = (tile_lo + j) * TN + c0;
        const int hi = row_valid ? qpos + 1 - first : 0;                 // keys [lo, hi) of these 32 are visible to the row
        const int lo = p.window > 0 ? hi - p.window : 0;
        const bool full = __all_sync(0xffffffffu, hi >= 32 && lo <= 0) != 0;
        const bool none = __all_sync(0xffffffffu, hi <= 0 || lo >= 32) != 0;
        mbar_wait_lim(&s_full[n & 1], (n >> 1) & 1, budget);
        __syncwarp();
        tc_fence_after();
        uint32_t pk[16];
        if (none) {
#pragma unroll
          for (int i = 0; i < 16; ++i) pk[i] = 0u;
        } else {
          uint32_t v[32];
          tmem_ld_32x32(t_s, v);
          tmem_ld_wait();
          float s[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) s[i] = __uint_as_float(v[i]);
          cap_exp<32>(s, p.cap);
          if (!full) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (i >= hi || i < lo) s[i] = 0.f;
          }
          uint64_t l[2] = {0ull, 0ull};
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            l[(i >> 1) & 1] = add2(l[(i >> 1) & 1], pair2(s[i], s[i + 1]));
            pk[i / 2] = pack2<T>(s[i], s[i + 1]);
          }
          const float2 lt = split2(add2(l[0], l[1]));
          l_run += lt.x + lt.y;
        }
        tmem_st_32x16(t_s, pk);
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) arrive_cluster(bar_p + (n & 1) * 8);
      }
      // ---- epilogue of a pair of value heads
      float* sm = sums + (ci & 1) * 512;
      sm[quarter * 128 + r] = l_run;
      asm volatile("bar.sync 1, 512;" ::: "memory");
      const float den = (sm[r] + sm[128 + r]) + (sm[256 + r] + sm[384 + r]) + sink;
      const float inv = row_valid && den > 0.f ? 1.f / den : 0.f;
      mbar_wait_lim(o_full, ci & 1, budget);
      __syncwarp();
      tc_fence_after();
      // two value heads: half of each per quarter of the warps; one: a quarter of it
      const int cv = (g0 + ci) * 2;
      T* orow = reinterpret_cast<T*>(p.out) + (((int64_t)(q0 + tok0 + tq) * p.Hq + hq) * p.nc + cv) * D;
      auto store = [&](const uint32_t (&o)[32], int at) {               // 32 columns of the row, whole sectors
        if (!row_valid) return;
#pragma unroll
        for (int i = 0; i < 32; i += 16) {
          uint32_t w[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) w[e] = pack2<T>(__uint_as_float(o[i + 2 * e]) * inv, __uint_as_float(o[i + 2 * e + 1]) * inv);
          asm volatile("st.global.v8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(orow + at + i), "r"(w[0]), "r"(w[1]), "r"(w[2]), "r"(w[3]),
                       "r"(w[4]), "r"(w[5]), "r"(w[6]), "r"(w[7]) : "memory");
        }
      };
      auto release = [&]() {                                            // the accumulators are in registers
        tmem_ld_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) arrive_cluster(bar_o);
      };
      uint32_t o0[32];
      if (heads_of(ci) == 2) {
        uint32_t o1[32];
        tmem_ld_32x32(tmem_o + quarter * 64 + t_lane, o0);
        tmem_ld_32x32(tmem_o + quarter * 64 + 32 + t_lane, o1);
        release();
        store(o0, quarter * 64);
        store(o1, quarter * 64 + 32);
      } else {
        tmem_ld_32x32(tmem_o + quarter * 32 + t_lane, o0);
        release();
        store(o0, quarter * 32);
      }
    }
    tc_fence_before();
  }
  __syncwarp();
  tc_fence_before();
  cluster_sync();                               // nobody leaves while the other CTA may still arrive on its barriers
  if (warp == 1) tmem2_dealloc(tmem_base, 512);
  if (budget < 0 && p.error) *p.error = 1;
}

// out[t, h, :] = turn_back( sum_g T[h, g] / den_g * sum_s o[s, t, g, c(h) - c0, :] ).  CTA = token x some value heads; thread = VP pairs of
// one value head, all heads of that KV head in tiles of four.  den null sums: o is normalised.
struct MixParams {
  const void* o; const float* l; const float* sinks; const float* talk;
  const int64_t* positions; const float* cos_sin;        // optional [positions, DV]: pair m turns by minus its angle
  void* out; int64_t out_stride;
  int T, H, G, DV, S, c0, nc, neox;
};
template <typename TO, int N> VB_DEVICE void load_n(const TO* p, float (&f)[N]) {
  if constexpr (N == 1) {
    f[0] = to_f32(p[0]);
  } else if constexpr (sizeof(TO) == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w;
  } else {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack2<TO>(x.x), c = unpack2<TO>(x.y);
    f[0] = a.x; f[1] = a.y; f[2] = c.x; f[3] = c.y;
  }
}
template <typename TO, typename T, int VP>
__global__ void __launch_bounds__(256) talk_mix_kernel(const MixParams p) {
  extern __shared__ float w[];                           // [nc here * G][H], then 1 / den [H]
  pdl_trigger();
  const int cpb = (p.nc + gridDim.y - 1) / gridDim.y, cb = blockIdx.y * cpb, ncb = min(cpb, p.nc - cb);
  if (ncb <= 0) return;
  const int rows = ncb * p.G, t = blockIdx.x, H = p.H;
  float* inv = w + cpb * p.G * H;
  pdl_wait();
  for (int g = threadIdx.x; g < H; g += blockDim.x) {
    float den = 1.f;
    if (p.l) {
      den = p.sinks ? expf(p.sinks[g]) : 0.f;
      for (int s = 0; s < p.S; ++s) den += p.l[((int64_t)s * p.T + t) * H + g];
    }
    inv[g] = den > 0.f ? 1.f / den : 0.f;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < rows * H; i += blockDim.x) w[i] = p.talk[(int64_t)(p.c0 + cb) * p.G * H + i] * inv[i % H];
  __syncthreads();
  const int half = p.DV / 2, per = half / VP;
  const float* cs = p.cos_sin ? p.cos_sin + p.positions[t] * p.DV : nullptr;
  const int64_t split = (int64_t)p.T * H * p.nc * p.DV;
  for (int it = threadIdx.x; it < ncb * per; it += blockDim.x) {
    const int c = it / per, m = (it - c * per) * VP;
    // VP > 1: pairs (m, m + half), also where nothing turns; else the layout of the rotation
    const bool halves = VP > 1 || p.neox;
    const int e0 = halves ? m : 2 * m, e1 = halves ? m + half : 2 * m + 1;
    const TO* o = reinterpret_cast<const TO*>(p.o) + ((int64_t)t * H * p.nc + cb + c) * p.DV;
    for (int j0 = 0; j0 < p.G; j0 += 4) {
      const int nj = min(4, p.G - j0);
      float a[4][VP], bq[4][VP];
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int q = 0; q < VP; ++q) { a[j][q] = 0.f; bq[j][q] = 0.f; }
      const float* wj = w + (c * p.G + j0) * H;
      for (int s = 0; s < p.S; ++s) {
#pragma unroll 4
        for (int g = 0; g < H; ++g) {
          float x[VP], y[VP];
          const TO* src = o + s * split + (int64_t)g * p.nc * p.DV;
          load_n<TO, VP>(src + e0, x);
          load_n<TO, VP>(src + e1, y);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float k = wj[(j < nj ? j : 0) * H + g];
#pragma unroll
            for (int q = 0; q < VP; ++q) { a[j][q] += k * x[q]; bq[j][q] += k * y[q]; }
          }
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j >= nj) break;
        T* dst = reinterpret_cast<T*>(p.out) + t * p.out_stride + (int64_t)((p.c0 + cb + c) * p.G + j0 + j) * p.DV;
        if (cs) {
#pragma unroll
          for (int q = 0; q < VP; ++q) {
            const float co = cs[m + q], si = cs[half + m + q], x = a[j][q], y = bq[j][q];
            a[j][q] = x * co + y * si;
            bq[j][q] = y * co - x * si;
          }
        }
        if constexpr (VP == 1) {
          dst[e0] = from_f32<T>(a[j][0]);
          dst[e1] = from_f32<T>(bq[j][0]);
        } else if constexpr (sizeof(T) == 4) {
          *reinterpret_cast<float4*>(dst + e0) = make_float4(a[j][0], a[j][1], a[j][2], a[j][3]);
          *reinterpret_cast<float4*>(dst + e1) = make_float4(bq[j][0], bq[j][1], bq[j][2], bq[j][3]);
        } else {
          *reinterpret_cast<uint2*>(dst + e0) = make_uint2(pack2<T>(a[j][0], a[j][1]), pack2<T>(a[j][2], a[j][3]));
          *reinterpret_cast<uint2*>(dst + e1) = make_uint2(pack2<T>(bq[j][0], bq[j][1]), pack2<T>(bq[j][2], bq[j][3]));
        }
      }
    }
  }
}

template <typename TO, typename T>
static int launch_mix(const MixParams& p, cudaStream_t st) {
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  // decode batches: one value head per CTA, so that there are enough of them
  const bool few = p.T <= 512;
  const bool vec = !few && (p.neox || !p.cos_sin) && p.DV % 8 == 0 && p.out_stride % 8 == 0 && al(p.o) && al(p.out);
  const int cpb = few ? 1 : p.nc, per = p.DV / 2 / (vec ? 4 : 1), items = cpb * per;
  const int thr = items >= 256 ? 256 : (items < 64 ? 64 : (items + 31) / 32 * 32);
  const size_t smem = ((size_t)cpb * p.G + 1) * p.H * 4;
  if (smem > 200 * 1024) return -3;
  const dim3 grid(p.T, (p.nc + cpb - 1) / cpb);
#define GO(N)                                                                                                   \
  do {                                                                                                          \
    auto k = talk_mix_kernel<TO, T, N>;                                                                         \
    static bool set = false;                                                                                    \
    if (!set) { cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); set = true; } \
    vb_launch(k, grid, dim3(thr), smem, st, p);                                                                 \
  } while (0)
  if (vec) GO(4); else GO(1);
#undef GO
  return (int)cudaGetLastError();
}

}  // namespace talk

// q [T, Hq * 128] (token stride free), kv_cache [nb, 2, Hkv, 64 x 128] with transposed value pages, bf16; out [T, Hq, nc, 128]: the
// normalised attention of every query head with the values of KV heads c0 .. c0 + nc - 1.  0 < soft_cap <= 60.
EXPORT int vb_talk_fold(const void* q, const void* kv_cache, int64_t num_blocks, const int* block_table, const int* seq_lens,
                        const int* qsl, void* out, int* error, int B, int T_total, int max_q_len, int Hq, int Hkv, int64_t q_stride,
                        int bt_stride, int window, float scale, float soft_cap, const float* sinks, int c0, int nc, cudaStream_t st) {
  using namespace talk;
  if (B == 0 || max_q_len <= 0) return 0;
  const int G = Hq / Hkv;
  if (G < 1 || G > 128 || 128 % G || Hq % Hkv || c0 < 0 || nc < 1 || c0 + nc > Hkv || q_stride % 8) return -4;
  if (!(soft_cap > 0.f && soft_cap <= MAX_CAP)) return -5;
  Params p;
  p.block_table = block_table; p.seq_lens = seq_lens; p.qsl = qsl; p.out = out; p.sinks = sinks; p.bt_stride = bt_stride; p.Hq = Hq;
  p.Hkv = Hkv; p.G = G; p.TQ = TM / G; p.window = window; p.c0 = c0; p.nc = nc; p.cap = make_cap(scale, soft_cap); p.error = error;
  CUtensorMap tq, tk, tv;
  int rc;
  if ((rc = map_queries(&tq, q, Hq, T_total, q_stride, G, p.TQ))) return rc;
  if ((rc = map_pages(&tk, &tv, kv_cache, num_blocks, Hkv, BS, 64))) return rc;
  const int smem = Q_BYTES + K_STAGES * K_BYTES + V_STAGES * V_BYTES + 32 * 8 + 16 + 4096 + 1024;
  static bool a = false;
  if (!a) { cudaFuncSetAttribute(talk_fold_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem); a = true; }
  const int pairs = (max_q_len + 2 * p.TQ - 1) / (2 * p.TQ), groups = (nc + 1) / 2;
  static int n_sms = 0;
  if (!n_sms) { int dv = 0; cudaGetDevice(&dv); cudaDeviceGetAttribute(&n_sms, cudaDevAttrMultiProcessorCount, dv); }
  // all pairs of value heads in one CTA where that still makes a few waves
  const int64_t ctas = (int64_t)2 * pairs * Hkv * B;
  p.per_cta = groups;
  while (p.per_cta > 1 && ctas * ((groups + p.per_cta - 1) / p.per_cta) < 4 * n_sms) p.per_cta = (p.per_cta + 1) / 2;
  if (B > 65535) return -6;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(2 * pairs, Hkv * ((groups + p.per_cta - 1) / p.per_cta), B); cfg.blockDim = dim3(NUM_THREADS); cfg.dynamicSmemBytes = (size_t)smem; cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 2; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;      // the pair is two neighbours along x
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = vb_pdl_enabled() ? 2 : 1;
  cudaLaunchKernelEx(&cfg, talk_fold_kernel, tq, tk, tv, p);
  return (int)cudaGetLastError();
}

// o [S, T, H, nc, DV] in fp32 (o_dtype DT_F32) or bf16; l [S, T, H]: sums of the weights (the denominators but for the sinks [H]) where o
// is not normalised yet; talk [H, H] fp32; writes heads c0 * G .. (c0 + nc) * G - 1 of out [T, H, DV] (token stride free).
EXPORT int vb_talk_mix(const void* o, int o_dtype, const float* l, const float* sinks, const float* talk_w, const int64_t* positions,
                       const float* cos_sin, int neox, void* out, int64_t out_stride, int T_, int H, int G, int DV, int S, int c0, int nc,
                       int dtype, cudaStream_t st) {
  using namespace talk;
  if (T_ == 0) return 0;
  if (DV < 2 || DV % 2 || H % G || S < 1 || nc < 1 || (c0 + nc) * G > H || (cos_sin && !positions)) return -1;
  MixParams p = {o, l, sinks, talk_w, positions, cos_sin, out, out_stride, T_, H, G, DV, S, c0, nc, neox};
  if (o_dtype == DT_BF16) return dtype == DT_BF16 ? launch_mix<__nv_bfloat16, __nv_bfloat16>(p, st) : -2;
  if (o_dtype != DT_F32) return -2;
  DISPATCH_DTYPE(dtype, T, return (launch_mix<float, T>(p, st)));
  return 0;
}
