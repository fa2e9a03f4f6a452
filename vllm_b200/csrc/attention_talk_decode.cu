// Decode attention with mixed heads (see attention_talk.cu for the form): one token per request, every query head with the values of every
// KV head.  "Swap-AB" as in attention_tc_decode.cu, but a CTA takes ALL heads of a request, so that keys and values are read once:
//
//   S^T_a[tok, g]  = K_a[tok, :] . Q_a[g, :]^T        for every KV head a   (M = 128 tokens, N = 16: its query heads, padded)
//   O^T_c[d, h]   += V_c^T[d, tok] . P[h, tok]^T      for every KV head c   (M = 128 dims, N = all query heads, padded)
//
// Capped scores need no maximum (talk.cuh): thread = token, one exponential per head, no exchange between threads until the end, and the
// partial sums of splits add up (talk_mix does that and divides).  Key and value tiles go through one ring of 32 KB slots in the order in
// which the products consume them: keys of tile j, then values of tile j - 1.
#include "common.cuh"
#include "talk.cuh"

namespace talkdec {

using talk::Cap;
constexpr int D = 128, BS = 64, TILE = 128, NQ = 16;
constexpr int NUM_THREADS = 192;
constexpr int SLOTS = 5, MAX_KV = 8;
constexpr int TILE_BYTES = TILE * D * 2;
constexpr int Q_BYTES = NQ * D * 2;              // per KV head: 2 k-blocks of [16 x 64]

struct Params {
  const int* block_table; const int* seq_lens;
  float* part_o;                // [S, B, H, G, D]
  float* part_l;                // [S, B, H]
  int bt_stride, B, H, Hkv, splits, window;
  Cap cap;
  int* error;
};

VB_DEVICE void tma_load_3d(void* dst, const void* tmap, int c0, int c1, int c2, uint64_t* bar) {
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
               ::"r"(smem_u32(dst)), "l"(tmap), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2) : "memory");
}
VB_DEVICE void bar_sync_softmax() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

// GH query heads per KV head, HP: all query heads, padded to 16 or 32
template <int GH, int HP>
__global__ void __launch_bounds__(NUM_THREADS, 1)
talk_decode_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                   const __grid_constant__ CUtensorMap tmap_v, const Params p) {
  using T = __nv_bfloat16;
  constexpr int P_BYTES = HP * TILE * 2;         // 2 k-blocks of [HP x 64 tokens]
  constexpr int GA = HP / GH < MAX_KV ? HP / GH : MAX_KV;
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* ring = smem;
  unsigned char* p_smem = ring + SLOTS * TILE_BYTES;          // 2 buffers
  unsigned char* q_smem = p_smem + 2 * P_BYTES;               // Hkv blocks
  uint64_t* bars = reinterpret_cast<uint64_t*>(q_smem + p.Hkv * Q_BYTES);
  uint64_t* q_full = bars;
  uint64_t* full = bars + 1;                     // [SLOTS]
  uint64_t* empty = full + SLOTS;
  uint64_t* s_full = empty + SLOTS;              // [2]
  uint64_t* s_empty = s_full + 2;
  uint64_t* p_full = s_empty + 2;                // [2]
  uint64_t* pv_done = p_full + 2;                // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 2);
  float* red = reinterpret_cast<float*>(tmem_slot + 2);       // [4][HP]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int budget = MBAR_BUDGET;
  const int G = p.Hkv, split = blockIdx.x, b = blockIdx.y;
  pdl_trigger();
  pdl_wait();
  const int seq_len = p.seq_lens[b];
  const int kv_begin = p.window > 0 ? max(0, seq_len - p.window) : 0;
  int tile_lo = kv_begin / TILE, tile_hi = (seq_len + TILE - 1) / TILE;
  {
    const int per = (tile_hi - tile_lo + p.splits - 1) / p.splits;
    tile_lo += split * per;
    tile_hi = min(tile_hi, tile_lo + per);
  }
  const int n_tiles = max(tile_hi - tile_lo, 0);
  const int64_t row0 = ((int64_t)split * p.B + b) * p.H;
  if (n_tiles == 0) {                            // uniform across the CTA
    for (int i = threadIdx.x; i < p.H * G * D; i += NUM_THREADS) p.part_o[row0 * G * D + i] = 0.f;
    for (int i = threadIdx.x; i < p.H; i += NUM_THREADS) p.part_l[row0 + i] = 0.f;
    return;
  }
  const uint32_t used = 2 * G * NQ + G * HP;
  const uint32_t cols = used <= 64 ? 64 : (used <= 128 ? 128 : (used <= 256 ? 256 : 512));
  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tmap_q); tma_prefetch_desc(&tmap_k); tma_prefetch_desc(&tmap_v);
    mbar_init(q_full, 1);
    for (int s = 0; s < SLOTS; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&s_empty[s], 128); mbar_init(&p_full[s], 128); mbar_init(&pv_done[s], 1); }
    mbar_fence_init();
  }
  if (warp == 1) tmem_alloc(tmem_slot, cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot, tmem_o = tmem_base + 2 * G * NQ;

  if (warp == 0) {
    if (lane == 0) {
      // ===== TMA producer.  Tiles are always whole: pages past the sequence are read from the null page (finite, masked)
      mbar_expect_tx(q_full, G * 2 * GH * 128);
      for (int a = 0; a < G; ++a)
        for (int kb = 0; kb < 2; ++kb) tma_load_3d(q_smem + a * Q_BYTES + kb * (NQ * 128), &tmap_q, kb * 64, a * GH, b, q_full);
      const int* bt = p.block_table + (int64_t)b * p.bt_stride;
      const int n_pages = (seq_len + BS - 1) / BS;
      int n = 0;
      auto slot = [&]() -> int {                 // the next slot of the ring, once its last reader is done
        const int s = n % SLOTS;
        mbar_wait_lim(&empty[s], ((n / SLOTS) & 1) ^ 1, budget);
        ++n;
        return s;
      };
      int blk[2] = {0, 0}, prev[2] = {0, 0};
      for (int j = 0; j <= n_tiles && budget >= 0; ++j) {
        if (j < n_tiles) {
          for (int u = 0; u < 2; ++u) {
            const int page = (tile_lo + j) * 2 + u;
            blk[u] = page < n_pages ? bt[page] : 0;
          }
          for (int a = 0; a < G; ++a) {
            const int s = slot();
            if (budget < 0) break;
            mbar_expect_tx(&full[s], TILE_BYTES);
            for (int u = 0; u < 2; ++u)
              for (int kb = 0; kb < 2; ++kb)
                tma_load_2d_hint(ring + s * TILE_BYTES + kb * (TILE * 128) + u * (BS * 128), &tmap_k, kb * 64,
                                 (blk[u] * 2 * G + a) * BS, &full[s], L2_EVICT_FIRST);
          }
        }
        if (j > 0 && budget >= 0) {
          for (int c = 0; c < G; ++c) {
            const int s = slot();
            if (budget < 0) break;
            mbar_expect_tx(&full[s], TILE_BYTES);
            for (int u = 0; u < 2; ++u)
              tma_load_2d_hint(ring + s * TILE_BYTES + u * (D * 128), &tmap_v, 0, ((prev[u] * 2 + 1) * G + c) * D, &full[s], L2_EVICT_FIRST);
          }
        }
        prev[0] = blk[0]; prev[1] = blk[1];
      }
      if (budget < 0) {                          // let the copies in flight land before the block gives up its memory
        for (int s = 0; s < SLOTS; ++s)
          for (int i = 0; i < 4096 && !(mbar_try_wait(&full[s], 0) || mbar_try_wait(&full[s], 1)); ++i) {}
      }
    }
  } else if (warp == 1) {
    // ===== MMA issuer
    const uint32_t idesc_s = umma_idesc_f16(128, NQ, true), idesc_o = umma_idesc_f16(128, HP, true);
    const uint64_t d_r = umma_desc_sw128(ring), d_q = umma_desc_sw128(q_smem), d_p = umma_desc_sw128(p_smem);
    int n = 0;
    mbar_wait_lim(q_full, 0, budget);
    __syncwarp();
    for (int j = 0; j <= n_tiles; ++j) {
      if (j < n_tiles) {
        mbar_wait_lim(&s_empty[j & 1], ((j >> 1) & 1) ^ 1, budget);
        for (int a = 0; a < G; ++a, ++n) {
          const int s = n % SLOTS;
          mbar_wait_lim(&full[s], (n / SLOTS) & 1, budget);
          tc_fence_after();
          if (lane == 0) {
#pragma unroll
            for (int kb = 0; kb < 2; ++kb)
#pragma unroll
              for (int k = 0; k < 4; ++k)
                umma_f16(tmem_base + ((j & 1) * G + a) * NQ, d_r + (uint64_t)(((s * TILE_BYTES + kb * TILE * 128) >> 4) + k * 2),
                         d_q + (uint64_t)(((a * Q_BYTES + kb * NQ * 128) >> 4) + k * 2), idesc_s, (kb | k) != 0);
            umma_commit(&empty[s]);
            if (a == G - 1) umma_commit(&s_full[j & 1]);
          }
          __syncwarp();
        }
      }
      if (j > 0) {
        const int jj = j - 1, pb = jj & 1;
        mbar_wait_lim(&p_full[pb], (jj >> 1) & 1, budget);
        for (int c = 0; c < G; ++c, ++n) {
          const int s = n % SLOTS;
          mbar_wait_lim(&full[s], (n / SLOTS) & 1, budget);
          tc_fence_after();
          if (lane == 0) {
#pragma unroll
            for (int kb = 0; kb < 2; ++kb)
#pragma unroll
              for (int k = 0; k < 4; ++k)
                umma_f16(tmem_o + c * HP, d_r + (uint64_t)(((s * TILE_BYTES + kb * D * 128) >> 4) + k * 2),
                         d_p + (uint64_t)(((pb * P_BYTES + kb * HP * 128) >> 4) + k * 2), idesc_o, (jj | kb | k) != 0);
            umma_commit(&empty[s]);
            if (c == G - 1) umma_commit(&pv_done[pb]);
          }
          __syncwarp();
        }
      }
    }
  } else {
    // ===== softmax: thread = token of the tile; later thread = output dim
    const int qd = warp & 3, t = qd * 32 + lane;
    const uint32_t t_lane = (uint32_t)(qd * 32) << 16;
    float l[HP];
#pragma unroll
    for (int h = 0; h < HP; ++h) l[h] = 0.f;
    for (int j = 0; j < n_tiles; ++j) {
      const int sb = j & 1;
      mbar_wait_lim(&s_full[sb], (j >> 1) & 1, budget);
      __syncwarp();
      tc_fence_after();
      float s[HP];
#pragma unroll
      for (int h = 0; h < HP; ++h) s[h] = 0.f;
#pragma unroll
      for (int a = 0; a < GA; ++a) {
        if (a < G) {
          uint32_t v[16];
          tmem_ld_32x16(tmem_base + (sb * G + a) * NQ + t_lane, v);
          tmem_ld_wait();
#pragma unroll
          for (int g = 0; g < GH; ++g) s[a * GH + g] = __uint_as_float(v[g]);
        }
      }
      tc_fence_before();
      mbar_arrive(&s_empty[sb]);
      const int kpos = (tile_lo + j) * TILE + t;
      const bool ok = kpos < seq_len && kpos >= kv_begin;
      if (!ok) {
#pragma unroll
        for (int h = 0; h < HP; ++h) s[h] = 0.f;
      }
      talk::cap_exp<HP>(s, p.cap);
      if (j >= 2) { mbar_wait_lim(&pv_done[sb], ((j >> 1) & 1) ^ 1, budget); __syncwarp(); }     // this P buffer is free again
      unsigned char* pcol = p_smem + sb * P_BYTES + (t >> 6) * (HP * 128) + (t & 7) * 2;
      const int chunk = (t & 63) >> 3;
#pragma unroll
      for (int h = 0; h < HP; ++h) {
        const float e = ok ? s[h] : 0.f;
        l[h] += e;
        *reinterpret_cast<T*>(pcol + h * 128 + ((chunk ^ (h & 7)) << 4)) = from_f32<T>(e);
      }
      fence_proxy_async();
      mbar_arrive(&p_full[sb]);
    }
    // ---- epilogue
#pragma unroll
    for (int h = 0; h < HP; ++h) {
      const float x = warp_sum(l[h]);
      if (lane == 0) red[qd * HP + h] = x;
    }
    bar_sync_softmax();
    if (t < p.H) p.part_l[row0 + t] = red[t] + red[HP + t] + red[2 * HP + t] + red[3 * HP + t];
    mbar_wait_lim(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1, budget);
    __syncwarp();
    tc_fence_after();
    for (int c = 0; c < G; ++c) {
#pragma unroll
      for (int h0 = 0; h0 < HP; h0 += 16) {
        uint32_t v[16];
        tmem_ld_32x16(tmem_o + c * HP + h0 + t_lane, v);
        tmem_ld_wait();
#pragma unroll
        for (int g = 0; g < 16; ++g)
          if (h0 + g < p.H) p.part_o[((row0 + h0 + g) * G + c) * D + t] = __uint_as_float(v[g]);
      }
    }
    tc_fence_before();
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, cols);
  if (budget < 0 && p.error) *p.error = 1;
}

template <int GH, int HP>
static int launch(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const Params& p, cudaStream_t st) {
  const int smem = SLOTS * TILE_BYTES + 2 * HP * TILE * 2 + p.Hkv * Q_BYTES + 32 * 8 + 16 + 4 * HP * 4 + 1024;
  if (smem > 227 * 1024) return -6;
  auto k = talk_decode_kernel<GH, HP>;
  static bool a = false;
  if (!a) { cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024); a = true; }
  vb_launch(k, dim3(p.splits, p.B), dim3(NUM_THREADS), (size_t)smem, st, tq, tk, tv, p);
  return (int)cudaGetLastError();
}

}  // namespace talkdec

// q [B, H * 128] (stride free), kv_cache as in vb_talk_fold; part_o [splits, B, H, Hkv, 128] and part_l [splits, B, H] fp32: sums of
// e^score times value, and of e^score.  H <= 32, Hkv <= 8, H / Hkv in {1, 2, 4, 8, 16}; 0 < soft_cap <= 60.
EXPORT int vb_talk_decode(const void* q, const void* kv_cache, int64_t num_blocks, const int* block_table, const int* seq_lens,
                          float* part_o, float* part_l, int* error, int B, int H, int Hkv, int64_t q_stride, int bt_stride, int splits,
                          int window, float scale, float soft_cap, cudaStream_t st) {
  using namespace talkdec;
  if (B == 0) return 0;
  const int GH = H / Hkv;
  if (H % Hkv || H > 32 || Hkv > MAX_KV || splits < 1 || q_stride % 8) return -4;
  if (!(soft_cap > 0.f && soft_cap <= talk::MAX_CAP)) return -5;
  Params p;
  p.block_table = block_table; p.seq_lens = seq_lens; p.part_o = part_o; p.part_l = part_l; p.bt_stride = bt_stride; p.B = B; p.H = H;
  p.Hkv = Hkv; p.splits = splits; p.window = window; p.cap = talk::make_cap(scale, soft_cap); p.error = error;
  CUtensorMap tq, tk, tv;
  int rc;
  if ((rc = talk::map_queries(&tq, q, H, B, q_stride, GH, 1))) return rc;
  if ((rc = talk::map_pages(&tk, &tv, kv_cache, num_blocks, Hkv, BS, D))) return rc;
#define GO(N) return H <= 16 ? launch<N, 16>(tq, tk, tv, p, st) : launch<N, 32>(tq, tk, tv, p, st)
  switch (GH) {
    case 1: return H <= 16 ? launch<1, 16>(tq, tk, tv, p, st) : -4;
    case 2: return H <= 16 ? launch<2, 16>(tq, tk, tv, p, st) : -4;
    case 4: GO(4);
    case 8: GO(8);
    case 16: GO(16);
  }
#undef GO
  return -4;
}
