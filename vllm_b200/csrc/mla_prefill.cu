// Latent-attention prefill on tcgen05: causal multi-head attention of a step's prompt portions over keys and values that
// were expanded from the latent cache (K = W_uk c, V = W_uv c, two GEMMs over the portion's whole context).
//
// Expanding costs one GEMM per layer but a score then takes `dim` multiplications instead of the latent width, and a
// value row `vdim`: for prompts that is several times fewer FLOPs than attending in the latent space (mla_decode.cu),
// which in turn never writes K / V and so is the better form for a handful of query tokens.
//
//   Q [T, H, dim]  K [KV, h, dim]  V [KV, h, vdim]   plain row-major GEMM outputs — no pages, no transposed copy:
//   S = Q · K^T    both operands K-major (dims contiguous), 128 x 128 tile, dim in 64-wide k-blocks
//   O += P · V     V is read as an MN-major B operand: a 128-byte swizzle row holds 64 dims of ONE token
// dim and vdim are multiples of 8 up to 128; TMA zero-fills the tail of a 64-wide block, so odd widths cost nothing else.
// A rotated part of the score (up to 64 wide, one key part for all heads) is one more k-block: its queries are columns of the query
// heads, its keys columns of the gathered cache rows, so nothing is copied together.  With a window, the request's key rows start at
// the first one that its portion sees.
//
// CTA = (request, head, 128 query tokens), heaviest (latest) query tiles first.  Warp roles: 0 TMA producer, 1 MMA
// issuer + TMEM owner, 2..5 softmax / rescale / epilogue with one thread per query row (row max and sum are
// thread-local).  TMEM: S double-buffered (2 x 128 columns), O (64 NV columns).  QK of tile j+1 is issued before PV of j.
#include "common.cuh"

namespace mlap {

constexpr int TM = 128, TN = 128;           // query rows, keys per tile
constexpr int NUM_THREADS = 192;
constexpr int STAGES = 2;
constexpr int BLK = 128 * 128;              // one [128 rows x 64 values] block, 16 KB

struct Params {
  const int* q_start;      // [B] first row of the request's portion in q / out
  const int* q_len;        // [B] rows of the portion
  const int* seq_len;      // [B] keys of the request (the portion is its tail)
  const int* kv_start;     // [B] first key row of the request in K / V
  void* out;               // [T, H, vdim]
  int64_t out_st, out_sh;
  int h0;                  // first head of this launch in q / out (K and V hold the launch's heads only)
  int vdim;
  int window;              // > 0: a query sees its last `window` keys
  float scale_log2;
  int* error;
};

VB_DEVICE void tma_load_3d(void* dst, const void* tmap, int c0, int c1, int c2, uint64_t* bar) {
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
               ::"r"(smem_u32(dst)), "l"(tmap), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2) : "memory");
}
VB_DEVICE void tmem_st_32x32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
        "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
        "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31]) : "memory");
}
VB_DEVICE void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// MN-major SW128 operand: 128-byte rows of 64 N-values (dims) of one K-value (token), 8 tokens per 1024-byte atom (SBO),
// the next 64 dims one block further (LBO)
VB_DEVICE uint64_t desc_mn(const void* smem_tile) {
  const uint32_t addr = smem_u32(smem_tile);
  uint64_t d = 0;
  d |= (uint64_t)((addr & 0x3FFFF) >> 4);
  d |= (uint64_t)((BLK >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

// NN blocks of unrotated and NR of rotated dimensions; VS stages of values
template <typename T, int NN, int NR, int NV, int VS>
__global__ void __launch_bounds__(NUM_THREADS, 1)
mla_prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                   const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_qr,
                   const __grid_constant__ CUtensorMap tmap_kr, const Params p) {
  constexpr int NQ = NN + NR;
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* q_smem = smem;                             // NQ blocks
  unsigned char* p_smem = q_smem + NQ * BLK;                // 2 blocks: [128 rows x 128 keys]
  unsigned char* k_smem = p_smem + 2 * BLK;                 // STAGES x NQ blocks
  unsigned char* v_smem = k_smem + STAGES * NQ * BLK;       // VS x NV blocks
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_smem + VS * NV * BLK);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;                 // [STAGES]
  uint64_t* v_full = k_full + STAGES;          // [STAGES]
  uint64_t* k_empty = v_full + STAGES;         // [STAGES]
  uint64_t* v_empty = k_empty + STAGES;        // [STAGES]
  uint64_t* s_full = v_empty + STAGES;         // [2]
  uint64_t* s_empty = s_full + 2;              // [2]
  uint64_t* p_full = s_empty + 2;
  uint64_t* pv_done = p_full + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int budget = MBAR_BUDGET;                    // failed polls left (mbar_wait_lim)
  const int b = blockIdx.z, h = blockIdx.y;
  pdl_trigger();
  pdl_wait();
  const int q_len = p.q_len[b];
  const int qt = (int)gridDim.x - 1 - (int)blockIdx.x;
  const int tok0 = qt * TM;
  if (tok0 >= q_len) return;                                // uniform over the CTA
  const int n_tok = min(TM, q_len - tok0);
  const int q0 = p.q_start[b] + tok0;
  const int kv0 = p.kv_start[b];
  const int pos0 = p.seq_len[b] - q_len + tok0;             // position of the tile's first query
  const int kv_end = pos0 + n_tok;                          // keys any query of the tile can see
  const int tile_lo = p.window > 0 ? max(0, pos0 - p.window + 1) / TN : 0;
  const int n_tiles = (kv_end + TN - 1) / TN - tile_lo;

  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tmap_q); tma_prefetch_desc(&tmap_k); tma_prefetch_desc(&tmap_v);
    mbar_init(q_full, 1);
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&k_full[s], 1); mbar_init(&v_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&s_empty[s], 128); }
    mbar_init(p_full, 128);
    mbar_init(pv_done, 1);
    mbar_fence_init();
  }
  if (warp == 1) tmem_alloc(tmem_slot, 512);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_o = tmem_base + 256;

  if (warp == 0) {
    if (lane == 0) {
      // ===== TMA producer.  Boxes are always whole: rows past the buffer read as zeros, rows of the next request are
      // masked by the softmax (finite values times a weight of 0).
      mbar_expect_tx(q_full, NQ * BLK);
#pragma unroll
      for (int i = 0; i < NN; ++i) tma_load_3d(q_smem + i * BLK, &tmap_q, i * 64, p.h0 + h, q0, q_full);
      if (NR) tma_load_3d(q_smem + NN * BLK, &tmap_qr, 0, p.h0 + h, q0, q_full);
      for (int j = 0; j < n_tiles; ++j) {
        const int s = j % STAGES, vs = j % VS;
        const uint32_t par = ((j / STAGES) & 1) ^ 1, v_par = ((j / VS) & 1) ^ 1;
        const int row = kv0 + (tile_lo + j) * TN;
        mbar_wait_lim(&k_empty[s], par, budget);
        if (budget < 0) break;
        mbar_expect_tx(&k_full[s], NQ * BLK);
#pragma unroll
        for (int i = 0; i < NN; ++i) tma_load_3d(k_smem + (s * NQ + i) * BLK, &tmap_k, i * 64, h, row, &k_full[s]);
        if (NR) tma_load_3d(k_smem + (s * NQ + NN) * BLK, &tmap_kr, 0, 0, row, &k_full[s]);
        mbar_wait_lim(&v_empty[vs], v_par, budget);
        if (budget < 0) break;
        mbar_expect_tx(&v_full[vs], NV * BLK);
#pragma unroll
        for (int i = 0; i < NV; ++i) tma_load_3d(v_smem + (vs * NV + i) * BLK, &tmap_v, i * 64, h, row, &v_full[vs]);
      }
      if (budget < 0) {                         // let the copies in flight land before the block gives up its memory
        for (int s = 0; s < STAGES; ++s)
          for (int n = 0; n < 4096 && !(mbar_try_wait(&k_full[s], 0) || mbar_try_wait(&k_full[s], 1)); ++n) {}
        for (int s = 0; s < VS; ++s)
          for (int n = 0; n < 4096 && !(mbar_try_wait(&v_full[s], 0) || mbar_try_wait(&v_full[s], 1)); ++n) {}
      }
    }
  } else if (warp == 1) {
    // ===== MMA issuer
    const bool bf16 = DTypeOf<T>::v == DT_BF16;
    const uint32_t idesc_s = umma_idesc_f16(TM, TN, bf16);
    const uint32_t idesc_o = umma_idesc_f16(TM, NV * 64, bf16) | (1u << 16);      // bit 16: B operand is MN-major
    const uint64_t d_q = umma_desc_sw128(q_smem), d_k = umma_desc_sw128(k_smem), d_p = umma_desc_sw128(p_smem);
    const uint64_t d_v = desc_mn(v_smem);
    mbar_wait_lim(q_full, 0, budget);
    __syncwarp();
    for (int j = 0; j <= n_tiles; ++j) {
      if (j < n_tiles) {
        const int s = j % STAGES, sb = j & 1;
        mbar_wait_lim(&k_full[s], (j / STAGES) & 1, budget);
        mbar_wait_lim(&s_empty[sb], ((j >> 1) & 1) ^ 1, budget);
        tc_fence_after();
        if (lane == 0) {
#pragma unroll
          for (int kb = 0; kb < NQ; ++kb) {
            const uint64_t da = d_q + (uint64_t)((kb * BLK) >> 4), db = d_k + (uint64_t)(((s * NQ + kb) * BLK) >> 4);
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma_f16(tmem_base + sb * 128, da + (uint64_t)(k * 2), db + (uint64_t)(k * 2), idesc_s, (kb | k) != 0);
          }
          umma_commit(&s_full[sb]);
          umma_commit(&k_empty[s]);
        }
        __syncwarp();
      }
      if (j > 0) {
        const int jj = j - 1, s = jj % VS;
        mbar_wait_lim(&v_full[s], (jj / VS) & 1, budget);
        mbar_wait_lim(p_full, jj & 1, budget);
        tc_fence_after();
        if (lane == 0) {
#pragma unroll
          for (int kk = 0; kk < TN / 16; ++kk) {                // 16 keys per MMA: 16 rows of 128 bytes of V
            const uint64_t da = d_p + (uint64_t)(((kk / 4) * BLK) >> 4) + (uint64_t)((kk & 3) * 2);
            const uint64_t db = d_v + (uint64_t)((s * NV * BLK + kk * 2048) >> 4);
            umma_f16(tmem_o, da, db, idesc_o, (jj | kk) != 0);
          }
          umma_commit(&v_empty[s]);
          umma_commit(pv_done);
        }
        __syncwarp();
      }
    }
  } else {
    // ===== softmax / rescale / epilogue: thread = query row = TMEM lane
    const int qd = warp & 3;
    const int r = qd * 32 + lane;
    const uint32_t t_lane = (uint32_t)(qd * 32) << 16;
    const bool row_valid = r < n_tok;
    float m_used = -INFINITY, l_run = 0.f;
    for (int j = 0; j < n_tiles; ++j) {
      const int sb = j & 1;
      const uint32_t t_s = tmem_base + sb * 128 + t_lane;
      mbar_wait_lim(&s_full[sb], (j >> 1) & 1, budget);
      __syncwarp();
      tc_fence_after();
      const int hi = row_valid ? pos0 + r + 1 - (tile_lo + j) * TN : 0;     // keys [lo, hi) of this tile are visible to the row
      const int lo = p.window > 0 ? hi - p.window : 0;
      const bool full = __all_sync(0xffffffffu, hi >= TN && lo <= 0) != 0;  // tiles inside every row's range: no masks
      // ---- pass 1: row max
      float mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < TN; c += 32) {
        uint32_t v[32];
        tmem_ld_32x32(t_s + c, v);
        tmem_ld_wait();
        if (full) {
#pragma unroll
          for (int i = 0; i < 32; ++i) mx = fmaxf(mx, __uint_as_float(v[i]) * p.scale_log2);
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c + i < hi && c + i >= lo) mx = fmaxf(mx, __uint_as_float(v[i]) * p.scale_log2);
        }
      }
      // keep the old reference maximum unless the new one is more than 2^8 above it
      float alpha = 1.f;
      bool rescale = false;
      if (mx > m_used + 8.f || (m_used == -INFINITY && mx > -INFINITY)) {
        rescale = m_used != -INFINITY;
        if (rescale) alpha = ex2(m_used - mx);
        m_used = mx;
      }
      const float m_ref = m_used == -INFINITY ? 0.f : m_used;
      if (j > 0) { mbar_wait_lim(pv_done, (j - 1) & 1, budget); __syncwarp(); tc_fence_after(); }   // P and O are free
      if (__any_sync(0xffffffffu, rescale)) {
        l_run *= alpha;
#pragma unroll
        for (int c = 0; c < NV * 64; c += 32) {
          uint32_t v[32];
          tmem_ld_32x32(tmem_o + t_lane + c, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
          tmem_st_32x32(tmem_o + t_lane + c, v);
        }
        tmem_st_wait();
      }
      // ---- pass 2: P = 2^(s - m), row sum, 16-bit copy in the swizzled K-major layout
#pragma unroll
      for (int c = 0; c < TN; c += 32) {
        uint32_t v[32];
        tmem_ld_32x32(t_s + c, v);
        tmem_ld_wait();
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float p0 = ex2(__uint_as_float(v[i]) * p.scale_log2 - m_ref), p1 = ex2(__uint_as_float(v[i + 1]) * p.scale_log2 - m_ref);
          if (!full) {
            if (c + i >= hi || c + i < lo) p0 = 0.f;
            if (c + i + 1 >= hi || c + i + 1 < lo) p1 = 0.f;
          }
          l_run += p0 + p1;
          pk[i / 2] = pack2<T>(p0, p1);
        }
        unsigned char* prow = p_smem + (c / 64) * BLK + r * 128;
#pragma unroll
        for (int ch = 0; ch < 4; ++ch) {
          const int chunk = ((c % 64) / 8 + ch) ^ (r & 7);
          *reinterpret_cast<uint4*>(prow + chunk * 16) = make_uint4(pk[ch * 4], pk[ch * 4 + 1], pk[ch * 4 + 2], pk[ch * 4 + 3]);
        }
      }
      tc_fence_before();
      fence_proxy_async();
      mbar_arrive(&s_empty[sb]);
      mbar_arrive(p_full);
    }
    // ---- epilogue
    mbar_wait_lim(pv_done, (n_tiles - 1) & 1, budget);
    __syncwarp();
    tc_fence_after();
    const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
    T* orow = reinterpret_cast<T*>(p.out) + (int64_t)(q0 + r) * p.out_st + (int64_t)(p.h0 + h) * p.out_sh;
#pragma unroll
    for (int c = 0; c < NV * 64; c += 32) {
      uint32_t v[32];
      tmem_ld_32x32(tmem_o + t_lane + c, v);
      tmem_ld_wait();
      if (row_valid) {
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          if (c + i >= p.vdim) break;
          uint4 o;
          o.x = pack2<T>(__uint_as_float(v[i]) * inv, __uint_as_float(v[i + 1]) * inv);
          o.y = pack2<T>(__uint_as_float(v[i + 2]) * inv, __uint_as_float(v[i + 3]) * inv);
          o.z = pack2<T>(__uint_as_float(v[i + 4]) * inv, __uint_as_float(v[i + 5]) * inv);
          o.w = pack2<T>(__uint_as_float(v[i + 6]) * inv, __uint_as_float(v[i + 7]) * inv);
          *reinterpret_cast<uint4*>(orow + c + i) = o;
        }
      }
    }
    tc_fence_before();
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 512);
  if (budget < 0 && p.error) *p.error = 1;
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static EncodeTiledFn get_encode() {
  static EncodeTiledFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess || !ptr) return nullptr;
    fn = reinterpret_cast<EncodeTiledFn>(ptr);
  }
  return fn;
}

// [rows, heads, width] with row stride `rs` and head stride `hs` elements; box = 128 rows of 64 values of one head
static int tmap(CUtensorMap* m, const void* ptr, int width, int heads, int64_t rows, int64_t rs, int64_t hs, bool bf16) {
  auto enc = get_encode();
  if (!enc) return -10;
  cuuint64_t dims[3] = {(cuuint64_t)width, (cuuint64_t)heads, (cuuint64_t)rows};
  cuuint64_t strides[2] = {(cuuint64_t)hs * 2, (cuuint64_t)rs * 2};
  cuuint32_t box[3] = {64, 1, 128};
  cuuint32_t es[3] = {1, 1, 1};
  return enc(m, bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 3, const_cast<void*>(ptr), dims,
             strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -11;
}

struct Maps { CUtensorMap q, k, v, qr, kr; };

template <typename T, int NN, int NR, int NV>
static int launch(const Maps& m, const Params& p, dim3 grid, cudaStream_t st) {
  constexpr int NQ = NN + NR;
  constexpr int VS = NQ + 2 + STAGES * (NQ + NV) <= 13 ? STAGES : 1;         // what fits into shared memory
  const int smem = (NQ + 2 + STAGES * NQ + VS * NV) * BLK + 32 * 8 + 16 + 1024;
  auto k = mla_prefill_kernel<T, NN, NR, NV, VS>;
  static bool a = false;
  if (!a) { cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem); a = true; }
  vb_launch(k, grid, dim3(NUM_THREADS), (size_t)smem, st, m.q, m.k, m.v, m.qr, m.kr, p);
  return (int)cudaGetLastError();
}

}  // namespace mlap

// q [T, H, dim + rot] and out [T, H, vdim] (row strides q_st / out_st); k [KV, hl, dim], v [KV, hl, vdim] hold the heads
// h0 .. h0 + hl - 1; k_pe [KV, rot] (row stride kr_st; rot = 0: none) is the rotated key part of all heads.  Request b owns query rows
// q_start[b] .. + q_len[b] and key rows kv_start[b] .. + seq_len[b], of which its portion is the tail.
EXPORT int vb_mla_prefill(const void* q, const void* k, const void* v, const void* k_pe, void* out, const int* q_start, const int* q_len,
                          const int* seq_len, const int* kv_start, int* error, int B, int T_, int64_t KV, int H, int h0, int hl,
                          int dim, int rot, int vdim, int64_t q_st, int64_t k_st, int64_t v_st, int64_t kr_st, int64_t out_st, int max_q,
                          int window, float scale, int dtype, cudaStream_t st) {
  using namespace mlap;
  if (B == 0 || T_ == 0 || max_q <= 0) return 0;
  if (dtype == DT_F32 || dim < 8 || dim > 128 || dim % 8 || vdim < 8 || vdim > 128 || vdim % 8 || rot < 0 || rot > 64 || rot % 8) return -1;
  if (q_st % 8 || k_st % 8 || v_st % 8 || out_st % 8 || h0 < 0 || h0 + hl > H || (rot && (!k_pe || kr_st % 8))) return -2;
  const bool bf16 = dtype == DT_BF16;
  Maps m;
  int rc;
  if ((rc = tmap(&m.q, q, dim, H, T_, q_st, dim + rot, bf16))) return rc;
  if ((rc = tmap(&m.k, k, dim, hl, KV, k_st, dim, bf16))) return rc;
  if ((rc = tmap(&m.v, v, vdim, hl, KV, v_st, vdim, bf16))) return rc;
  m.qr = m.q; m.kr = m.k;
  if (rot) {
    if ((rc = tmap(&m.qr, reinterpret_cast<const char*>(q) + (int64_t)dim * 2, rot, H, T_, q_st, dim + rot, bf16))) return rc;
    if ((rc = tmap(&m.kr, k_pe, rot, 1, KV, kr_st, kr_st, bf16))) return rc;
  }
  Params p;
  p.q_start = q_start; p.q_len = q_len; p.seq_len = seq_len; p.kv_start = kv_start; p.out = out; p.out_st = out_st;
  p.out_sh = vdim; p.h0 = h0; p.vdim = vdim; p.window = window; p.scale_log2 = scale * 1.4426950408889634f; p.error = error;
  const dim3 grid((max_q + TM - 1) / TM, hl, B);
  const int nq = (dim + 63) / 64, nv = (vdim + 63) / 64;
#define GV(TT, N, R) (nv == 1 ? launch<TT, N, R, 1>(m, p, grid, st) : launch<TT, N, R, 2>(m, p, grid, st))
#define GO(TT) (rot ? (nq == 1 ? GV(TT, 1, 1) : GV(TT, 2, 1)) : (nq == 1 ? GV(TT, 1, 0) : GV(TT, 2, 0)))
  return bf16 ? GO(__nv_bfloat16) : GO(__half);
#undef GO
#undef GV
}
