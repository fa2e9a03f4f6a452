// What the attention kernels with mixed heads share (attention_talk.cu, attention_talk_decode.cu): exponentials of capped scores and the
// tensor maps of queries and of pages in the tensor-core layout (head size 128, 64 tokens per page, values transposed).
#pragma once
#include "common.cuh"

namespace talk {

constexpr float MAX_CAP = 60.f;

// e^(cap tanh(s scale / cap)) of a raw score s, in powers of two: 2^(c2 tanh(s ku)), c2 = cap log2(e), ku = scale / cap
struct Cap {
  float c2, e2, ku, k0, k1, k2, k3;             // e2: s -> the exponent of e^(2 s ku); k0..k3: series of c2 tanh(s ku) in s
};
inline Cap make_cap(float scale, float cap) {
  const double l2e = 1.4426950408889634, c2 = cap * l2e, ku = (double)scale / cap;
  Cap c;
  c.c2 = (float)c2; c.ku = (float)(ku < 0 ? -ku : ku); c.e2 = (float)(2 * ku * l2e);
  c.k0 = (float)(c2 * ku); c.k1 = (float)(-c2 * ku * ku * ku / 3);
  c.k2 = (float)(c2 * ku * ku * ku * ku * ku * 2 / 15); c.k3 = (float)(-c2 * ku * ku * ku * ku * ku * ku * ku * 17 / 315);
  return c;
}
VB_DEVICE float rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// pairs of floats: one instruction per pair
VB_DEVICE uint64_t pair2(float a, float b) { uint64_t r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b)); return r; }
VB_DEVICE float2 split2(uint64_t v) { float2 r; asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v)); return r; }
VB_DEVICE uint64_t add2(uint64_t a, uint64_t b) { uint64_t r; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
VB_DEVICE uint64_t mul2(uint64_t a, uint64_t b) { uint64_t r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
VB_DEVICE uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r;
}

VB_DEVICE float max3(float a, float b, float c) { float r; asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c)); return r; }

// In place, for N scores of a thread; the whole warp takes part.  Where all scores of the warp are below a quarter of the cap the Taylor
// series of tanh to the seventh power is exact to 3e-7 and needs no more special functions than a plain softmax.
template <int N> VB_DEVICE void cap_exp(float (&s)[N], const Cap& c) {
  uint64_t x[N / 2], q[N / 2];
  float m4[4] = {0.f, 0.f, 0.f, 0.f};                      // (squares: no signs)
#pragma unroll
  for (int i = 0; i < N / 2; ++i) {
    x[i] = pair2(s[2 * i], s[2 * i + 1]);
    q[i] = mul2(x[i], x[i]);
    const float2 f = split2(q[i]);
    m4[i & 3] = max3(m4[i & 3], f.x, f.y);
  }
  const float m = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
  if (__all_sync(0xffffffffu, m * c.ku * c.ku < 0.0625f)) {
    const uint64_t k0 = pair2(c.k0, c.k0), k1 = pair2(c.k1, c.k1), k2 = pair2(c.k2, c.k2), k3 = pair2(c.k3, c.k3);
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
      const float2 f = split2(mul2(x[i], fma2(q[i], fma2(q[i], fma2(q[i], k3, k2), k1), k0)));
      s[2 * i] = ex2(f.x);
      s[2 * i + 1] = ex2(f.y);
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) s[i] = ex2(c.c2 - 2.f * c.c2 * rcp(1.f + ex2(s[i] * c.e2)));
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
inline EncodeTiledFn get_encode() {
  static EncodeTiledFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess || !ptr) return nullptr;
    fn = reinterpret_cast<EncodeTiledFn>(ptr);
  }
  return fn;
}
inline int encode(CUtensorMap* m, const void* ptr, int rank, const cuuint64_t* dims, const cuuint64_t* strides, const cuuint32_t* box) {
  auto enc = get_encode();
  if (!enc) return -10;
  const cuuint32_t es[3] = {1, 1, 1};
  return enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(ptr), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -11;
}
// q [T, Hq, 128] with a token stride; box = 64 dims x G heads x TQ tokens
inline int map_queries(CUtensorMap* m, const void* q, int Hq, int T, int64_t stride, int G, int TQ) {
  const cuuint64_t dims[3] = {128, (cuuint64_t)Hq, (cuuint64_t)T}, strides[2] = {256, (cuuint64_t)stride * 2};
  const cuuint32_t box[3] = {64, (cuuint32_t)G, (cuuint32_t)TQ};
  return encode(m, q, 3, dims, strides, box);
}
// key pages as rows of 128 dims (box 64 x k_rows tokens), value pages as rows of 64 tokens (box 64 x v_rows dims)
inline int map_pages(CUtensorMap* k, CUtensorMap* v, const void* cache, int64_t blocks, int Hkv, int k_rows, int v_rows) {
  const cuuint64_t kd[2] = {128, (cuuint64_t)blocks * 2 * Hkv * 64}, ks[1] = {256};
  const cuuint64_t vd[2] = {64, (cuuint64_t)blocks * 2 * Hkv * 128}, vs[1] = {128};
  const cuuint32_t kb[2] = {64, (cuuint32_t)k_rows}, vb[2] = {64, (cuuint32_t)v_rows};
  int rc = encode(k, cache, 2, kd, ks, kb);
  return rc ? rc : encode(v, cache, 2, vd, vs, vb);
}

}  // namespace talk
