// Latent attention: a position leaves one low-rank vector (the latent, RMS-normed) and one rotated key part that all heads
// share; a head's unrotated key and its value are W_uk c and W_uv c. The cache row of a position is [latent | rotated part],
// each padded with zeros to a multiple of 16 elements, whatever the number of heads.
//
//  * prompts: keys and values are rebuilt per head by one GEMM over the visible latents, then the tcgen05 prefill kernel
//    runs on them (attention_tc.cu). Here: the projection's rows into rotated queries and cache rows.
//  * decode: nothing is rebuilt. A head's query is carried into latent space (q' = q W_uk), so that q' . c replaces
//    q . W_uk c, all heads read the same cache row (the heads are the columns of the MMA tile) and the weighted sum of latents
//    goes through W_uv once per head. Three launches: queries into latent space beside everything else the projection
//    feeds (rotation, cache append, activation); split-key attention, merged inside a cluster; W_uv.
//  * any other width, and fp32: one block per row and head, straight from the cache.
//
// Scores, softmax weights, norms and rotations are fp32; the weights enter the product with the latents as two bf16 terms
// (hi + lo), whose sum carries 16 mantissa bits.
#include <cuda.h>

#include <algorithm>
#include <mutex>

#include "common.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t s, const void* g, bool valid) {
  int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(g), "r"(sz));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x2(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void mbar_init(uint32_t bar, uint32_t count) { asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count)); }
__device__ __forceinline__ void mbar_expect_tx(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
// Bounded wait for the phase with the given parity. Returns false when the limit expired.
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity) {
  for (uint32_t i = 0; i < (1u << 22); i++) {
    uint32_t done;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(done)
        : "r"(bar), "r"(parity)
        : "memory");
    if (done) return true;
  }
  return false;
}
// by one elected lane of a warp that runs converged
__device__ __forceinline__ void tma_load_2d_warp(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar, uint64_t policy) {
  asm volatile(
      "{\n\t.reg .pred e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "@e cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint [%0], [%1, {%2, %3}], [%4], %5;\n\t}" ::"r"(dst),
      "l"(map), "r"(x), "r"(y), "r"(bar), "l"(policy)
      : "memory");
}
__device__ __forceinline__ void mbar_expect_tx_warp(uint32_t bar, uint32_t bytes) {
  asm volatile(
      "{\n\t.reg .pred e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "@e mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;\n\t}" ::"r"(bar),
      "r"(bytes)
      : "memory");
}
// the address of this block's shared-memory location in block `rank` of the cluster
__device__ __forceinline__ uint32_t map_to_rank(uint32_t local, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(local), "r"(rank));
  return r;
}
__device__ __forceinline__ float2 ld_cluster2(uint32_t addr) {
  float2 v;
  asm volatile("ld.shared::cluster.v2.f32 {%0,%1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// not volatile: the compiler may move fragment loads ahead of products that do not need them
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two fp32 values as two bf16 terms, p = hi + lo to 2^-17
__device__ __forceinline__ void split_bf16x2(float p0, float p1, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(p0 - __uint_as_float(hi << 16), p1 - __uint_as_float(hi & 0xFFFF0000u));
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) { return f32_to_bf16_bits(lo) | (f32_to_bf16_bits(hi) << 16); }
__device__ __forceinline__ int ld_volatile_i32(const int32_t* p) {
  int v;
  asm volatile("ld.volatile.global.s32 %0, [%1];" : "=r"(v) : "l"(p) : "memory");
  return v;
}
template <typename T>
__device__ __forceinline__ T to_t(float v);
template <>
__device__ __forceinline__ float to_t<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 to_t<bf16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }

// ------------------------------------------------------------------ projection rows -> queries and cache rows
struct SplitDev {
  int H, dim, rot, rank, rank_p, row, q_head, q_rot;
  const float* in;
  int64_t ld_in;
  int splits;
  const int32_t *seq, *pos, *lens;
  const float *cos_t, *sin_t;
  int max_pos, maxlen;
  const float* norm_w;
  float eps;
  void* q_out;
  void* cache;
};
__device__ __forceinline__ float proj(const SplitDev& a, int64_t T, int64_t t, int64_t col) {
  float v = 0.f;
  for (int s = 0; s < a.splits; s++) v += a.in[((int64_t)s * T + t) * a.ld_in + col];
  return v;
}
// four columns at a time (col and the row stride multiples of 4; at most 8 splits), every split's load in flight at once
__device__ __forceinline__ float4 proj4(const SplitDev& a, int64_t T, int64_t t, int64_t col) {
  if (a.splits == 1) return *(const float4*)(a.in + t * a.ld_in + col);
  float4 p[8], v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int s = 0; s < 8; s++)
    if (s < a.splits) p[s] = *(const float4*)(a.in + ((int64_t)s * T + t) * a.ld_in + col);
#pragma unroll
  for (int s = 0; s < 8; s++)
    if (s < a.splits) { v.x += p[s].x; v.y += p[s].y; v.z += p[s].z; v.w += p[s].w; }
  return v;
}
// pair i of a rotated vector (dimension 2i with 2i + 1)
__device__ __forceinline__ void rotate(const SplitDev& a, int p, int i, float& u, float& v) {
  const float c = a.cos_t[(int64_t)p * (a.rot / 2) + i], s = a.sin_t[(int64_t)p * (a.rot / 2) + i];
  const float x = u, y = v;
  u = __fsub_rn(__fmul_rn(x, c), __fmul_rn(y, s));
  v = __fadd_rn(__fmul_rn(y, c), __fmul_rn(x, s));
}
// Latent and rotated key part of row t, columns n_q.. of the projection, into the cache row of position p. Whole block.
template <typename T>
__device__ __forceinline__ void append_latent(const SplitDev& a, int64_t rows, int64_t t, int b, int p, float* red) {
  const int64_t c0 = (int64_t)a.H * (a.dim + a.rot);
  T* dst = (T*)a.cache + ((int64_t)b * a.maxlen + p) * a.row;
  // the rotated part is requested first, by threads from the end of the block, so that its loads run beside the latent's
  const int ri = (int)blockDim.x - 1 - (int)threadIdx.x;
  float u = 0.f, v = 0.f;
  if (ri < a.rot / 2) { u = proj(a, rows, t, c0 + a.rank + 2 * ri); v = proj(a, rows, t, c0 + a.rank + 2 * ri + 1); }
  float x[4], ss = 0.f;  // the first 4 * blockDim columns stay in registers
#pragma unroll
  for (int j = 0; j < 4; j++) {
    const int i = j * (int)blockDim.x + (int)threadIdx.x;
    x[j] = i < a.rank ? proj(a, rows, t, c0 + i) : 0.f;
  }
#pragma unroll
  for (int j = 0; j < 4; j++) ss += x[j] * x[j];
  for (int i = 4 * (int)blockDim.x + (int)threadIdx.x; i < a.rank; i += blockDim.x) {
    const float w = proj(a, rows, t, c0 + i);
    ss += w * w;
  }
  ss = block_sum(ss, red);
  const float r = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)a.rank), a.eps)));
#pragma unroll
  for (int j = 0; j < 4; j++) {
    const int i = j * (int)blockDim.x + (int)threadIdx.x;
    if (i < a.rank) dst[i] = to_t<T>(x[j] * r * a.norm_w[i]);
  }
  for (int i = 4 * (int)blockDim.x + (int)threadIdx.x; i < a.rank; i += blockDim.x) dst[i] = to_t<T>(proj(a, rows, t, c0 + i) * r * a.norm_w[i]);
  if (ri < a.rot / 2) {
    rotate(a, p, ri, u, v);
    dst[a.rank_p + 2 * ri] = to_t<T>(u);
    dst[a.rank_p + 2 * ri + 1] = to_t<T>(v);
  }
  for (int i = (int)blockDim.x + ri; i < a.rot / 2; i += blockDim.x) {
    u = proj(a, rows, t, c0 + a.rank + 2 * i);
    v = proj(a, rows, t, c0 + a.rank + 2 * i + 1);
    rotate(a, p, i, u, v);
    dst[a.rank_p + 2 * i] = to_t<T>(u);
    dst[a.rank_p + 2 * i + 1] = to_t<T>(v);
  }
}

// grid (T, 2 with latents of its own, else 1)
template <typename T>
__global__ void __launch_bounds__(256) latent_split_kernel(SplitDev a, int64_t rows) {
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const int b = a.seq ? a.seq[t] : (int)t, p = a.pos ? a.pos[t] : a.lens[b];
  if (p < 0 || p >= a.maxlen || p >= a.max_pos) return;  // host validates; never index outside the cache
  if (blockIdx.y == 1) {  // the latent's half of the row
    append_latent<T>(a, rows, t, b, p, red);
    return;
  }
  T* q = (T*)a.q_out + t * a.H * a.q_head;
  if (((a.dim | a.rot) & 3) == 0 && a.splits == 1 && a.ld_in % 4 == 0) {
    // four columns at a time, four requests in flight per thread
    const int quarter = (a.dim + a.rot) / 4, n = a.H * quarter;
    const float4* in = (const float4*)(a.in + t * a.ld_in);
    for (int i0 = threadIdx.x; i0 < n; i0 += 4 * (int)blockDim.x) {
      float4 w[4];
#pragma unroll
      for (int u = 0; u < 4; u++)
        if (i0 + u * (int)blockDim.x < n) w[u] = __ldcs(in + i0 + u * (int)blockDim.x);
#pragma unroll
      for (int u = 0; u < 4; u++) {
        const int i = i0 + u * (int)blockDim.x;
        if (i < n) {
          const int h = i / quarter, j = (i - h * quarter) * 4;
          if (j >= a.dim) {
            rotate(a, p, (j - a.dim) / 2, w[u].x, w[u].y);
            rotate(a, p, (j - a.dim) / 2 + 1, w[u].z, w[u].w);
          }
          T* dst = q + h * a.q_head + (j < a.dim ? j : a.q_rot + j - a.dim);
          if (sizeof(T) == 2) *(uint2*)dst = make_uint2(pack_bf16(w[u].x, w[u].y), pack_bf16(w[u].z, w[u].w));
          else *(float4*)dst = w[u];
        }
      }
    }
  } else {
    for (int i = threadIdx.x; i < a.H * a.dim; i += blockDim.x) {
      const int h = i / a.dim, j = i - h * a.dim;
      q[h * a.q_head + j] = to_t<T>(proj(a, rows, t, (int64_t)h * (a.dim + a.rot) + j));
    }
    for (int i = threadIdx.x; i < a.H * (a.rot / 2); i += blockDim.x) {
      const int h = i / (a.rot / 2), j = i - h * (a.rot / 2);
      const int64_t col = (int64_t)h * (a.dim + a.rot) + a.dim + 2 * j;
      float u = proj(a, rows, t, col), v = proj(a, rows, t, col + 1);
      rotate(a, p, j, u, v);
      q[h * a.q_head + a.q_rot + 2 * j] = to_t<T>(u);
      q[h * a.q_head + a.q_rot + 2 * j + 1] = to_t<T>(v);
    }
  }
}

__global__ void __launch_bounds__(128) latent_gather_kernel(const bf16* __restrict__ cache, int64_t maxlen, int row, const int32_t* __restrict__ koff,
                                                            const int32_t* __restrict__ kpos0, const int32_t* __restrict__ lens, bf16* __restrict__ dst) {
  const int j = blockIdx.y;
  const int n = lens[j] - kpos0[j], vec = row / 8;
  const uint4* src = (const uint4*)(cache + ((int64_t)j * maxlen + kpos0[j]) * row);
  uint4* d = (uint4*)(dst + (int64_t)koff[j] * row);
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < (int64_t)n * vec; i += (int64_t)gridDim.x * blockDim.x) d[i] = src[i];
}

// ------------------------------------------------------------------ decode: queries into latent space, cache append, activation
struct DecodeInDev {
  SplitDev a;
  const bf16* wkv;
  int kv_head;
  bf16* q_abs;
  int act_col, n_act;
  float act_pos, act_neg;
  bf16* act;
  int64_t ld_act;
  int n_rt, n_grp;      // latent tiles of 128 and token groups of 16: blocks of the first role
  int rot_blocks;       // blocks per token of the rotation (256 pairs each)
  int act_blocks;       // ... and of the activation
};
constexpr int QA_COLS = 128, QA_LD = QA_COLS + 8;
__host__ __device__ inline int decode_in_smem(int dim) {
  const int d16 = (dim + 15) & ~15;
  return d16 * QA_LD * 2 + 16 * (d16 + 8) * 2;
}
// One launch, four roles by block index: H * n_rt * n_grp blocks multiply queries with W_uk (128 latents of one head,
// 16 tokens), then B * rot_blocks rotate the queries' second part, B append the cache row (a layer with latents of its own),
// B * act_blocks run the activation.
__global__ void __launch_bounds__(256) latent_decode_in_kernel(DecodeInDev d, int B) {
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float red[32];
  SB_TRACE_BEGIN();
  pdl_trigger();
  const SplitDev& a = d.a;
  int blk = blockIdx.x;
  const int n_mul = a.H * d.n_rt * d.n_grp;
  if (blk < n_mul) {
    const int grp = blk % d.n_grp, rt = blk / d.n_grp % d.n_rt, h = blk / d.n_grp / d.n_rt;
    const int r0 = rt * QA_COLS, b0 = grp * 16, d16 = (a.dim + 15) & ~15;
    bf16* wt = (bf16*)smem;           // [d16][QA_LD]
    bf16* qt = wt + d16 * QA_LD;      // [16][d16 + 8]
    for (int c = threadIdx.x; c < d16 * (QA_COLS / 8); c += blockDim.x) {
      const int dd = c / (QA_COLS / 8), cc = c % (QA_COLS / 8);
      const bool ok = dd < a.dim && r0 + cc * 8 < a.rank_p;
      cp_async16(smem_u32(wt + dd * QA_LD + cc * 8), ok ? d.wkv + (int64_t)(h * d.kv_head + dd) * a.rank_p + r0 + cc * 8 : d.wkv, ok);
    }
    cp_async_commit();
    pdl_wait();
    SB_TRACE_WAITED();
    if (((a.dim | a.rot) & 3) == 0 && a.ld_in % 4 == 0) {
      for (int i = threadIdx.x; i < 4 * d16; i += blockDim.x) {
        const int m = i / (d16 / 4), k = (i - m * (d16 / 4)) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (b0 + m < B && k < a.dim) v = proj4(a, B, b0 + m, (int64_t)h * (a.dim + a.rot) + k);
        *(uint2*)(qt + m * (d16 + 8) + k) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
      }
    } else for (int i = threadIdx.x; i < 16 * d16; i += blockDim.x) {
      const int m = i / d16, k = i - m * d16;
      qt[m * (d16 + 8) + k] = b0 + m < B && k < a.dim ? __float2bfloat16_rn(proj(a, B, b0 + m, (int64_t)h * (a.dim + a.rot) + k)) : __float2bfloat16_rn(0.f);
    }
    cp_async_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3, r8 = lane & 7;
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    for (int k = 0; k < d16; k += 16) {
      uint32_t qa[4], wb[4];
      ldsm_x4(smem_u32(qt + ((mi & 1) * 8 + r8) * (d16 + 8) + k + (mi >> 1) * 8), qa);
      ldsm_x4_t(smem_u32(wt + (k + (mi & 1) * 8 + r8) * QA_LD + warp * 16 + (mi >> 1) * 8), wb);
      mma_bf16(acc[0], qa, wb[0], wb[1]);
      mma_bf16(acc[1], qa, wb[2], wb[3]);
    }
    const int g = lane >> 2;
#pragma unroll
    for (int j = 0; j < 2; j++) {
      const int col = r0 + warp * 16 + j * 8 + 2 * (lane & 3);
      if (col < a.rank_p) {
        if (b0 + g < B) *(uint32_t*)(d.q_abs + ((int64_t)(b0 + g) * a.H + h) * a.row + col) = pack_bf16(acc[j][0], acc[j][1]);
        if (b0 + g + 8 < B) *(uint32_t*)(d.q_abs + ((int64_t)(b0 + g + 8) * a.H + h) * a.row + col) = pack_bf16(acc[j][2], acc[j][3]);
      }
    }
    SB_TRACE_END(SB_K_ROPE, 0);
    return;
  }
  pdl_wait();
  SB_TRACE_WAITED();
  blk -= n_mul;
  if (blk < B * d.rot_blocks) {
    const int b = blk / d.rot_blocks, p = a.lens[b], rp = a.row - a.rank_p;
    if (p < 0 || p >= a.maxlen || p >= a.max_pos) return;
    const int i = (blk % d.rot_blocks) * 256 + (int)threadIdx.x, h = i / (rp / 2), j = i - h * (rp / 2);
    if (h < a.H) {
      float u = 0.f, v = 0.f;
      if (2 * j < a.rot) {
        const int64_t col = (int64_t)h * (a.dim + a.rot) + a.dim + 2 * j;
        u = proj(a, B, b, col);
        v = proj(a, B, b, col + 1);
        rotate(a, p, j, u, v);
      }
      *(uint32_t*)(d.q_abs + ((int64_t)b * a.H + h) * a.row + a.rank_p + 2 * j) = pack_bf16(u, v);
    }
    SB_TRACE_END(SB_K_ROPE, 0);
    return;
  }
  blk -= B * d.rot_blocks;
  if (a.cache && blk < B) {
    const int p = a.lens[blk];
    if (p < 0 || p >= a.maxlen || p >= a.max_pos) return;
    append_latent<bf16>(a, B, blk, blk, p, red);
    SB_TRACE_END(SB_K_ROPE, 0);
    return;
  }
  if (a.cache) blk -= B;
  const int b = blk / d.act_blocks, c0 = (blk % d.act_blocks) * 1024;
  bf16* act = d.act + (int64_t)b * d.ld_act;
  if (((d.act_col | d.n_act) & 3) == 0 && a.ld_in % 4 == 0 && ((uintptr_t)act & 7) == 0) {
    const int i = c0 + (int)threadIdx.x * 4;
    if (i < d.n_act) {
      const float4 v = proj4(a, B, b, d.act_col + i);
      *(uint2*)(act + i) = make_uint2(pack_bf16(sb_xielu_bf16(v.x, d.act_pos, d.act_neg), sb_xielu_bf16(v.y, d.act_pos, d.act_neg)),
                                      pack_bf16(sb_xielu_bf16(v.z, d.act_pos, d.act_neg), sb_xielu_bf16(v.w, d.act_pos, d.act_neg)));
    }
  } else {
    for (int i = c0 + (int)threadIdx.x; i < min(c0 + 1024, d.n_act); i += blockDim.x) act[i] = __float2bfloat16_rn(sb_xielu_bf16(proj(a, B, b, d.act_col + i), d.act_pos, d.act_neg));
  }
  SB_TRACE_END(SB_K_ROPE, 0);
}

// ------------------------------------------------------------------ decode: split-key attention over the latents
// grid (nsplit, ceil(H / 32), B), 256 threads; the nsplit blocks of a (sequence, head group) are one cluster. The work is two
// products per tile of 64 keys on the tcgen05 tensor cores, with the long dimension of each as the tensor-memory lanes:
//   S^T = K Q^T      A = the key tile [64 keys x row] (K-major), B = the queries [32 heads x row] (K-major, staged once);
//                    key 16 q + r = lane r of quarter q of tensor memory (M = 64), column = head.
//   O^T += c^T P     A = the same tile read MN-major, [128 latents x 64 keys] per block of 128 latents, B = the weights
//                    [64 keys x 64], MN-major: columns 0..31 the heads' hi terms, 32..63 their lo terms (P = hi + lo);
//                    lane = latent, column = head; the two halves are added at the end
// Roles by warp: 0..3 softmax (16 keys each, all heads), 4 MMA issue, 5 TMA producer. S^T is double-buffered, so S^T(t+1)
// runs under the softmax of tile t. A head's running maximum is followed lazily (only when it grew by more than 2^8, as in the
// prompt's kernel), so O^T is hardly ever rescaled.
// Key tiles are TMA atoms of 64 columns (128-byte swizzle) in a ring; an atom group's part of S^T is issued as soon as it has
// arrived. At the end every block of the cluster gets the others' sums of its share of the heads (bulk copies between the
// blocks' shared memories) and weighs them; what leaves is one bf16 row of latents per head.
// Every mbarrier wait is bounded: on expiry the error word is set and the block runs to its end.
constexpr int LKT = 64, LHEADS = 32;         // keys per tile (M of the first product), heads per block
constexpr int MAX_SPLITS = 8;               // blocks of a cluster
constexpr int ATOM = LKT * 128;             // bytes of a key tile's 64-column atom
constexpr int Q_ATOM = LHEADS * 128;        // ... and of the queries'
constexpr int P_BYTES = LKT * 128;
struct AttnDecodeDev {
  const int32_t* lens;
  int H, row, rank_p, maxlen, window, chunk, nsplit, stages;
  float scale_log2;
  bf16* out;   // [B, H, rank_p] weighted sum of latents
  int prefetch;
  int* status;
};
constexpr int MAX_STAGES = 4, GROUPS = 3;   // a tile's atoms arrive in up to three groups, each with a barrier of its own
inline int decode_atoms(int row) { return (row + 63) / 64; }
inline size_t attn_decode_smem(int row, int stages) {
  return 1024 /* round-up to the swizzle's alignment */ + (size_t)stages * decode_atoms(row) * ATOM + (size_t)decode_atoms(row) * Q_ATOM + 2 * P_BYTES;
}
// stages of the ring: as many as leave room for two blocks on an SM where the rows are short, else what one block can have
inline int decode_stages(int row, bool two_blocks) {
  for (int n = MAX_STAGES; n > 2; n--)
    if (attn_decode_smem(row, n) + 4096 <= (size_t)(two_blocks ? 113 : 226) * 1024) return n;
  return 2;
}

__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
// The issuing warps run converged, so that addresses and descriptors stay in uniform registers: one elected lane issues (a
// whole batch of products inside one elected branch measured fastest; an election per product costs 10 % of the kernel).
__device__ __forceinline__ void tc_commit_warp(uint32_t bar) {
  asm volatile(
      "{\n\t.reg .pred e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "@e tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}" ::"r"(bar)
      : "memory");
}
__device__ __forceinline__ bool elect_one() {
  uint32_t e;
  asm volatile("{\n\t.reg .pred e;\n\telect.sync _|e, 0xffffffff;\n\tselp.u32 %0, 1, 0, e;\n\t}" : "=r"(e));
  return e != 0;
}
__device__ __forceinline__ void tc_mma(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t}"
      :
      : "r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(0u)
      : "memory");
}
__device__ __forceinline__ void tc_ld16(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]),
        "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr));
}
// 16 lanes x 32 columns as four 16 x 8 tiles, each laid out like an mma.sync accumulator (rows lane / 4 and + 8, two columns)
__device__ __forceinline__ void tc_ld_16x256(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.16x256b.x4.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]),
        "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr));
}
__device__ __forceinline__ void tc_st16(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]),
      "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void tc_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tc_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// K-major operand: 128-byte rows (64 elements of the reduction dimension, 128-byte swizzle), groups of 8 rows 1024 bytes apart.
__device__ __forceinline__ uint64_t desc_kmajor(uint32_t addr) {
  return (uint64_t)((addr >> 4) & 0x3FFF) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
// MN-major operand: rows are the reduction dimension, 64 contiguous elements of the other one per row; groups of 8 rows 1024
// bytes apart, the next 64 elements in the next atom.
__device__ __forceinline__ uint64_t desc_mnmajor(uint32_t addr) {
  return (uint64_t)((addr >> 4) & 0x3FFF) | ((uint64_t)(ATOM >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
// Reduction of 8 values per lane over the 8 lanes of the same lane % 4, op = max or sum: afterwards lane 4 g + i holds the
// result of value g. Every exchange halves the values a lane still carries.
template <typename Op>
__device__ __forceinline__ float transposed_reduce(const float* v, int lane, Op op) {
  float a[4], b[2];
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const float keep = lane & 16 ? v[4 + i] : v[i], send = lane & 16 ? v[i] : v[4 + i];
    a[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 16));
  }
#pragma unroll
  for (int i = 0; i < 2; i++) {
    const float keep = lane & 8 ? a[2 + i] : a[i], send = lane & 8 ? a[i] : a[2 + i];
    b[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 8));
  }
  const float keep = lane & 4 ? b[1] : b[0], send = lane & 4 ? b[0] : b[1];
  return op(keep, __shfl_xor_sync(0xffffffffu, send, 4));
}

__global__ void __launch_bounds__(256) latent_attn_decode_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_q, AttnDecodeDev a) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024 - (smem_u32(smem_raw) & 1023)) & 1023);
  __shared__ __align__(8) uint64_t k_full[MAX_STAGES][GROUPS], k_empty[MAX_STAGES], q_full, bar_s[2], bar_p, bar_o[2], bar_m;
  __shared__ uint32_t tmem_slot;
  __shared__ float corr_s[4][LHEADS], mx_s[2][4][LHEADS];  // [softmax warp], [tile parity][softmax warp]
  __shared__ float2 ml_s[LHEADS];
  __shared__ float fs[LHEADS][MAX_SPLITS];
  SB_TRACE_BEGIN();
  const int split = blockIdx.x, h0 = blockIdx.y * LHEADS, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_atoms = (a.row + 63) / 64, stage_bytes = n_atoms * ATOM, n_mb = (a.rank_p + 127) / 128, per_group = (n_atoms + GROUPS - 1) / GROUPS;
  const uint32_t sK = smem_u32(smem), sQ = sK + (uint32_t)(a.stages * stage_bytes), sP = sQ + (uint32_t)(n_atoms * Q_ATOM);
  const uint32_t tmem_cols = n_mb <= 2 ? 256u : 512u;  // two S^T tiles of 32 columns, then 64 columns per block of latents
  if (threadIdx.x == 0) {
    for (int i = 0; i < a.stages; i++) {
      for (int g = 0; g < GROUPS; g++) mbar_init(smem_u32(&k_full[i][g]), 1);
      mbar_init(smem_u32(&k_empty[i]), 1);
    }
    mbar_init(smem_u32(&q_full), 1);
    mbar_init(smem_u32(&bar_m), 1);
    mbar_init(smem_u32(&bar_p), 128);
    for (int i = 0; i < 2; i++) { mbar_init(smem_u32(&bar_s[i]), 1); mbar_init(smem_u32(&bar_o[i]), 1); }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 5 && lane < 2) asm volatile("prefetch.tensormap [%0];" ::"l"(lane ? &map_q : &map_k) : "memory");
  if (warp == 4) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(tmem_cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  // Only now may the following kernels begin: one that also takes tensor memory and waits for this one must find this block's
  // share already allocated.
  pdl_trigger();

  auto range = [&](int len, int& kb, int& ke) {
    const int lo = a.window > 0 ? max(0, len - a.window) : 0;
    kb = lo + split * a.chunk;
    ke = min(len, kb + a.chunk);
  };
  const uint64_t policy = l2_evict_first_policy();
  uint64_t policy_q;  // the queries stay: the other blocks of the cluster read them too
  asm volatile("createpolicy.fractional.L2::evict_last.b64 %0, 1.0;" : "=l"(policy_q));
  // The producer warp. Rows beyond the chunk are whatever the cache holds there (finite, or zeros beyond its end); their
  // weights are zero.
  auto load_tile = [&](int st, int row) {
#pragma unroll
    for (int g = 0; g < GROUPS; g++) {
      const int first = g * per_group, n = min(per_group, n_atoms - first);
      if (n <= 0) break;
      const uint32_t bar = smem_u32(&k_full[st][g]);
      mbar_expect_tx_warp(bar, (uint32_t)(n * ATOM));
#pragma unroll 1
      for (int i = first; i < first + n; i++) tma_load_2d_warp(sK + (uint32_t)(st * stage_bytes + i * ATOM), &map_k, i * 64, row, bar, policy);
    }
  };
  // Tiles that hold rows of earlier steps only are requested before the dependency wait; the length they are derived from is
  // read again after it. (It belongs to the previous step and has not changed; if it had, the step would report an error.)
  int kb, ke, n_early = 0;
  const int len_early = min(ld_volatile_i32(a.lens + b) + 1, a.maxlen);
  range(len_early, kb, ke);
  if (a.prefetch)
    for (; n_early < a.stages && kb + (n_early + 1) * LKT <= min(ke, len_early - 1); n_early++)
      if (warp == 5) load_tile(n_early, b * a.maxlen + kb + n_early * LKT);
  pdl_wait();
  SB_TRACE_WAITED();
  const int len = min(ld_volatile_i32(a.lens + b) + 1, a.maxlen);
  int err = 0;
  if (len != len_early && n_early) err = 17;
  else range(len, kb, ke);
  const int ntiles = kb < ke ? (ke - kb + LKT - 1) / LKT : 0;
  auto wait = [&](uint64_t* bar, int parity, int code) {
    if (!err && !mbar_wait(smem_u32(bar), (uint32_t)parity & 1)) err = code;
    return err == 0;
  };
  if (warp == 5) {
    // ---- TMA producer, the whole warp in step
    if (ntiles > 0) {
      mbar_expect_tx_warp(smem_u32(&q_full), (uint32_t)(n_atoms * Q_ATOM));
#pragma unroll 1
      for (int i = 0; i < n_atoms; i++) tma_load_2d_warp(sQ + (uint32_t)(i * Q_ATOM), &map_q, i * 64, b * a.H + h0, smem_u32(&q_full), policy_q);
      int st = n_early == a.stages ? 0 : n_early, free_parity = 1;  // the first pass over the ring needs no waiting
      for (int t = n_early; t < ntiles; t++) {
        if (st == 0 && t > 0) free_parity ^= 1;
        if (t >= a.stages && !__all_sync(0xffffffffu, wait(&k_empty[st], free_parity, 18))) break;
        load_tile(st, b * a.maxlen + kb + t * LKT);
        if (++st == a.stages) st = 0;
      }
    }
  } else if (warp == 4) {
    // ---- MMA issue, the whole warp in step: O^T of the current tile when its weights are there, else S^T of the
    // next one as far as its atoms have arrived
    // D = F32, A = B = BF16; M = 64 keys, N = 32 heads, or M = 128 latents, N = 64 with both operands MN-major
    constexpr uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(LHEADS >> 3) << 17) | ((uint32_t)(LKT >> 4) << 24);
    constexpr uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 15) | (1u << 16) | ((uint32_t)(64 >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
    // an operand advances by constants: 16 columns = 32 bytes, an atom = ATOM bytes, 16 keys = 2048 bytes (units of 16 bytes)
    const uint64_t dk0 = desc_kmajor(sK), dq0 = desc_kmajor(sQ), dc0 = desc_mnmajor(sK), dp0 = desc_mnmajor(sP);
    const uint32_t td = __shfl_sync(0xffffffffu, tmem, 0);
    const int stage16 = stage_bytes >> 4;
    int st = 0, ps = 0;  // ring stages of the next S^T and the next O^T product,
    int sp = 0, pr = 0;  // the parities of their barriers,
    int sg = 0;          // and the group of atoms the next S^T continues with
    int ns = 0, np = 0;  // tiles whose S^T / O^T product has been issued
    auto ready = [&](uint64_t* bar, int parity) {
      uint32_t done;
      asm volatile(
          "{\n\t.reg .pred p;\n\t"
          "mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
          "selp.u32 %0, 1, 0, p;\n\t}"
          : "=r"(done)
          : "r"(smem_u32(bar)), "r"((uint32_t)parity)
          : "memory");
      return __all_sync(0xffffffffu, done);
    };
    if (ntiles > 0) wait(&q_full, 0, 20);
    bool go = __all_sync(0xffffffffu, err == 0);
    uint32_t spins = 0;
    while (np < ntiles && go) {
      if (ns > np && ready(&bar_p, pr)) {  // the weights are in shared memory, O^T follows the new maxima
        tc_fence_after();
        const uint64_t dc = dc0 + (uint64_t)(uint32_t)(ps * stage16), dp = dp0 + (uint64_t)(uint32_t)((np & 1) * (P_BYTES >> 4));
        if (elect_one()) {
#pragma unroll
          for (int s = 0; s < LKT / 16; s++)  // 16 keys = 16 rows of 128 bytes; the blocks of latents take turns
#pragma unroll
            for (int mb = 0; mb < 4; mb++)
              if (mb < n_mb) tc_mma(td + 64u + (uint32_t)(mb * 64), dc + (uint64_t)((2 * mb * ATOM + s * 2048) >> 4), dp + (uint64_t)(s * 2048 >> 4), idesc_pv, (np | s) ? 1u : 0u);
        }
        __syncwarp();
        tc_commit_warp(smem_u32(&bar_o[np & 1]));
        tc_commit_warp(smem_u32(&k_empty[ps]));
        np++;
        pr ^= 1;
        if (++ps == a.stages) ps = 0;
        spins = 0;
      } else if (ns < ntiles && ns <= np + 1 && ready(&k_full[st][sg], sp)) {
        tc_fence_after();
        const int first = sg * per_group, last = min(n_atoms, first + per_group);
        const uint32_t d = td + (uint32_t)((ns & 1) * LHEADS);
        const uint64_t dkb = dk0 + (uint64_t)(uint32_t)(st * stage16 + first * (ATOM >> 4)), dqb = dq0 + (uint64_t)(uint32_t)(first * (Q_ATOM >> 4));
        if (elect_one()) {
#pragma unroll
          for (int i = 0; i < 4; i++)  // a group is at most four atoms; a row's last one is zero beyond its width
            if (first + i < last) {
              const uint64_t dk = dkb + (uint64_t)(i * (ATOM >> 4)), dq = dqb + (uint64_t)(i * (Q_ATOM >> 4));
              tc_mma(d, dk, dq, idesc_s, first + i ? 1u : 0u);
              tc_mma(d, dk + 2, dq + 2, idesc_s, 1u);
              tc_mma(d, dk + 4, dq + 4, idesc_s, 1u);
              tc_mma(d, dk + 6, dq + 6, idesc_s, 1u);
            }
        }
        __syncwarp();
        sg++;
        if (last == n_atoms) {
          tc_commit_warp(smem_u32(&bar_s[ns & 1]));
          ns++;
          sg = 0;
          if (++st == a.stages) { st = 0; sp ^= 1; }
        }
        spins = 0;
      } else if (++spins > (1u << 24)) {
        err = 21;
        go = false;
      }
    }
  } else if (warp < 4) {
    // ---- softmax. A thread has two keys (rows g and g + 8 of its warp's 16) of eight heads (columns 8 j + 2 tig, + 1); lane L
    // also keeps head L's running maximum, the same in all four warps.
    const int g = lane >> 2, tig = lane & 3, key = warp * 16 + g;
    float m_run = -INFINITY, l_run[8];
#pragma unroll
    for (int i = 0; i < 8; i++) l_run[i] = 0.f;
    uint8_t* const p_row = smem + (sP - sK) + warp * 2048 + g * 128 + tig * 4;
    for (int t = 0; t < ntiles; t++) {
      wait(&bar_s[t & 1], t >> 1, 23);
      if (t == 0) SB_TRACE_MARK(0);
      __syncwarp();
      tc_fence_after();
      uint32_t r[16];
      tc_ld_16x256(tmem + (uint32_t)((t & 1) * LHEADS) + ((uint32_t)(warp * 32) << 16), r);
      tc_wait_ld();
      const int left = ke - kb - t * LKT - key;
      float v[16], mx[8];
#pragma unroll
      for (int j = 0; j < 4; j++)
#pragma unroll
        for (int k = 0; k < 2; k++) {
          v[4 * j + k] = left > 0 ? __uint_as_float(r[4 * j + k]) * a.scale_log2 : -INFINITY;
          v[4 * j + 2 + k] = left > 8 ? __uint_as_float(r[4 * j + 2 + k]) * a.scale_log2 : -INFINITY;
          mx[2 * j + k] = fmaxf(v[4 * j + k], v[4 * j + 2 + k]);
        }
      mx_s[t & 1][warp][8 * (g >> 1) + 2 * tig + (g & 1)] = transposed_reduce(mx, lane, [](float x, float y) { return fmaxf(x, y); });
      asm volatile("bar.sync 1, 128;" ::: "memory");
      const float m_tile = fmaxf(fmaxf(mx_s[t & 1][0][lane], mx_s[t & 1][1][lane]), fmaxf(mx_s[t & 1][2][lane], mx_s[t & 1][3][lane]));
      const bool grow = m_tile > m_run + 8.0f;  // also for the first tile (m_run = -inf)
      if (__any_sync(0xffffffffu, grow)) {      // the same in all four warps
        const float m_use = grow ? m_tile : m_run, corr = grow ? ex2_approx(m_run - m_use) : 1.0f;
        m_run = m_use;
#pragma unroll
        for (int i = 0; i < 8; i++) l_run[i] *= __shfl_sync(0xffffffffu, corr, 8 * (i >> 1) + 2 * tig + (i & 1));
        if (t > 0) {
          corr_s[warp][lane] = corr;
          wait(&bar_o[(t - 1) & 1], (t - 1) >> 1, 24);  // the previous product must have finished writing O^T
          __syncwarp();
          tc_fence_after();
          const uint32_t base = tmem + 64u + ((uint32_t)(warp * 32) << 16);
          for (int c = 0; c < n_mb * 4; c++) {
            uint32_t x[16];
            tc_ld16(base + (uint32_t)(c * 16), x);
            tc_wait_ld();
#pragma unroll
            for (int j = 0; j < 16; j++) x[j] = __float_as_uint(__uint_as_float(x[j]) * corr_s[warp][(c & 1) * 16 + j]);
            tc_st16(base + (uint32_t)(c * 16), x);
          }
          tc_wait_st();
        }
      }
      if (t >= 2) wait(&bar_o[t & 1], (t - 2) >> 1, 25);  // this half of the weight buffer is free
      __syncwarp();
      uint8_t* const pw = p_row + (t & 1) * P_BYTES;
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const float m0 = __shfl_sync(0xffffffffu, m_run, 8 * j + 2 * tig), m1 = __shfl_sync(0xffffffffu, m_run, 8 * j + 2 * tig + 1);
#pragma unroll
        for (int k = 0; k < 2; k++) {
          const float p0 = ex2_approx(v[4 * j + 2 * k] - m0), p1 = ex2_approx(v[4 * j + 2 * k + 1] - m1);
          l_run[2 * j] += p0;
          l_run[2 * j + 1] += p1;
          uint32_t hi, lo;
          split_bf16x2(p0, p1, hi, lo);
          *(uint32_t*)(pw + k * 1024 + ((j ^ g) << 4)) = hi;
          *(uint32_t*)(pw + k * 1024 + (((4 + j) ^ g) << 4)) = lo;
        }
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // the tensor cores read what these stores wrote
      tc_fence_before();
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&bar_p)) : "memory");
    }
    // sums over the keys; the barrier keeps them out of maxima that are still being read
    asm volatile("bar.sync 1, 128;" ::: "memory");
    mx_s[0][warp][8 * (g >> 1) + 2 * tig + (g & 1)] = transposed_reduce(l_run, lane, [](float x, float y) { return x + y; });
    if (warp == 0) ml_s[lane].x = m_run;
  }
  __syncwarp();
  if (ntiles > 0) wait(&bar_o[(ntiles - 1) & 1], (ntiles - 1) >> 1, 26);  // every product is complete
  __syncwarp();
  tc_fence_after();
  SB_TRACE_MARK(1);
  __syncthreads();  // the ring is free: it holds this block's sums now
  float* so = (float*)smem;  // [32][rank_p + 4]
  const int so_ld = a.rank_p + 4;
  if (ntiles > 0) {
    for (int mb = warp >> 2; mb < n_mb; mb += 2) {
      const int lat = mb * 128 + (warp & 3) * 32 + lane;
      const uint32_t base = tmem + 64u + (uint32_t)(mb * 64) + ((uint32_t)((warp & 3) * 32) << 16);
#pragma unroll
      for (int c = 0; c < 2; c++) {
        uint32_t x[16], y[16];
        tc_ld16(base + (uint32_t)(c * 16), x);
        tc_ld16(base + (uint32_t)(32 + c * 16), y);
        tc_wait_ld();
        if (lat < a.rank_p) {
#pragma unroll
          for (int j = 0; j < 16; j++) so[(c * 16 + j) * so_ld + lat] = __uint_as_float(x[j]) + __uint_as_float(y[j]);
        }
      }
    }
  }
  if (threadIdx.x < LHEADS) {
    const float l = (mx_s[0][0][threadIdx.x] + mx_s[0][1][threadIdx.x]) + (mx_s[0][2][threadIdx.x] + mx_s[0][3][threadIdx.x]);
    ml_s[threadIdx.x].y = l;  // without keys: (-inf, 0)
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // the copies below read what the stores above wrote
  tc_fence_before();
  __syncthreads();
  if (warp == 4) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(tmem_cols) : "memory");
  }
  // Every block owns some of the heads: the others' rows of those heads come as one bulk copy each, [source][own head][rank_p + 4].
  const int own = (LHEADS + a.nsplit - 1) / a.nsplit, first = split * own, n_own = max(0, min(own, LHEADS - first));
  const uint32_t slot_bytes = (uint32_t)(own * so_ld * 4);
  uint8_t* recv = smem + LHEADS * so_ld * 4;
  if (threadIdx.x == 0 && a.nsplit > 1) mbar_expect_tx(smem_u32(&bar_m), (uint32_t)((a.nsplit - 1) * n_own * so_ld * 4));
  cluster_sync();  // every block's sums are complete and every ring is free
  if (threadIdx.x < a.nsplit && (int)threadIdx.x != split) {
    const int to = threadIdx.x, n = max(0, min(own, LHEADS - to * own));
    if (n > 0)
      asm volatile("cp.async.bulk.shared::cluster.shared::cta.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(map_to_rank(smem_u32(recv) + (uint32_t)split * slot_bytes, to)),
                   "r"(smem_u32(so + to * own * so_ld)), "r"((uint32_t)(n * so_ld * 4)), "r"(map_to_rank(smem_u32(&bar_m), to))
                   : "memory");
  }
  {  // weights of the chunks: eight neighbouring threads per head, one per chunk
    const int h = threadIdx.x >> 3, p = threadIdx.x & 7;
    float2 ml = make_float2(-INFINITY, 0.f);
    if (h < n_own && p < a.nsplit) ml = ld_cluster2(map_to_rank(smem_u32(&ml_s[first + h]), p));
    float M = ml.x;
#pragma unroll
    for (int off = 1; off < 8; off <<= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, off));
    const float f = ml.y > 0.f ? ex2_approx(ml.x - M) : 0.f;
    float L = f * ml.y;
#pragma unroll
    for (int off = 1; off < 8; off <<= 1) L += __shfl_xor_sync(0xffffffffu, L, off);
    fs[h][p] = f > 0.f ? f / L : 0.f;
  }
  __syncthreads();
  if (a.nsplit > 1) wait(&bar_m, 0, 27);
  SB_TRACE_MARK(2);
  const int c4n = a.rank_p / 4, heads = min(n_own, a.H - h0 - first);
  for (int i = threadIdx.x; i < heads * c4n; i += 256) {
    const int h = i / c4n, c = (i - h * c4n) * 4;
    const float* mine = so + (first + h) * so_ld + c;
    const float* theirs = (const float*)recv + h * so_ld + c;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 1
    for (int p = 0; p < a.nsplit; p++, theirs += own * so_ld) {
      const float w = fs[h][p];
      if (w != 0.f) {  // a block without keys has weight zero
        const float4 x = *(const float4*)(p == split ? mine : theirs);
        acc.x += w * x.x; acc.y += w * x.y; acc.z += w * x.z; acc.w += w * x.w;
      }
    }
    *(uint2*)(a.out + ((int64_t)b * a.H + h0 + first + h) * a.rank_p + c) = make_uint2(pack_bf16(acc.x, acc.y), pack_bf16(acc.z, acc.w));
  }
  if (err) { *(volatile int*)a.status = err; __threadfence_system(); }
  cluster_sync();  // nobody leaves while another block may still read its shared memory
  SB_TRACE_END(SB_K_ATTN, 0);
}

// grid (H, ceil(vdim / 64), ceil(B / 16)), 256 threads: 64 value columns of one head for 16 tokens, W_uv times the weighted
// latents (W_uv is a constant, requested before the dependency wait).
struct ValueDev {
  const bf16* lat;  // [B, H, rank_p]
  int B, H, rank_p, vdim;
  const bf16* wv;   // value rows: head h, value v at (h * kv_head + v) * rank_p
  int kv_head;
  bf16* out;
  int64_t ldo;
};
__global__ void __launch_bounds__(256) latent_value_kernel(ValueDev a) {
  extern __shared__ __align__(128) uint8_t smem[];
  SB_TRACE_BEGIN();
  pdl_trigger();
  const int h = blockIdx.x, v0 = blockIdx.y * 64, b0 = blockIdx.z * 16, ld = a.rank_p + 8;
  bf16* wt = (bf16*)smem;      // [64][ld]
  bf16* ot = wt + 64 * ld;     // [16][ld]
  const int cpr = a.rank_p / 8;
  for (int c = threadIdx.x; c < 64 * cpr; c += 256) {
    const int r = c / cpr, cc = c - r * cpr;
    const bool ok = v0 + r < a.vdim;
    cp_async16(smem_u32(wt + r * ld + cc * 8), a.wv + ((int64_t)h * a.kv_head + (ok ? v0 + r : 0)) * a.rank_p + cc * 8, ok);
  }
  pdl_wait();
  SB_TRACE_WAITED();
  for (int c = threadIdx.x; c < 16 * cpr; c += 256) {
    const int m = c / cpr, cc = c - m * cpr;
    const bool ok = b0 + m < a.B;
    cp_async16(smem_u32(ot + m * ld + cc * 8), a.lat + ((int64_t)(ok ? b0 + m : 0) * a.H + h) * a.rank_p + cc * 8, ok);
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3, r8 = lane & 7;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < a.rank_p; k0 += 64) {
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int k = k0 + 16 * i;
      if (k < a.rank_p) {
        uint32_t oa[4], wb[2];
        ldsm_x4(smem_u32(ot + ((mi & 1) * 8 + r8) * ld + k + (mi >> 1) * 8), oa);
        ldsm_x2(smem_u32(wt + (warp * 8 + r8) * ld + k + (mi & 1) * 8), wb);
        mma_bf16(acc[i], oa, wb[0], wb[1]);
      }
    }
  }
  const int g = lane >> 2, v = v0 + warp * 8 + 2 * (lane & 3);
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int b = b0 + g + (i >> 1) * 8, vc = v + (i & 1);
    if (b < a.B && vc < a.vdim)
      a.out[(int64_t)b * a.ldo + (int64_t)h * a.vdim + vc] = __float2bfloat16_rn((acc[0][i] + acc[1][i]) + (acc[2][i] + acc[3][i]));
  }
  SB_TRACE_END(SB_K_COMBINE, 0);
}

// ------------------------------------------------------------------ any width, bf16 or fp32
// grid (H, T), 256 threads; 256 keys per step, fp32 arithmetic throughout.
template <typename T>
__global__ void __launch_bounds__(256) latent_attn_any_kernel(LatentShape s, const T* __restrict__ q, const T* __restrict__ cache, const T* __restrict__ wkv,
                                                              const int32_t* __restrict__ seq, const int32_t* __restrict__ pos,
                                                              const int32_t* __restrict__ lens, int maxlen, T* __restrict__ out, int64_t ldo) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int64_t t = blockIdx.y;
  const int b = seq ? seq[t] : (int)t, p = pos ? pos[t] : lens[b];
  if (p < 0 || p >= maxlen) return;
  const int rank_p = s.rank_p(), row = s.row();
  float* qa = sm;                // [rank] the query in latent space
  float* qr = qa + s.rank;       // [rot]
  float* ol = qr + s.rot;        // [rank] weighted sum of latents
  float* sc = ol + s.rank;       // [256]
  float* qu = sc + 256;          // [dim]
  const T* qp = q + (t * s.H + h) * s.q_head();
  for (int i = tid; i < s.dim; i += 256) qu[i] = to_f(qp[i]);
  for (int i = tid; i < s.rot; i += 256) qr[i] = to_f(qp[s.dim_p() + i]);
  for (int i = tid; i < s.rank; i += 256) ol[i] = 0.f;
  __syncthreads();
  for (int r = tid; r < s.rank; r += 256) {
    const T* w = wkv + (int64_t)h * s.kv_head() * rank_p + r;
    float acc = 0.f;
    for (int d = 0; d < s.dim; d++) acc += qu[d] * to_f(w[(int64_t)d * rank_p]);
    qa[r] = acc;
  }
  __syncthreads();
  const T* base = cache + (int64_t)b * maxlen * row;
  const int lo = s.window > 0 ? max(0, p - s.window + 1) : 0;
  float m_run = -INFINITY, l_run = 0.f;
  for (int k0 = lo; k0 <= p; k0 += 256) {
    const int n = min(256, p + 1 - k0);
    for (int j = warp; j < n; j += 8) {
      const T* c = base + (int64_t)(k0 + j) * row;
      float acc = 0.f;
      for (int r = lane; r < s.rank; r += 32) acc += qa[r] * to_f(c[r]);
      for (int r = lane; r < s.rot; r += 32) acc += qr[r] * to_f(c[rank_p + r]);
      acc = warp_sum(acc);
      if (lane == 0) sc[j] = acc * s.scale;
    }
    __syncthreads();
    const float mine = tid < n ? sc[tid] : -INFINITY;
    const float m_new = fmaxf(m_run, block_max(mine, red));
    const float e = tid < n ? expf(mine - m_new) : 0.f;
    const float corr = expf(m_run - m_new);
    l_run = l_run * corr + block_sum(e, red);
    m_run = m_new;
    sc[tid] = e;
    __syncthreads();
    for (int r = tid; r < s.rank; r += 256) {
      float acc = ol[r] * corr;
      for (int j = 0; j < n; j++) acc += sc[j] * to_f(base[(int64_t)(k0 + j) * row + r]);
      ol[r] = acc;
    }
    __syncthreads();
  }
  const float inv = 1.0f / l_run;
  const T* wv = wkv + (int64_t)(s.H + h) * s.kv_head() * rank_p;
  for (int v = warp; v < s.vdim; v += 8) {
    float acc = 0.f;
    for (int r = lane; r < s.rank; r += 32) acc += ol[r] * to_f(wv[(int64_t)v * rank_p + r]);
    acc = warp_sum(acc);
    if (lane == 0) out[t * ldo + (int64_t)h * s.vdim + v] = to_t<T>(acc * inv);
  }
}

SplitDev split_dev(const LatentSplitArgs& a) {
  const LatentShape& s = a.s;
  return SplitDev{s.H, s.dim, s.rot, s.rank, s.rank_p(), s.row(), s.q_head(), s.dim_p(), a.in, a.ld_in, a.splits, a.seq, a.pos, a.lens, a.cos_t, a.sin_t,
                  a.max_pos, a.maxlen, a.norm_w, a.eps, a.q_out, a.cache};
}

// Shared-memory limit of a kernel, raised per device to the largest size asked for.
template <typename F>
int allow_smem(strictb200_ctx* ctx, F kernel, size_t bytes, size_t* have /* [64] of this kernel */) {
  static std::mutex mu;
  std::lock_guard<std::mutex> lock(mu);
  size_t& h = have[ctx->device & 63];
  if (bytes > 32 * 1024 && bytes > h) {  // the default limit of 48 KB counts the static share too
    SB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    h = bytes;
  }
  return STRICTB200_OK;
}
constexpr size_t SMEM_MAX = 227 * 1024 - 1024;  // what a block may take, less the kernels' static share

typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                             const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
// 2D map of bf16 rows [rows, row], box = box_rows x 64 columns (128 bytes), 128-byte swizzle.
int rows_map(CUtensorMap* map, const bf16* base, int64_t rows, int row, int box_rows) {
  static EncodeFn encode = nullptr;
  if (!encode) {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult q;
    SB_CUDA(cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q));
    if (!fn || q != cudaDriverEntryPointSuccess) return sb_fail(STRICTB200_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    encode = (EncodeFn)fn;
  }
  cuuint64_t dims[2] = {(cuuint64_t)row, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)row * 2};
  cuuint32_t box[2] = {64u, (cuuint32_t)box_rows};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<bf16*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                      CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return sb_fail(STRICTB200_ERR_CUDA, "cuTensorMapEncodeTiled failed with code " + std::to_string((int)r));
  return STRICTB200_OK;
}

}  // namespace

SB_TRACE_TU(latent)

int k_latent_split(strictb200_ctx* ctx, const LatentSplitArgs& a, int64_t T) {
  const SplitDev d = split_dev(a);
  const dim3 grid((unsigned)T, a.cache ? 2u : 1u);
  if (a.f32) SB_CUDA(sb_launch(ctx, latent_split_kernel<float>, grid, dim3(256), 0, d, T));
  else SB_CUDA(sb_launch(ctx, latent_split_kernel<bf16>, grid, dim3(256), 0, d, T));
  ctx->launches++;
  return STRICTB200_OK;
}

int k_latent_gather(strictb200_ctx* ctx, const bf16* cache, int64_t maxlen, int row, const int32_t* koff, const int32_t* kpos0, const int32_t* lens, int nb,
                    int max_n, bf16* dst) {
  const int64_t vec = (int64_t)max_n * (row / 8);
  const unsigned gx = (unsigned)std::min<int64_t>((vec + 127) / 128, 512);
  latent_gather_kernel<<<dim3(gx, (unsigned)nb), 128, 0, ctx->stream>>>(cache, maxlen, row, koff, kpos0, lens, dst);
  SB_LAUNCHED(ctx);
  return STRICTB200_OK;
}

bool sb_latent_decode_fits(const LatentShape& s) {
  return s.rank_p() <= 512 && s.row() <= 640 && s.dim <= 512 && decode_in_smem(s.dim) <= (int)SMEM_MAX;  // 512 latents fill the tensor memory
}

int k_latent_decode_in(strictb200_ctx* ctx, const LatentDecodeInArgs& x, int64_t B) {
  static size_t have[64] = {};
  const LatentShape& s = x.a.s;
  DecodeInDev d{split_dev(x.a), x.wkv, s.kv_head(), x.q_abs, x.act_col, x.n_act, x.act_pos, x.act_neg, x.act, x.ld_act,
                (s.rank_p() + QA_COLS - 1) / QA_COLS, (int)((B + 15) / 16), (s.H * (s.row() - s.rank_p()) / 2 + 255) / 256, (x.n_act + 1023) / 1024};
  const size_t smem = decode_in_smem(s.dim);
  SB_TRY(allow_smem(ctx, latent_decode_in_kernel, smem, have));
  const int64_t blocks = (int64_t)s.H * d.n_rt * d.n_grp + B * (d.rot_blocks + (x.a.cache ? 1 : 0) + d.act_blocks);
  if (x.a.splits > 8) return sb_fail(STRICTB200_ERR_INVALID_ARG, "latent decode: at most 8 partial sums");
  SB_CUDA(sb_launch(ctx, latent_decode_in_kernel, dim3((unsigned)blocks), dim3(256), smem, d, (int)B));
  ctx->launches++;
  return STRICTB200_OK;
}

// Two blocks on an SM: half of the tensor memory each, and a ring of at least three stages in half of the shared memory.
bool two_decode_blocks(const LatentShape& s) { return s.rank_p() <= 256 && attn_decode_smem(s.row(), 3) + 4096 <= 113 * 1024; }

// Keys per block: waves of blocks x (key tiles per block + what a block costs besides), over the multiples of the tile that
// leave at most MAX_SPLITS chunks of the window (or of the planned length, where that is shorter). The chunks of a (sequence,
// head group) are one cluster, and clusters of 3, 5, 6 or 7 blocks pack the SMs of a GPC badly: 1, 2, 4 or 8 chunks.
int sb_latent_decode_chunk(strictb200_ctx* ctx, const LatentShape& s, int B, int len_plan) {
  const int n = s.window > 0 ? std::min(s.window, len_plan) : len_plan, tiles = std::max(1, (n + LKT - 1) / LKT);
  const int64_t slots = (int64_t)ctx->sm_count * (two_decode_blocks(s) ? 2 : 1), pairs = (int64_t)B * ((s.H + LHEADS - 1) / LHEADS);
  int best = tiles;
  double best_cost = 1e30;
  for (int k = 1; k <= MAX_SPLITS && k <= tiles; k *= 2) {
    const int c = (tiles + k - 1) / k;
    const int64_t blocks = pairs * k, waves = (blocks + slots - 1) / slots;
    const double cost = (double)waves * (c + 3);
    if (cost < best_cost - 1e-9) { best_cost = cost; best = c; }
  }
  return best * LKT;
}
size_t sb_latent_decode_scratch(const LatentShape& s, int B) { return (size_t)B * s.H * s.rank_p() * sizeof(bf16); }

int k_latent_attn_decode(strictb200_ctx* ctx, const LatentShape& s, const bf16* q_abs, const bf16* cache, const int32_t* lens, int B, int maxlen, int chunk,
                         int nsplit, bf16* scratch, const bf16* wkv, bf16* out, int64_t ldo) {
  if (!sb_latent_decode_fits(s)) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "latent decode attention: rows too wide for the tensor-core kernel");
  if (nsplit < 1 || nsplit > MAX_SPLITS || chunk < LKT || chunk % LKT || B > 65535) return sb_fail(STRICTB200_ERR_INVALID_ARG, "latent decode attention: bad key chunks");
  if ((int64_t)B * maxlen > INT32_MAX) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "latent decode attention: cache too large for 32-bit tile coordinates");
  const int rp = s.rank_p(), stages = decode_stages(s.row(), two_decode_blocks(s));
  CUtensorMap map_k, map_q;
  SB_TRY(rows_map(&map_k, cache, (int64_t)B * maxlen, s.row(), LKT));
  SB_TRY(rows_map(&map_q, q_abs, (int64_t)B * s.H, s.row(), LHEADS));
  AttnDecodeDev a{lens, s.H, s.row(), rp, maxlen, s.window, chunk, nsplit, stages, s.scale * LOG2E, scratch, ctx->opt.attn_prefetch, ctx->d_status};
  {
    static size_t have[64] = {};
    // The blocks of a cluster wait for one another, so no block may wait for tensor memory that a waiting block holds: shared
    // memory admits no more blocks to an SM than its tensor memory does (one with all 512 columns, or two with 256).
    const size_t smem = std::max(attn_decode_smem(s.row(), stages), (size_t)(rp > 256 ? 116 : 78) * 1024);
    SB_TRY(allow_smem(ctx, latent_attn_decode_kernel, smem, have));
    SB_CUDA(sb_launch_cluster(ctx, latent_attn_decode_kernel, dim3(nsplit, (s.H + LHEADS - 1) / LHEADS, B), dim3(256), smem, dim3(nsplit, 1, 1), map_k, map_q, a));
    ctx->launches++;
  }
  sb_prof_split(ctx, STRICTB200_K_ATTN_MERGE);
  static size_t have[64] = {};
  const size_t smem = (size_t)(64 + 16) * (rp + 8) * 2;
  SB_TRY(allow_smem(ctx, latent_value_kernel, smem, have));
  ValueDev m{scratch, B, s.H, rp, s.vdim, wkv + (int64_t)s.H * s.kv_head() * rp, s.kv_head(), out, ldo};
  SB_CUDA(sb_launch(ctx, latent_value_kernel, dim3(s.H, (s.vdim + 63) / 64, (B + 15) / 16), dim3(256), smem, m));
  ctx->launches++;
  return STRICTB200_OK;
}

int k_latent_attn_any(strictb200_ctx* ctx, const LatentShape& s, bool f32, const void* q, const void* cache, const void* wkv, const int32_t* seq,
                      const int32_t* pos, const int32_t* lens, int64_t T, int maxlen, void* out, int64_t ldo) {
  const size_t smem = ((size_t)2 * s.rank + s.rot + s.dim + 256) * sizeof(float);
  if (smem > SMEM_MAX) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "latent attention: the latent does not fit a block's shared memory");
  static size_t have_f[64] = {}, have_b[64] = {};
  const size_t es = f32 ? 4 : 2;
  for (int64_t t0 = 0; t0 < T; t0 += 32768) {  // rows are the grid's second dimension
    const int64_t n = std::min<int64_t>(32768, T - t0);
    if (!seq && t0) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "latent attention: too many sequences");
    const void* qt = (const char*)q + (size_t)t0 * s.H * s.q_head() * es;
    void* ot = (char*)out + (size_t)t0 * ldo * es;
    const int32_t *sq = seq ? seq + t0 : nullptr, *ps = pos ? pos + t0 : nullptr;
    if (f32) {
      SB_TRY(allow_smem(ctx, latent_attn_any_kernel<float>, smem, have_f));
      SB_CUDA(sb_launch(ctx, latent_attn_any_kernel<float>, dim3(s.H, (unsigned)n), dim3(256), smem, s, (const float*)qt, (const float*)cache, (const float*)wkv, sq,
                        ps, lens, maxlen, (float*)ot, ldo));
    } else {
      SB_TRY(allow_smem(ctx, latent_attn_any_kernel<bf16>, smem, have_b));
      SB_CUDA(sb_launch(ctx, latent_attn_any_kernel<bf16>, dim3(s.H, (unsigned)n), dim3(256), smem, s, (const bf16*)qt, (const bf16*)cache, (const bf16*)wkv, sq, ps,
                        lens, maxlen, (bf16*)ot, ldo));
    }
    ctx->launches++;
  }
  return STRICTB200_OK;
}
