// Latent attention: a position leaves one low-rank vector (the latent, RMS-normed) and one rotated key part that all heads
// share; a head's unrotated key and its value are W_uk c and W_uv c. The cache row of a position is [latent | rotated part],
// each padded with zeros to a multiple of 16 elements, whatever the number of heads.
//
//  * prompts: keys and values are rebuilt per head by one GEMM over the visible latents, then the tcgen05 prefill kernel
//    runs on them (attention_tc.cu). Here: the projection's rows into rotated queries and cache rows.
//  * decode: nothing is rebuilt. A head's query is carried into latent space (q' = q W_uk), so that q' . c replaces
//    q . W_uk c, all heads read the same cache row (the heads are the rows of the MMA tile) and the weighted sum of latents
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
__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar, uint64_t policy) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint [%0], [%1, {%2, %3}], [%4], %5;" ::"r"(dst),
               "l"(map), "r"(x), "r"(y), "r"(bar), "l"(policy)
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
__device__ __forceinline__ float4 ld_cluster4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
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
// the same with a zero accumulator
__device__ __forceinline__ void mma_bf16_zero(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%10,%10,%10,%10};\n"
      : "=f"(d[0]), "=f"(d[1]), "=f"(d[2]), "=f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1), "f"(0.f));
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
// grid (nsplit, ceil(H / (16 MT)), B), 32 NW threads; the nsplit blocks of a (sequence, head group) are one cluster. Rows of
// the MMA tiles = up to 16 MT heads, 32 keys per step. Three products of three different steps share an iteration:
//   S(t+1) partials  warp (ks, kh): reduction steps ks, ks + SL, .. of the cache row for the 16 keys of half kh; its share of
//                    the queries stays in registers for the whole block, so a step reads the key tile from shared memory once
//   softmax(t)       the SL partial scores of a (head, key) are added in slice order; running maximum and sum per head
//   O += P(t-1) c    every warp owns 8 NV latent columns of all heads; the key tile is its operand again
// A key tile is copied by TMA in atoms of 32 rows x 64 columns (128-byte swizzle: 16-byte chunk c of row r lies at c ^ (r & 7));
// tiles pass through a ring of four stages (t-1, t, t+1 in use, t+2 in flight). At the end the cluster's blocks weigh each other's sums through distributed shared memory, so what leaves
// is one bf16 row of latents per head.
constexpr int LKT = 32, NS = 4;
constexpr int MAX_SPLITS = 8;  // blocks of a cluster
struct AttnDecodeDev {
  const bf16* q;
  const int32_t* lens;
  int H, row, rank_p, maxlen, window, chunk, nsplit;
  float scale_log2;
  bf16* out;   // [B, H, rank_p] weighted sum of latents
  int prefetch;
  int* status;
};
constexpr int SP_LD = 36, PP_LD = 40;  // row strides of the score (fp32) and weight (bf16) tiles
constexpr int ATOM = LKT * 128;        // bytes of a tile's 64-column atom
constexpr size_t attn_decode_smem(int mt, int nw, int row) {
  return 1024 /* round-up to the swizzle's alignment */ + (size_t)NS * ((row + 63) / 64) * ATOM + (size_t)(nw / 2) * mt * 16 * SP_LD * 4 + (size_t)2 * 2 * mt * 16 * PP_LD * 2 + 2 * mt * 16 * 4;
}

template <int MT, int NW, int KSM, int NV>
__global__ void __launch_bounds__(NW * 32) latent_attn_decode_kernel(const __grid_constant__ CUtensorMap map, AttnDecodeDev a) {
  constexpr int R = MT * 16, SL = NW / 2, NT = NW * 32;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024 - (smem_u32(smem_raw) & 1023)) & 1023);
  __shared__ __align__(8) uint64_t full[NS];
  __shared__ float2 ml_s[R];
  __shared__ float fs[R][MAX_SPLITS];
  SB_TRACE_BEGIN();
  pdl_trigger();
  const int split = blockIdx.x, h0 = blockIdx.y * R, b = blockIdx.z;
  const int n_atoms = (a.row + 63) / 64, stage_bytes = n_atoms * ATOM;
  float* sp = (float*)(smem + NS * stage_bytes);       // [SL][R][SP_LD], behind the ring of key tiles
  bf16* pp = (bf16*)(sp + SL * R * SP_LD);             // [2][hi, lo][R][PP_LD]
  float* corr_s = (float*)(pp + 2 * 2 * R * PP_LD);    // [2][R]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tig = lane & 3, mi = lane >> 3, r8 = lane & 7;
  if (threadIdx.x == 0) {
    for (int i = 0; i < NS; i++) mbar_init(smem_u32(&full[i]), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  const uint64_t policy = l2_evict_first_policy();
  // One thread. Rows beyond the chunk are whatever the cache holds there (finite, or zeros beyond its end); their weights are zero.
  auto load_tile = [&](int t, int kb) {
    const uint32_t bar = smem_u32(&full[t & (NS - 1)]), dst = smem_u32(smem) + (uint32_t)((t & (NS - 1)) * stage_bytes);
    mbar_expect_tx(bar, (uint32_t)stage_bytes);
    for (int i = 0; i < n_atoms; i++) tma_load_2d(dst + i * ATOM, &map, i * 64, b * a.maxlen + kb + t * LKT, bar, policy);
  };
  auto range = [&](int len, int& kb, int& ke) {
    const int lo = a.window > 0 ? max(0, len - a.window) : 0;
    kb = lo + split * a.chunk;
    ke = min(len, kb + a.chunk);
  };
  // Tiles that hold rows of earlier steps only are requested before the dependency wait; the length they are derived from is
  // read again after it. (It belongs to the previous step and has not changed; if it had, the sequence would be refused below.)
  int kb, ke;
  const int len_early = min(ld_volatile_i32(a.lens + b) + 1, a.maxlen);
  range(len_early, kb, ke);
  int n_early = 0;
  if (a.prefetch)
    for (; n_early < NS - 2 && kb + (n_early + 1) * LKT <= min(ke, len_early - 1); n_early++)
      if (threadIdx.x == 0) load_tile(n_early, kb);
  pdl_wait();
  SB_TRACE_WAITED();
  const int len = min(ld_volatile_i32(a.lens + b) + 1, a.maxlen);
  bool bad = len != len_early && n_early;
  if (!bad) range(len, kb, ke);
  const int ntiles = kb < ke ? (ke - kb + LKT - 1) / LKT : 0;
  if (threadIdx.x == 0)
    for (int t = n_early; t < min(NS - 2, ntiles); t++) load_tile(t, kb);
  const int ks = warp % SL, kh = warp / SL;
  const int nks = a.row / 16;

  uint32_t qf[MT][KSM][4];
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int k = 0; k < KSM; k++) {
      const int step = ks + SL * k, ha = h0 + m * 16 + g, hb = ha + 8;
      const bf16* q0 = a.q + ((int64_t)b * a.H + ha) * a.row + step * 16 + 2 * tig;
      const bf16* q1 = q0 + 8 * (int64_t)a.row;
      const bool v = step < nks;
      qf[m][k][0] = v && ha < a.H ? *(const uint32_t*)q0 : 0u;
      qf[m][k][1] = v && hb < a.H ? *(const uint32_t*)q1 : 0u;
      qf[m][k][2] = v && ha < a.H ? *(const uint32_t*)(q0 + 8) : 0u;
      qf[m][k][3] = v && hb < a.H ? *(const uint32_t*)(q1 + 8) : 0u;
    }
  float o[MT][NV][4];
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int j = 0; j < NV; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) o[m][j][i] = 0.f;
  constexpr int TPR = NT / R, KPT = LKT / TPR;  // softmax: threads per head row (16 or 32: never across warps), keys per thread
  const int srow = threadIdx.x / TPR, skey = (threadIdx.x % TPR) * KPT;
  float m_run = -INFINITY, l_run = 0.f;
  const int dim0 = warp * NV * 8;
  const bool has_cols = dim0 < a.rank_p;

  float s[MT][2][4];
  // this lane's place in an atom of the key tile: reduction steps ks, ks + SL, .. all lie in the same two 16-byte chunks
  const uint32_t k_lane = smem_u32(smem) + (uint32_t)((ks >> 2) * ATOM + (kh * 16 + (mi >> 1) * 8 + r8) * 128 + ((((ks & 3) * 2 + (mi & 1)) ^ r8) << 4));
  auto scores = [&](int t) {  // into registers
    const uint32_t tile = k_lane + (uint32_t)((t & (NS - 1)) * stage_bytes);
#pragma unroll
    for (int k = 0; k < KSM; k++) {
      if (ks + SL * k < nks) {
        uint32_t kf[4];
        ldsm_x4(tile + (uint32_t)(SL / 4 * k * ATOM), kf);
#pragma unroll
        for (int m = 0; m < MT; m++) {
          if (k == 0) {
            mma_bf16_zero(s[m][0], qf[m][k], kf[0], kf[1]);
            mma_bf16_zero(s[m][1], qf[m][k], kf[2], kf[3]);
          } else {
            mma_bf16(s[m][0], qf[m][k], kf[0], kf[1]);
            mma_bf16(s[m][1], qf[m][k], kf[2], kf[3]);
          }
        }
      } else if (k == 0) {
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
          for (int i = 0; i < 4; i++) s[m][0][i] = s[m][1][i] = 0.f;
      }
    }
  };
  float* const sp_w = sp + (ks * R + g) * SP_LD + kh * 16 + 2 * tig;
  auto store_scores = [&]() {
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int j = 0; j < 2; j++) {
        float* w = sp_w + m * 16 * SP_LD + j * 8;
        *(float2*)w = make_float2(s[m][j][0], s[m][j][1]);
        *(float2*)(w + 8 * SP_LD) = make_float2(s[m][j][2], s[m][j][3]);
      }
  };
  const float* const sp_r = sp + srow * SP_LD + skey;
  float v[KPT];
  auto fetch_scores = [&]() {  // the slices' sums, in slice order
#pragma unroll
    for (int i = 0; i < KPT; i++) v[i] = sp_r[i];
#pragma unroll
    for (int p = 1; p < SL; p++)
#pragma unroll
      for (int i = 0; i < KPT; i++) v[i] += sp_r[p * R * SP_LD + i];
  };
  auto softmax = [&](int t) {
    const int lim = ke - kb - t * LKT;
    float mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < KPT; i++) {
      v[i] = skey + i < lim ? v[i] * a.scale_log2 : -INFINITY;
      mx = fmaxf(mx, v[i]);
    }
#pragma unroll
    for (int off = 1; off < TPR; off <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    const float m_new = fmaxf(m_run, mx);  // finite: every tile holds a visible key
    const float corr = ex2_approx(m_run - m_new);
    m_run = m_new;
    float ls = 0.f;
    bf16* ph = pp + ((t & 1) * 2 * R + srow) * PP_LD + skey;
    if (KPT == 1) {
      const float p0 = ex2_approx(v[0] - m_new), a0 = round_bf16(p0);
      ls = p0;
      ph[0] = __float2bfloat16_rn(a0);
      ph[R * PP_LD] = __float2bfloat16_rn(p0 - a0);
    } else {
#pragma unroll
      for (int i = 0; i + 1 < KPT; i += 2) {
        const float p0 = ex2_approx(v[i] - m_new), p1 = ex2_approx(v[i + 1] - m_new);
        ls += p0 + p1;
        uint32_t hi, lo;
        split_bf16x2(p0, p1, hi, lo);
        *(uint32_t*)(ph + i) = hi;
        *(uint32_t*)(ph + R * PP_LD + i) = lo;
      }
    }
    l_run = l_run * corr + ls;
    if (skey == 0) corr_s[(t & 1) * R + srow] = corr;
  };
  uint32_t v_chunk[NV / 2];  // swizzled place of this lane's 16-byte chunk of the warp's latent columns (all in one atom)
#pragma unroll
  for (int jp = 0; jp < NV / 2; jp++) v_chunk[jp] = (uint32_t)(((((dim0 >> 3) & 7) + jp * 2 + (mi >> 1)) ^ r8) << 4);
  auto accumulate = [&](int t) {
    if (!has_cols) return;
    const float* cs = corr_s + (t & 1) * R;
#pragma unroll
    for (int m = 0; m < MT; m++) {
      const float c0 = cs[m * 16 + g], c1 = cs[m * 16 + g + 8];
      if (!__all_sync(0xffffffffu, c0 == 1.0f && c1 == 1.0f)) {
#pragma unroll
        for (int j = 0; j < NV; j++) { o[m][j][0] *= c0; o[m][j][1] *= c0; o[m][j][2] *= c1; o[m][j][3] *= c1; }
      }
    }
    const uint32_t tile = smem_u32(smem) + (uint32_t)((t & (NS - 1)) * stage_bytes + (dim0 >> 6) * ATOM + ((mi & 1) * 8 + r8) * 128);
    const uint32_t ps = smem_u32(pp + (t & 1) * 2 * R * PP_LD + ((mi & 1) * 8 + r8) * PP_LD + (mi >> 1) * 8);
#pragma unroll
    for (int kk = 0; kk < LKT / 16; kk++) {
      uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
      for (int m = 0; m < MT; m++) {
        ldsm_x4(ps + (uint32_t)((m * 16 * PP_LD + kk * 16) * 2), ph[m]);
        ldsm_x4(ps + (uint32_t)(((R + m * 16) * PP_LD + kk * 16) * 2), pl[m]);
      }
#pragma unroll
      for (int jp = 0; jp < NV / 2; jp++) {
        if (dim0 + jp * 16 < a.rank_p) {
          uint32_t vf[4];
          ldsm_x4_t(tile + (uint32_t)(kk * 16 * 128) + v_chunk[jp], vf);
#pragma unroll
          for (int m = 0; m < MT; m++) {
            mma_bf16(o[m][2 * jp], ph[m], vf[0], vf[1]);
            mma_bf16(o[m][2 * jp + 1], ph[m], vf[2], vf[3]);
          }
#pragma unroll
          for (int m = 0; m < MT; m++) {
            mma_bf16(o[m][2 * jp], pl[m], vf[0], vf[1]);
            mma_bf16(o[m][2 * jp + 1], pl[m], vf[2], vf[3]);
          }
        }
      }
    }
  };
  auto arrived = [&](int t) {  // tile t has landed (bounded)
    if (!mbar_wait(smem_u32(&full[t & (NS - 1)]), (uint32_t)(t / NS) & 1)) bad = true;
  };

  if (ntiles > 0) {
    arrived(0);
    scores(0);
    store_scores();
    for (int t = 0; t <= ntiles; t++) {
      if (t + 1 < ntiles) arrived(t + 1);
      __syncthreads();  // S(t) and P(t-1) of every thread; everyone has left tile t - 2
      if (threadIdx.x == 0 && t + 2 < ntiles) load_tile(t + 2, kb);
      if (t < ntiles) fetch_scores();
      if (t + 1 < ntiles) scores(t + 1);
      __syncthreads();  // everyone has fetched S(t)
      if (t + 1 < ntiles) store_scores();
      if (t < ntiles) softmax(t);
      if (t > 0) accumulate(t - 1);
    }
  }
#pragma unroll
  for (int off = 1; off < TPR; off <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, off);
  __syncthreads();  // the ring is free: it holds this block's sums now
  float* so = (float*)smem;  // [R][rank_p + 4]
  const int so_ld = a.rank_p + 4;
  if (skey == 0) ml_s[srow] = make_float2(m_run, l_run);
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int j = 0; j < NV; j++) {
      const int col = dim0 + j * 8 + 2 * tig;
      if (col < a.rank_p) {
        *(float2*)(so + (m * 16 + g) * so_ld + col) = make_float2(o[m][j][0], o[m][j][1]);
        *(float2*)(so + (m * 16 + g + 8) * so_ld + col) = make_float2(o[m][j][2], o[m][j][3]);
      }
    }
  cluster_sync();
  if (threadIdx.x < R) {
    float2 ml[MAX_SPLITS];
    float M = -INFINITY, L = 0.f;
#pragma unroll
    for (int i = 0; i < MAX_SPLITS; i++)
      if (i < a.nsplit) { ml[i] = ld_cluster2(map_to_rank(smem_u32(&ml_s[threadIdx.x]), i)); M = fmaxf(M, ml[i].x); }
#pragma unroll
    for (int i = 0; i < MAX_SPLITS; i++)
      if (i < a.nsplit) { ml[i].x = ml[i].y > 0.f ? exp2f(ml[i].x - M) : 0.f; L += ml[i].x * ml[i].y; }
    const float inv = 1.0f / L;
#pragma unroll
    for (int i = 0; i < MAX_SPLITS; i++)
      if (i < a.nsplit) fs[threadIdx.x][i] = ml[i].x * inv;
  }
  __syncthreads();
  const int c4n = a.rank_p / 4, heads = min(R, a.H - h0);
  const uint32_t so_a = smem_u32(so);
  for (int i = split * NT + (int)threadIdx.x; i < heads * c4n; i += a.nsplit * NT) {
    const int h = i / c4n, c = (i - h * c4n) * 4;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f), x[MAX_SPLITS];
#pragma unroll
    for (int p = 0; p < MAX_SPLITS; p++)
      if (p < a.nsplit) x[p] = ld_cluster4(map_to_rank(so_a + (uint32_t)((h * so_ld + c) * 4), p));
#pragma unroll
    for (int p = 0; p < MAX_SPLITS; p++)
      if (p < a.nsplit && fs[h][p] != 0.f) {  // a block without keys holds zeros; its weight is zero
        const float w = fs[h][p];
        acc.x += w * x[p].x; acc.y += w * x[p].y; acc.z += w * x[p].z; acc.w += w * x[p].w;
      }
    *(uint2*)(a.out + ((int64_t)b * a.H + h0 + h) * a.rank_p + c) = make_uint2(pack_bf16(acc.x, acc.y), pack_bf16(acc.z, acc.w));
  }
  if (bad && lane == 0) { *(volatile int*)a.status = 17; __threadfence_system(); }
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
// 2D map of a layer's cache rows [rows, row], box = 32 rows x 64 columns (128 bytes), 128-byte swizzle.
int cache_map(CUtensorMap* map, const bf16* base, int64_t rows, int row) {
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
  cuuint32_t box[2] = {64u, (cuuint32_t)LKT};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<bf16*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                      CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return sb_fail(STRICTB200_ERR_CUDA, "cuTensorMapEncodeTiled failed with code " + std::to_string((int)r));
  return STRICTB200_OK;
}

// The kernel's shapes: warps, reduction steps per slice, latent columns per warp. Rows of up to 192 (rank 128), 384 (rank 256)
// and 640 (rank 512) elements.
int decode_shape(const LatentShape& s) {
  const int rp = s.rank_p(), row = s.row();
  return rp <= 128 && row <= 192 ? 0 : rp <= 256 && row <= 384 ? 1 : 2;
}
int decode_warps(const LatentShape& s) { return decode_shape(s) == 0 ? 8 : 16; }

template <int MT, int NW, int KSM, int NV>
int launch_attn_decode(strictb200_ctx* ctx, const CUtensorMap& map, const AttnDecodeDev& a, int B) {
  static size_t have[64] = {};
  const size_t smem = attn_decode_smem(MT, NW, a.row);
  SB_TRY(allow_smem(ctx, latent_attn_decode_kernel<MT, NW, KSM, NV>, smem, have));
  SB_CUDA(sb_launch_cluster(ctx, latent_attn_decode_kernel<MT, NW, KSM, NV>, dim3(a.nsplit, (a.H + MT * 16 - 1) / (MT * 16), B), dim3(NW * 32), smem,
                            dim3(a.nsplit, 1, 1), map, a));
  ctx->launches++;
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
  return s.rank_p() <= 512 && s.row() <= 640 && s.dim <= 512 && decode_in_smem(s.dim) <= (int)SMEM_MAX;
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

// Keys per block: waves of blocks x (key tiles per block + what a block costs besides), over the multiples of the tile that
// leave at most MAX_SPLITS chunks of the window (or of the planned length, where that is shorter). The chunks of a (sequence,
// head group) are one cluster, and clusters of 3, 5, 6 or 7 blocks pack the SMs of a GPC badly: 1, 2, 4 or 8 chunks.
int sb_latent_decode_chunk(strictb200_ctx* ctx, const LatentShape& s, int B, int len_plan) {
  const int n = s.window > 0 ? std::min(s.window, len_plan) : len_plan, tiles = std::max(1, (n + LKT - 1) / LKT);
  const int mt = s.H <= 16 ? 1 : 2;
  const int per_sm = std::max<int>(1, std::min<int>(2, (int)(227 * 1024 / (attn_decode_smem(mt, decode_warps(s), s.row()) + 2048))));
  const int64_t slots = (int64_t)ctx->sm_count * per_sm, pairs = (int64_t)B * ((s.H + mt * 16 - 1) / (mt * 16));
  int best = tiles;
  double best_cost = 1e30;
  for (int k = 1; k <= MAX_SPLITS && k <= tiles; k *= 2) {
    const int c = (tiles + k - 1) / k;
    const int64_t blocks = pairs * k, waves = (blocks + slots - 1) / slots;
    const double cost = (double)waves * (c + 4);
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
  CUtensorMap map;
  SB_TRY(cache_map(&map, cache, (int64_t)B * maxlen, s.row()));
  AttnDecodeDev a{q_abs, lens, s.H, s.row(), s.rank_p(), maxlen, s.window, chunk, nsplit, s.scale * LOG2E, scratch, ctx->opt.attn_prefetch, ctx->d_status};
  const int rp = s.rank_p(), shape = decode_shape(s);
#define LATENT_DECODE(NW, KSM, NV) SB_TRY((s.H <= 16 ? launch_attn_decode<1, NW, KSM, NV>(ctx, map, a, B) : launch_attn_decode<2, NW, KSM, NV>(ctx, map, a, B)))
  if (shape == 0) LATENT_DECODE(8, 3, 2);
  else if (shape == 1) LATENT_DECODE(16, 3, 2);
  else LATENT_DECODE(16, 5, 4);
#undef LATENT_DECODE
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
