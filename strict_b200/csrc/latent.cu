// Latent attention: a position leaves one low-rank vector (the latent, RMS-normed) and one rotated key part that all heads
// share; a head's unrotated key and its value are W_uk c and W_uv c. The cache row of a position is [latent | rotated part],
// each padded with zeros to a multiple of 16 elements, whatever the number of heads.
//
//  * prompts: keys and values are rebuilt per head by one GEMM over the visible latents, then the tcgen05 prefill kernel
//    runs on them (attention_tc.cu). Here: the projection's rows into rotated queries and cache rows.
//  * decode: nothing is rebuilt. A head's query is carried into latent space (q' = q W_uk), so that q' . c replaces
//    q . W_uk c, all heads read the same cache row (the heads are the rows of the MMA tile) and the weighted sum of latents
//    goes through W_uv once per head. Three launches: queries into latent space beside everything else the projection
//    feeds (rotation, cache append, activation); split-key attention; merge of the key chunks + W_uv.
//  * any other width, and fp32: one block per row and head, straight from the cache.
//
// Scores, softmax weights, norms and rotations are fp32; the weights enter the product with the latents as two bf16 terms
// (hi + lo), whose sum carries 16 mantissa bits.
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
__device__ __forceinline__ void ldsm_x2_t(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
// not volatile: the compiler may move fragment loads ahead of products that do not need them
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
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
  int n_rt, n_grp;      // latent tiles of 64 and token groups of 16: blocks of the first role
  int rot_blocks;       // blocks per token of the rotation (256 pairs each)
  int act_blocks;       // ... and of the activation
};
constexpr int QA_COLS = 64, QA_LD = QA_COLS + 8;
__host__ __device__ inline int decode_in_smem(int dim) {
  const int d16 = (dim + 15) & ~15;
  return d16 * QA_LD * 2 + 16 * (d16 + 8) * 2;
}
// One launch, four roles by block index: H * n_rt * n_grp blocks multiply queries with W_uk (64 latents of one head, 16
// tokens), then B * rot_blocks rotate the queries' second part, B append the cache row (a layer with latents of its own),
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
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k = 0; k < d16; k += 16) {
      uint32_t qa[4], wb[2];
      ldsm_x4(smem_u32(qt + ((mi & 1) * 8 + r8) * (d16 + 8) + k + (mi >> 1) * 8), qa);
      ldsm_x2_t(smem_u32(wt + (k + (mi & 1) * 8 + r8) * QA_LD + warp * 8), wb);
      mma_bf16(acc, qa, wb[0], wb[1]);
    }
    const int g = lane >> 2, col = r0 + warp * 8 + 2 * (lane & 3);
    if (col < a.rank_p) {
      if (b0 + g < B) *(uint32_t*)(d.q_abs + ((int64_t)(b0 + g) * a.H + h) * a.row + col) = pack_bf16(acc[0], acc[1]);
      if (b0 + g + 8 < B) *(uint32_t*)(d.q_abs + ((int64_t)(b0 + g + 8) * a.H + h) * a.row + col) = pack_bf16(acc[2], acc[3]);
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
// grid (nsplit, ceil(H / (16 MT)), B), 256 threads. Rows of the MMA tiles = up to 16 MT heads, 32 keys per step. Three
// products of three different steps share an iteration, so one barrier per step is enough:
//   S(t+1) partials  warp (ks, kh): reduction steps ks, ks + 4, .. of the cache row for the 16 keys of half kh; its share of
//                    the queries stays in registers for the whole block, so a step reads the key tile from shared memory once
//   softmax(t)       the four partial scores of a (head, key) are added in slice order; running maximum and sum per head
//   O += P(t-1) c    every warp owns 8 NV latent columns of all heads; the key tile is its operand again
// Key tiles pass through a ring of NS stages (t-1, t, t+1 in use, the rest in flight).
constexpr int LKT = 32;
struct AttnDecodeDev {
  const bf16* q;
  const bf16* cache;
  const int32_t* lens;
  int H, row, rank_p, maxlen, window, chunk, nsplit;
  float scale_log2;
  float* o_part;
  float* ml_part;
  int prefetch;
};
constexpr int SP_LD = 36, PP_LD = 40;  // row strides of the score (fp32) and weight (bf16) tiles
constexpr int decode_stages(int ksm) { return ksm > 5 ? 4 : 6; }
constexpr size_t attn_decode_smem(int mt, int ksm, int row) {
  return (size_t)decode_stages(ksm) * LKT * (row * 2 + 16) + (size_t)2 * 4 * mt * 16 * SP_LD * 4 + (size_t)2 * 2 * mt * 16 * PP_LD * 2 + 2 * mt * 16 * 4;
}

template <int MT, int KSM, int NV>
__global__ void __launch_bounds__(256) latent_attn_decode_kernel(AttnDecodeDev a) {
  constexpr int NS = decode_stages(KSM), R = MT * 16;
  extern __shared__ __align__(128) uint8_t smem[];
  SB_TRACE_BEGIN();
  pdl_trigger();
  const int split = blockIdx.x, h0 = blockIdx.y * R, b = blockIdx.z;
  const int RS = a.row * 2 + 16;  // shared-memory row stride: an odd number of 16-byte chunks
  uint8_t* tiles = smem;                               // [NS][LKT][RS]
  float* sp = (float*)(smem + NS * LKT * RS);          // [2][4][R][SP_LD]
  bf16* pp = (bf16*)(sp + 2 * 4 * R * SP_LD);          // [2][hi, lo][R][PP_LD]
  float* corr_s = (float*)(pp + 2 * 2 * R * PP_LD);    // [2][R]
  const bf16* base = a.cache + (int64_t)b * a.maxlen * a.row;
  const int cpr = a.row / 8;  // 16-byte chunks per row
  const int ld_r = (int)threadIdx.x / cpr, ld_c = (int)threadIdx.x % cpr, st_r = 256 / cpr, st_c = 256 % cpr;
  auto load_tile = [&](int stage, int key0, int n) {
    const uint32_t dst = smem_u32(tiles + stage * LKT * RS);
    for (int r = ld_r, c = ld_c; r < LKT;) {
      const bool ok = r < n;
      cp_async16(dst + r * RS + c * 16, base + (int64_t)(key0 + (ok ? r : 0)) * a.row + c * 8, ok);
      r += st_r;
      c += st_c;
      if (c >= cpr) { c -= cpr; r++; }
    }
  };
  auto range = [&](int len, int& kb, int& ke) {
    const int lo = a.window > 0 ? max(0, len - a.window) : 0;
    kb = lo + split * a.chunk;
    ke = min(len, kb + a.chunk);
  };
  // Tiles that hold rows of earlier steps only are requested before the dependency wait; the length they are derived from is
  // read again after it.
  int kb, ke;
  const int len_early = min(ld_volatile_i32(a.lens + b) + 1, a.maxlen);
  range(len_early, kb, ke);
  int n_early = 0;
  if (a.prefetch)
    for (; n_early < NS - 2 && kb + (n_early + 1) * LKT <= min(ke, len_early - 1); n_early++) { load_tile(n_early, kb + n_early * LKT, LKT); cp_async_commit(); }
  pdl_wait();
  SB_TRACE_WAITED();
  const int len = min(ld_volatile_i32(a.lens + b) + 1, a.maxlen);
  if (len != len_early && n_early) {  // not expected: the length belongs to the previous step
    cp_async_wait<0>();
    __syncthreads();
    n_early = 0;
  }
  range(len, kb, ke);
  if (kb >= ke) return;
  const int ntiles = (ke - kb + LKT - 1) / LKT;
  for (int t = n_early; t < NS - 2; t++) {  // one group per tile, empty beyond the last
    if (t < ntiles) load_tile(t, kb + t * LKT, min(LKT, ke - kb - t * LKT));
    cp_async_commit();
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tig = lane & 3, mi = lane >> 3, r8 = lane & 7;
  const int ks = warp & 3, kh = warp >> 2;
  const int nks = a.row / 16;

  uint32_t qf[MT][KSM][4];
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int k = 0; k < KSM; k++) {
      const int step = ks + 4 * k, ha = h0 + m * 16 + g, hb = ha + 8;
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
  constexpr int TPR = 256 / R, KPT = LKT / TPR;  // softmax: threads per head row, keys per thread (2 or 4)
  const int srow = threadIdx.x / TPR, skey = (threadIdx.x % TPR) * KPT;
  float m_run = -INFINITY, l_run = 0.f;
  const int dim0 = warp * NV * 8;

  auto scores = [&](int t) {
    const uint32_t tile = smem_u32(tiles + (t % NS) * LKT * RS) + (uint32_t)((kh * 16 + (mi >> 1) * 8 + r8) * RS + (mi & 1) * 16);
    float s[MT][2][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int j = 0; j < 2; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) s[m][j][i] = 0.f;
#pragma unroll
    for (int k = 0; k < KSM; k++) {
      const int step = ks + 4 * k;
      if (step < nks) {
        uint32_t kf[4];
        ldsm_x4(tile + (uint32_t)(step * 32), kf);
#pragma unroll
        for (int m = 0; m < MT; m++) {
          mma_bf16(s[m][0], qf[m][k], kf[0], kf[1]);
          mma_bf16(s[m][1], qf[m][k], kf[2], kf[3]);
        }
      }
    }
    float* w0 = sp + (((t & 1) * 4 + ks) * R + g) * SP_LD + kh * 16 + 2 * tig;
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int j = 0; j < 2; j++) {
        float* w = w0 + m * 16 * SP_LD + j * 8;
        *(float2*)w = make_float2(s[m][j][0], s[m][j][1]);
        *(float2*)(w + 8 * SP_LD) = make_float2(s[m][j][2], s[m][j][3]);
      }
  };
  auto softmax = [&](int t) {
    float v[KPT];
    const float* sr = sp + ((t & 1) * 4 * R + srow) * SP_LD + skey;
#pragma unroll
    for (int i = 0; i < KPT; i += 2) {
      float2 x[4];
#pragma unroll
      for (int p = 0; p < 4; p++) x[p] = *(const float2*)(sr + p * R * SP_LD + i);
      v[i] = ((x[0].x + x[1].x) + x[2].x) + x[3].x;
      v[i + 1] = ((x[0].y + x[1].y) + x[2].y) + x[3].y;
    }
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
    const float corr = exp2f(m_run - m_new);
    m_run = m_new;
    float ls = 0.f;
    bf16* ph = pp + ((t & 1) * 2 * R + srow) * PP_LD + skey;
#pragma unroll
    for (int i = 0; i < KPT; i += 2) {
      const float p0 = exp2f(v[i] - m_new), p1 = exp2f(v[i + 1] - m_new);
      ls += p0 + p1;
      const float a0 = round_bf16(p0), a1 = round_bf16(p1);
      *(uint32_t*)(ph + i) = pack_bf16(a0, a1);
      *(uint32_t*)(ph + R * PP_LD + i) = pack_bf16(p0 - a0, p1 - a1);
    }
    l_run = l_run * corr + ls;
    if (skey == 0) corr_s[(t & 1) * R + srow] = corr;
  };
  auto accumulate = [&](int t) {
    if (dim0 >= a.rank_p) return;
    const float* cs = corr_s + (t & 1) * R;
#pragma unroll
    for (int m = 0; m < MT; m++) {
      const float c0 = cs[m * 16 + g], c1 = cs[m * 16 + g + 8];
      if (!__all_sync(0xffffffffu, c0 == 1.0f && c1 == 1.0f)) {
#pragma unroll
        for (int j = 0; j < NV; j++) { o[m][j][0] *= c0; o[m][j][1] *= c0; o[m][j][2] *= c1; o[m][j][3] *= c1; }
      }
    }
    const uint32_t tile = smem_u32(tiles + (t % NS) * LKT * RS) + (uint32_t)(((mi & 1) * 8 + r8) * RS + (dim0 + (mi >> 1) * 8) * 2);
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
          ldsm_x4_t(tile + (uint32_t)(kk * 16 * RS + jp * 32), vf);
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

  cp_async_wait<NS - 3>();
  __syncthreads();
  scores(0);
  for (int t = 0; t <= ntiles; t++) {
    cp_async_wait<NS - 4>();  // tile t + 1 has landed
    __syncthreads();          // S(t), P(t-1) and tile t + 1 of every thread; everyone has left tile t - 2
    const int next = t + NS - 2;
    if (next < ntiles) load_tile(next % NS, kb + next * LKT, min(LKT, ke - kb - next * LKT));
    cp_async_commit();
    if (t + 1 < ntiles) scores(t + 1);
    if (t < ntiles) softmax(t);
    if (t > 0) accumulate(t - 1);
  }
#pragma unroll
  for (int off = 1; off < TPR; off <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, off);
  if (skey == 0 && h0 + srow < a.H) *(float2*)(a.ml_part + (((int64_t)b * a.H + h0 + srow) * a.nsplit + split) * 2) = make_float2(m_run, l_run);
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int j = 0; j < NV; j++) {
      const int col = dim0 + j * 8 + 2 * tig, ha = h0 + m * 16 + g;
      if (col < a.rank_p) {
        if (ha < a.H) *(float2*)(a.o_part + (((int64_t)b * a.H + ha) * a.nsplit + split) * a.rank_p + col) = make_float2(o[m][j][0], o[m][j][1]);
        if (ha + 8 < a.H) *(float2*)(a.o_part + (((int64_t)b * a.H + ha + 8) * a.nsplit + split) * a.rank_p + col) = make_float2(o[m][j][2], o[m][j][3]);
      }
    }
  SB_TRACE_END(SB_K_ATTN, 0);
}

// grid (H, ceil(vdim / 64), ceil(B / 16)), 256 threads: merges the key chunks of one head for 16 tokens, then its 64 value
// columns from W_uv (a constant, requested before the dependency wait).
constexpr int MAX_SPLITS = 16;
struct MergeDev {
  const float* o_part;
  const float* ml_part;
  const int32_t* lens;
  int B, H, rank_p, vdim, window, maxlen, chunk, nsplit;
  const bf16* wv;   // value rows: head h, value v at (h * kv_head + v) * rank_p
  int kv_head;
  bf16* out;
  int64_t ldo;
};
__global__ void __launch_bounds__(256) latent_merge_kernel(MergeDev a) {
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float fs[16][MAX_SPLITS];
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
  cp_async_commit();
  pdl_wait();
  SB_TRACE_WAITED();
  {
    const int m = threadIdx.x >> 4, l16 = threadIdx.x & 15, b = b0 + m;
    const int len = b < a.B ? min(a.lens[b] + 1, a.maxlen) : 0;
    const int n = a.window > 0 ? min(len, a.window) : len, ns = (n + a.chunk - 1) / a.chunk;
    const int64_t base = ((int64_t)(b < a.B ? b : 0) * a.H + h) * a.nsplit;
    float2 ml = l16 < ns ? *(const float2*)(a.ml_part + (base + l16) * 2) : make_float2(-INFINITY, 0.f);
    float M = ml.x;
#pragma unroll
    for (int off = 1; off < 16; off <<= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, off));
    float f = l16 < ns ? exp2f(ml.x - M) : 0.f, L = f * ml.y;
#pragma unroll
    for (int off = 1; off < 16; off <<= 1) L += __shfl_xor_sync(0xffffffffu, L, off);
    fs[m][l16] = l16 < ns ? f / L : 0.f;
  }
  __syncthreads();
  // every thread of the block takes groups of four columns of any of the tokens; all chunks' loads of a group in flight at once
  const int c4n = a.rank_p / 4;
#pragma unroll 2
  for (int i = threadIdx.x; i < 16 * c4n; i += 256) {
    const int m = i / c4n, c = (i - m * c4n) * 4, b = b0 + m;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (b < a.B) {
      const float* src = a.o_part + (((int64_t)b * a.H + h) * a.nsplit) * a.rank_p + c;
      for (int s0 = 0; s0 < a.nsplit; s0 += 8) {
        float4 x[8];
#pragma unroll
        for (int s = 0; s < 8; s++)
          if (s0 + s < a.nsplit && fs[m][s0 + s] != 0.f) x[s] = *(const float4*)(src + (int64_t)(s0 + s) * a.rank_p);
#pragma unroll
        for (int s = 0; s < 8; s++)
          if (s0 + s < a.nsplit && fs[m][s0 + s] != 0.f) {
            const float w = fs[m][s0 + s];
            acc.x += w * x[s].x; acc.y += w * x[s].y; acc.z += w * x[s].z; acc.w += w * x[s].w;
          }
      }
    }
    *(uint2*)(ot + m * ld + c) = make_uint2(pack_bf16(acc.x, acc.y), pack_bf16(acc.z, acc.w));
  }
  cp_async_wait<0>();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mi = lane >> 3, r8 = lane & 7;
  float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
  for (int k = 0; k < a.rank_p; k += 16) {
    uint32_t oa[4], wb[2];
    ldsm_x4(smem_u32(ot + ((mi & 1) * 8 + r8) * ld + k + (mi >> 1) * 8), oa);
    ldsm_x2(smem_u32(wt + (warp * 8 + r8) * ld + k + (mi & 1) * 8), wb);
    mma_bf16(acc[(k >> 4) & 1], oa, wb[0], wb[1]);
  }
  const int g = lane >> 2, v = v0 + warp * 8 + 2 * (lane & 3);
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int b = b0 + g + (i >> 1) * 8, vc = v + (i & 1);
    if (b < a.B && vc < a.vdim) a.out[(int64_t)b * a.ldo + (int64_t)h * a.vdim + vc] = __float2bfloat16_rn(acc[0][i] + acc[1][i]);
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
  if (bytes > 48 * 1024 && bytes > h) {
    SB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    h = bytes;
  }
  return STRICTB200_OK;
}
constexpr size_t SMEM_MAX = 227 * 1024 - 1024;  // what a block may take, less the kernels' static share

template <int MT, int KSM, int NV>
int launch_attn_decode(strictb200_ctx* ctx, const AttnDecodeDev& a, int B) {
  static size_t have[64] = {};
  const size_t smem = attn_decode_smem(MT, KSM, a.row);
  SB_TRY(allow_smem(ctx, latent_attn_decode_kernel<MT, KSM, NV>, smem, have));
  SB_CUDA(sb_launch(ctx, latent_attn_decode_kernel<MT, KSM, NV>, dim3(a.nsplit, (a.H + MT * 16 - 1) / (MT * 16), B), dim3(256), smem, a));
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
  return s.rank_p() <= 512 && s.row() <= 576 && decode_in_smem(s.dim) <= (int)SMEM_MAX && s.dim <= 512;
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

// Reduction steps per slice the kernel is built for: rows of up to 192, 320 and 576 elements.
int decode_ksm(const LatentShape& s) {
  const int nks = (s.row() / 16 + 3) / 4;
  return s.rank_p() <= 128 && nks <= 3 ? 3 : s.rank_p() <= 256 && nks <= 5 ? 5 : 9;
}

// Keys per block: waves of blocks x (key tiles per block + what a block costs besides), over the multiples of the tile that
// leave at most MAX_SPLITS chunks of the window (or of the planned length, where that is shorter).
int sb_latent_decode_chunk(strictb200_ctx* ctx, const LatentShape& s, int B, int len_plan) {
  const int n = s.window > 0 ? std::min(s.window, len_plan) : len_plan, tiles = std::max(1, (n + LKT - 1) / LKT);
  const int mt = s.H <= 16 ? 1 : 2;
  const int per_sm = std::max<int>(1, std::min<int>(2, (int)(227 * 1024 / (attn_decode_smem(mt, decode_ksm(s), s.row()) + 1024))));
  const int64_t slots = (int64_t)ctx->sm_count * per_sm, pairs = (int64_t)B * ((s.H + mt * 16 - 1) / (mt * 16));
  int best = tiles;
  double best_cost = 1e30;
  for (int c = (tiles + MAX_SPLITS - 1) / MAX_SPLITS; c <= tiles; c++) {
    const int64_t blocks = pairs * ((tiles + c - 1) / c), waves = (blocks + slots - 1) / slots;
    const double cost = (double)waves * (c + 3) + 0.05 * ((tiles + c - 1) / c);  // every chunk adds to the merge
    if (cost < best_cost - 1e-9) { best_cost = cost; best = c; }
  }
  return best * LKT;
}
size_t sb_latent_decode_scratch(const LatentShape& s, int B) { return (size_t)B * s.H * MAX_SPLITS * (s.rank_p() + 2) * sizeof(float); }

int k_latent_attn_decode(strictb200_ctx* ctx, const LatentShape& s, const bf16* q_abs, const bf16* cache, const int32_t* lens, int B, int maxlen, int chunk,
                         int nsplit, float* scratch, const bf16* wkv, bf16* out, int64_t ldo) {
  if (!sb_latent_decode_fits(s)) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "latent decode attention: rows too wide for the tensor-core kernel");
  if (nsplit < 1 || nsplit > MAX_SPLITS || chunk < LKT || chunk % LKT || B > 65535) return sb_fail(STRICTB200_ERR_INVALID_ARG, "latent decode attention: bad key chunks");
  float* ml = scratch + (size_t)B * s.H * nsplit * s.rank_p();
  AttnDecodeDev a{q_abs, cache, lens, s.H, s.row(), s.rank_p(), maxlen, s.window, chunk, nsplit, s.scale * LOG2E, scratch, ml, ctx->opt.attn_prefetch};
  const int rp = s.rank_p(), ksm = decode_ksm(s);
#define LATENT_DECODE(KSM, NV) SB_TRY((s.H <= 16 ? launch_attn_decode<1, KSM, NV>(ctx, a, B) : launch_attn_decode<2, KSM, NV>(ctx, a, B)))
  if (ksm == 3) LATENT_DECODE(3, 2);
  else if (ksm == 5) LATENT_DECODE(5, 4);
  else LATENT_DECODE(9, 8);
#undef LATENT_DECODE
  sb_prof_split(ctx, STRICTB200_K_ATTN_MERGE);
  static size_t have[64] = {};
  const size_t smem = (size_t)(64 + 16) * (rp + 8) * 2;
  SB_TRY(allow_smem(ctx, latent_merge_kernel, smem, have));
  MergeDev m{scratch, ml, lens, B, s.H, rp, s.vdim, s.window, maxlen, chunk, nsplit, wkv + (int64_t)s.H * s.kv_head() * rp, s.kv_head(), out, ldo};
  SB_CUDA(sb_launch(ctx, latent_merge_kernel, dim3(s.H, (s.vdim + 63) / 64, (B + 15) / 16), dim3(256), smem, m));
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
