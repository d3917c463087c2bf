// Softmax attention over grouped heads of any width: query/key dims and value dims may differ, the rotation may cover part of a
// head, rotated queries and keys may be divided by their root mean square, the softmax may have a sink (one more key of score 0
// in the denominator, without a value), and a head's output may be multiplied by a sigmoid gate.
//
//  * k_head_split: the projection's rows become rotated queries and cache rows (or dense rows, for retention), beside the
//    feed-forward's activation in a decode step. One warp per head.
//  * attention itself: prompts on the tcgen05 kernel (attention_tc.cu), decode on the split-key kernel (attention.cu) with the
//    merge here, both for heads of up to 128 dims; k_head_attn_any for any width and for fp32.
// Norms, rotations, scores, softmax weights and gates are fp32.
#include "mixers.cuh"

using namespace mix;

namespace {

// One head of four dims per lane (widths multiples of 4, at most 128; so is the rotated half): rotation, norm, factor. c and d are
// this lane's cosines, and its sines with the sign of its half; src the lane that holds the other half of its pairs.
__device__ __forceinline__ float4 rotate_head(const HeadShape& s, float4 x, const float4& c, const float4& d, int src, float post, float eps, int lane) {
  float4 o;
  o.x = __shfl_sync(0xffffffffu, x.x, src); o.y = __shfl_sync(0xffffffffu, x.y, src);
  o.z = __shfl_sync(0xffffffffu, x.z, src); o.w = __shfl_sync(0xffffffffu, x.w, src);
  if (lane * 4 < s.rot) {
    x.x = fmaf(x.x, c.x, o.x * d.x); x.y = fmaf(x.y, c.y, o.y * d.y);
    x.z = fmaf(x.z, c.z, o.z * d.z); x.w = fmaf(x.w, c.w, o.w * d.w);
  }
  float r = post;
  if (s.qk_norm) {
    const float ss = warp_sum(x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w);
    r *= __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)s.dim), eps)));
  }
  return make_float4(x.x * r, x.y * r, x.z * r, x.w * r);
}
__device__ __forceinline__ void lane_angles(const HeadSplitArgs& a, int p, int lane, float4* c, float4* d, int* src) {
  const int e = lane * 4, half = a.s.rot / 2;
  *src = (e < half ? lane + half / 4 : lane - half / 4) & 31;
  *c = *d = make_float4(0.f, 0.f, 0.f, 0.f);
  if (e < a.s.rot) {
    const int64_t i = (int64_t)p * half + (e < half ? e : e - half);
    *c = *(const float4*)(a.cos_t + i);
    *d = *(const float4*)(a.sin_t + i);
    if (e < half) *d = make_float4(-d->x, -d->y, -d->z, -d->w);
  }
}
// any width: one head through shared memory
template <typename T>
__device__ __forceinline__ void head_any(const HeadSplitArgs& a, int64_t rows, int64_t t, int64_t col, int n, bool is_v, float post, int p, T* dst, float* buf, int lane) {
  const HeadShape& s = a.s;
  const int half = s.rot / 2, row = s.row();
  const float *cs = a.cos_t + (int64_t)p * half, *sn = a.sin_t + (int64_t)p * half;
  for (int e = lane; e < n; e += 32) buf[e] = proj(a.p, rows, t, col + e);
  __syncwarp();
  auto value = [&](int e) {
    if (is_v || e >= s.rot) return buf[e];
    const int i = e < half ? e : e - half;
    return e < half ? buf[e] * cs[i] - buf[e + half] * sn[i] : buf[e] * cs[i] + buf[e - half] * sn[i];
  };
  float r = post;
  if (s.qk_norm && !is_v) {
    float ss = 0.f;
    for (int e = lane; e < n; e += 32) { const float v = value(e); ss += v * v; }
    r *= __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(warp_sum(ss), (float)s.dim), a.eps)));
  }
  for (int e = lane; e < row; e += 32) dst[e] = to_t<T>(e < n ? value(e) * r : 0.f);
}

// grid rows * (item blocks + activation blocks), 256 threads: warp w of an item block owns item 8 * block + w of the row: a query
// head, a key head, a value head, or (the last item) all gates. For decode steps and any widths.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) head_split_kernel(HeadSplitArgs a, int64_t rows, int item_blocks, int act_blks) {
  extern __shared__ float sm[];
  SB_TRACE_BEGIN();
  pdl_trigger();
  const int per_row = item_blocks + act_blks;
  const int64_t t = blockIdx.x / per_row;
  const int blk = blockIdx.x % per_row;
  const HeadShape& s = a.s;
  pdl_wait();
  SB_TRACE_WAITED();
  if (blk >= item_blocks) {
    act_block<T>(a.act, a.p, rows, t, blk - item_blocks);
  } else {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_heads = s.H + 2 * s.G, item = blk * 8 + warp;
    const int b = a.seq ? a.seq[t] : (int)t, p = a.pos ? a.pos[t] : a.lens[b];
    const int row = s.row();
    if (p >= 0 && p < a.max_pos && (a.dense || p < a.maxlen)) {  // the host validates; never index outside the cache
      if (item < n_heads) {
        const bool is_q = item < s.H, is_v = item >= s.H + s.G;
        const int h = is_q ? item : is_v ? item - s.H - s.G : item - s.H, n = is_v ? s.vdim : s.dim;
        const int64_t col = is_v ? (int64_t)(s.H + s.G) * s.dim + (int64_t)h * s.vdim : (int64_t)item * s.dim;
        T* dst = is_q ? (T*)a.q_out + (t * s.H + h) * row
                      : (T*)(is_v ? a.v_out : a.k_out) + (a.dense ? (t * s.G + h) * row : (((int64_t)b * s.G + h) * a.maxlen + p) * row);
        const float post = is_q ? 1.f : s.k_scale;
        if constexpr (VEC) {
          float4 x = make_float4(0.f, 0.f, 0.f, 0.f), c, d;
          int src;
          if (lane * 4 < n) x = proj4(a.p, rows, t, col + lane * 4);
          if (!is_v) {
            lane_angles(a, p, lane, &c, &d, &src);
            x = rotate_head(s, x, c, d, src, post, a.eps, lane);
          }
          if (lane * 4 < row) store4<T>(dst + lane * 4, x);
        } else {
          head_any<T>(a, rows, t, col, n, is_v, is_v ? 1.f : post, p, dst, sm + warp * max(s.dim, s.vdim), lane);
        }
      } else if (item == n_heads && s.gate) {
        const int64_t col = (int64_t)(s.H + s.G) * s.dim + (int64_t)s.G * s.vdim;
        for (int h = lane; h < s.H; h += 32) a.gate_out[t * s.H + h] = sigmoid(proj(a.p, rows, t, col + h));
      }
    }
  }
  SB_TRACE_END(SB_K_ROPE, 0);
}

// Prompt rows of a finished projection, four dims per lane: one block per row, a warp walks every eighth head with four heads'
// loads in flight.
template <typename T>
__device__ __forceinline__ void walk_heads(const HeadShape& s, const float* in, int n, int heads, int warp, int lane, bool rotated, const float4& c, const float4& d,
                                           int src, float post, float eps, T* dst, int64_t stride) {
  const int row = s.row(), e = lane * 4;
  for (int h0 = warp; h0 < heads; h0 += 32) {
    float4 x[4];
#pragma unroll
    for (int i = 0; i < 4; i++) {
      x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (h0 + 8 * i < heads && e < n) x[i] = __ldcs((const float4*)(in + (h0 + 8 * i) * n + e));
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int h = h0 + 8 * i;
      if (h >= heads) break;
      if (rotated) x[i] = rotate_head(s, x[i], c, d, src, post, eps, lane);
      if (e < row) store4<T>(dst + h * stride + e, x[i]);
    }
  }
}
template <typename T>
__global__ void __launch_bounds__(256) head_rows_kernel(HeadSplitArgs a) {
  const HeadShape& s = a.s;
  const int64_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = s.row();
  pdl_trigger();
  pdl_wait();
  const int b = a.seq[t], p = a.pos[t];
  if (p < 0 || p >= a.max_pos || (!a.dense && p >= a.maxlen)) return;
  float4 c, d;
  int src;
  lane_angles(a, p, lane, &c, &d, &src);
  const float* in = a.p.in + t * a.p.ld;
  const int64_t at = a.dense ? t * s.G * row : ((int64_t)b * s.G * a.maxlen + p) * row, stride = a.dense ? row : (int64_t)a.maxlen * row;
  walk_heads<T>(s, in, s.dim, s.H, warp, lane, true, c, d, src, 1.f, a.eps, (T*)a.q_out + t * s.H * row, (int64_t)row);
  walk_heads<T>(s, in + s.H * s.dim, s.dim, s.G, warp, lane, true, c, d, src, s.k_scale, a.eps, (T*)a.k_out + at, stride);
  walk_heads<T>(s, in + (s.H + s.G) * s.dim, s.vdim, s.G, warp, lane, false, c, d, src, 1.f, a.eps, (T*)a.v_out + at, stride);
  if (s.gate)
    for (int h = threadIdx.x; h < s.H; h += 256) a.gate_out[t * s.H + h] = sigmoid(in[(s.H + s.G) * s.dim + s.G * s.vdim + h]);
}

template <typename T>
__global__ void __launch_bounds__(256) act_rows_kernel(ProjRows p, ActArgs a, int64_t rows, int blocks) {
  pdl_trigger();
  pdl_wait();
  act_block<T>(a, p, rows, blockIdx.x / blocks, blockIdx.x % blocks);
}

// grid (H, T), 256 threads; 256 keys per step, fp32 arithmetic throughout.
template <typename T>
__global__ void __launch_bounds__(256) head_attn_any_kernel(HeadShape s, const T* __restrict__ q, const T* __restrict__ kc, const T* __restrict__ vc,
                                                            const float* __restrict__ gate, const int32_t* __restrict__ seq, const int32_t* __restrict__ pos,
                                                            const int32_t* __restrict__ lens, int maxlen, T* __restrict__ out, int64_t ldo) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int64_t t = blockIdx.y;
  const int b = seq ? seq[t] : (int)t, p = pos ? pos[t] : lens[b];
  if (p < 0 || p >= maxlen) return;
  const int row = s.row();
  float* qs = sm;               // [dim]
  float* ol = qs + s.dim;       // [vdim]
  float* sc = ol + s.vdim;      // [256]
  float* pv = sc + 256;         // [256] partial sums of the value columns
  const int64_t base = ((int64_t)b * s.G + h / (s.H / s.G)) * maxlen * row;
  for (int i = tid; i < s.dim; i += 256) qs[i] = to_f(q[(t * s.H + h) * row + i]);
  for (int i = tid; i < s.vdim; i += 256) ol[i] = 0.f;
  __syncthreads();
  // the sink is a key of score 0 that was seen first
  float m_run = s.sink ? 0.f : -INFINITY, l_run = s.sink ? 1.f : 0.f;
  const int parts = s.vdim <= 256 ? 256 / s.vdim : 1;  // threads that share a value column
  for (int k0 = 0; k0 <= p; k0 += 256) {
    const int n = min(256, p + 1 - k0);
    for (int j = warp; j < n; j += 8) {
      const T* c = kc + base + (int64_t)(k0 + j) * row;
      float acc = 0.f;
      for (int r = lane; r < s.dim; r += 32) acc += qs[r] * to_f(c[r]);
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
    for (int v0 = 0; v0 < s.vdim; v0 += 256) {
      const int v = parts > 1 ? tid % s.vdim : v0 + tid, part = parts > 1 ? tid / s.vdim : 0;
      float acc = 0.f;
      if (v < s.vdim && part < parts)
        for (int j = part; j < n; j += parts) acc += sc[j] * to_f(vc[base + (int64_t)(k0 + j) * row + v]);
      if (parts > 1) {
        pv[tid] = acc;
        __syncthreads();
        if (part == 0) {
          for (int i = 1; i < parts; i++) acc += pv[i * s.vdim + v];
          ol[v] = ol[v] * corr + acc;
        }
      } else if (v < s.vdim) {
        ol[v] = ol[v] * corr + acc;
      }
    }
    __syncthreads();
  }
  const float inv = (gate ? gate[t * s.H + h] : 1.f) / l_run;
  for (int v = tid; v < s.vdim; v += 256) out[t * ldo + (int64_t)h * s.vdim + v] = to_t<T>(ol[v] * inv);
}

// grid (B, heads in groups of 8), 256 threads: a warp merges the key chunks of one head (at most 8), a lane owns HD / 32 dims.
template <int HD>
__global__ void __launch_bounds__(256) head_combine_kernel(HeadShape s, const float* __restrict__ o_part, const float* __restrict__ ml_part,
                                                           const float* __restrict__ gate, const int32_t* __restrict__ lens, int maxlen, int chunk, int nsplit,
                                                           bf16* __restrict__ out, int64_t ldo) {
  constexpr int PER = HD / 32;
  SB_TRACE_BEGIN();
  pdl_trigger();
  pdl_wait();
  SB_TRACE_WAITED();
  const int b = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h < s.H) {
    const int64_t base = ((int64_t)b * s.H + h) * nsplit;
    float o[8][PER];
    float2 ml[8];
    // slots of chunks beyond the length hold stale data and stay out of the arithmetic
#pragma unroll
    for (int i = 0; i < 8; i++)
      if (i < nsplit) {
        ml[i] = *(const float2*)(ml_part + (base + i) * 2);
#pragma unroll
        for (int j = 0; j < PER; j++) o[i][j] = o_part[(base + i) * HD + lane * PER + j];
      }
    const int ns = (min(lens[b] + 1, maxlen) + chunk - 1) / chunk;
    float M = s.sink ? 0.f : -INFINITY;
#pragma unroll
    for (int i = 0; i < 8; i++)
      if (i < ns) M = fmaxf(M, ml[i].x);
    float L = s.sink ? exp2f(-M) : 0.f, O[PER];
#pragma unroll
    for (int j = 0; j < PER; j++) O[j] = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++)
      if (i < ns) {
        const float f = exp2f(ml[i].x - M);
        L += ml[i].y * f;
#pragma unroll
        for (int j = 0; j < PER; j++) O[j] += o[i][j] * f;
      }
    const float inv = (gate ? gate[(int64_t)b * s.H + h] : 1.f) / L;
    bf16* dst = out + b * ldo + (int64_t)h * s.vdim;
#pragma unroll
    for (int j = 0; j < PER; j++)
      if (lane * PER + j < s.vdim) dst[lane * PER + j] = __float2bfloat16_rn(O[j] * inv);
  }
  SB_TRACE_END(SB_K_COMBINE, 0);
}

}  // namespace

SB_TRACE_TU(heads)

int k_head_split(strictb200_ctx* ctx, const HeadSplitArgs& a, int64_t T) {
  const HeadShape& s = a.s;
  const int items = s.H + 2 * s.G + (s.gate ? 1 : 0), act_blks = act_blocks(a.act);
  const bool vec = s.dim <= 128 && s.vdim <= 128 && ((s.dim | s.vdim | (s.rot / 2) | (int)(a.p.ld & 3)) & 3) == 0;
  if (vec && a.seq && a.p.splits == 1 && !act_blks && T <= INT32_MAX) {
    if (a.f32) SB_CUDA(sb_launch(ctx, head_rows_kernel<float>, dim3((unsigned)T), dim3(256), 0, a));
    else SB_CUDA(sb_launch(ctx, head_rows_kernel<bf16>, dim3((unsigned)T), dim3(256), 0, a));
    ctx->launches++;
    return STRICTB200_OK;
  }
  const int item_blocks = (items + 7) / 8;
  const int64_t blocks = T * (item_blocks + act_blks);
  if (blocks > INT32_MAX || a.p.splits > 8) return sb_fail(STRICTB200_ERR_INVALID_ARG, "head split: too many rows or partial sums");
  const size_t smem = vec ? 0 : (size_t)8 * std::max(s.dim, s.vdim) * sizeof(float);
  if (smem > 48 * 1024) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "heads of more than 1536 dims");
  auto go = [&](auto kernel) { return sb_launch(ctx, kernel, dim3((unsigned)blocks), dim3(256), smem, a, T, item_blocks, act_blks); };
  if (a.f32) SB_CUDA(vec ? go(head_split_kernel<float, true>) : go(head_split_kernel<float, false>));
  else SB_CUDA(vec ? go(head_split_kernel<bf16, true>) : go(head_split_kernel<bf16, false>));
  ctx->launches++;
  return STRICTB200_OK;
}

int k_act_rows(strictb200_ctx* ctx, const ProjRows& p, const ActArgs& a, bool f32, int64_t T) {
  const int blocks = act_blocks(a);
  if (!blocks) return STRICTB200_OK;
  if (f32) SB_CUDA(sb_launch(ctx, act_rows_kernel<float>, dim3((unsigned)(T * blocks)), dim3(256), 0, p, a, T, blocks));
  else SB_CUDA(sb_launch(ctx, act_rows_kernel<bf16>, dim3((unsigned)(T * blocks)), dim3(256), 0, p, a, T, blocks));
  ctx->launches++;
  return STRICTB200_OK;
}

int k_head_attn_any(strictb200_ctx* ctx, const HeadShape& s, bool f32, const void* q, const void* kc, const void* vc, const float* gate, const int32_t* seq,
                    const int32_t* pos, const int32_t* lens, int64_t T, int maxlen, void* out, int64_t ldo) {
  const size_t smem = (size_t)(s.dim + s.vdim + 512) * sizeof(float);
  if (smem > 40 * 1024) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "attention: heads too wide");
  if (T > 65535) return sb_fail(STRICTB200_ERR_INVALID_ARG, "attention: too many rows for the any-width kernel");
  const dim3 grid((unsigned)s.H, (unsigned)T);
  if (f32) SB_CUDA(sb_launch(ctx, head_attn_any_kernel<float>, grid, dim3(256), smem, s, (const float*)q, (const float*)kc, (const float*)vc, gate, seq, pos, lens, maxlen, (float*)out, ldo));
  else SB_CUDA(sb_launch(ctx, head_attn_any_kernel<bf16>, grid, dim3(256), smem, s, (const bf16*)q, (const bf16*)kc, (const bf16*)vc, gate, seq, pos, lens, maxlen, (bf16*)out, ldo));
  ctx->launches++;
  return STRICTB200_OK;
}

int k_head_combine(strictb200_ctx* ctx, const HeadShape& s, const float* o_part, const float* ml_part, const float* gate, const int32_t* lens, int B, int maxlen,
                   int chunk, int nsplit, bf16* out, int64_t ldo) {
  if (nsplit > 8) return sb_fail(STRICTB200_ERR_INVALID_ARG, "attention: at most 8 key chunks");
  const dim3 grid((unsigned)B, (unsigned)((s.H + 7) / 8));
  auto go = [&](auto kernel) { return sb_launch(ctx, kernel, grid, dim3(256), 0, s, o_part, ml_part, gate, lens, maxlen, chunk, nsplit, out, ldo); };
  SB_CUDA(s.row() == 64 ? go(head_combine_kernel<64>) : go(head_combine_kernel<128>));
  ctx->launches++;
  return STRICTB200_OK;
}
