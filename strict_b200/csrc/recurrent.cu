// Layers that carry a state per sequence instead of a cache. All states are fp32 and are advanced in place, so a prompt may be
// cut anywhere.
//
// Real-gated linear recurrence: u = causal convolution of x per channel; r, i = sigmoid of block-diagonal products of u;
//   log a = -8 r softplus(lam), S <- a S + sqrt(1 - a^2) i u, out = S gelu(y).
//   * k_gated_conv: u as the operand of the gate product (rounded to bf16 there, so that the product of bf16 matrices with fp32
//     sums is the exact product of what the recurrence uses), and the convolution's last inputs.
//   * k_gated_scan: prompts run 64, 128 or 256 tokens at a time in a block of 32 channels: every warp folds eight tokens into one (a, b)
//     pair, the pairs meet in shared memory, and each warp replays its tokens from the state before them. Decode is one
//     step per channel. sqrt(1 - a^2) is taken as sqrt(-expm1(2 log a)), which stays exact where a is close to one.
// Retention: S <- decay S + k v^T, o = S^T q.
//   * k_retention_decode: one block per head streams the state once, from the projection's partial sums to the gated output.
//   * k_retention_any: any widths, token by token. Prompts of usual widths: retention_tc.cu.
#include <algorithm>

#include "mixers.cuh"

using namespace mix;

namespace {

// ------------------------------------------------------------------ convolution
// grid rows * (channel blocks + activation blocks), 256 threads
template <typename T>
__global__ void __launch_bounds__(256) gated_conv_kernel(GatedArgs a, int64_t rows, int ch_blocks, int act_blks) {
  SB_TRACE_BEGIN();
  pdl_trigger();
  const int per_row = ch_blocks + act_blks;
  const int64_t t = blockIdx.x / per_row;
  const int blk = blockIdx.x % per_row, w = a.s.width, taps = a.s.taps;
  pdl_wait();
  SB_TRACE_WAITED();
  if (blk >= ch_blocks) {
    act_block<T>(a.act, a.p, rows, t, blk - ch_blocks);
  } else {
    const int c = blk * 256 + (int)threadIdx.x;
    if (c < w) {
      const int b = a.seq ? a.seq[t] : (int)t;
      const int64_t li = a.seq ? t - a.qstart[b] : 0;  // tokens of this launch before the row
      float* hist = a.hist + (int64_t)b * (taps - 1) * w + c;
      const float* k = a.conv + (int64_t)c * taps;
      const float xb = a.x_bias[c], now = proj(a.p, rows, t, w + c) + xb;
      float acc = a.conv_bias[c];
      for (int j = 0; j < taps - 1; j++) {  // oldest first
        const int64_t back = taps - 1 - j;
        const float x = back <= li ? proj(a.p, rows, t - back, w + c) + xb : hist[(taps - 1 + li - back) * w];
        acc = fmaf(k[j], x, acc);
      }
      acc = fmaf(k[taps - 1], now, acc);
      const int bs = a.s.bs(), g = c / bs;
      T* u = (T*)a.u + t * a.s.ld_u() + (int64_t)g * a.s.bs_p() + c - g * bs;
      *u = to_t<T>(acc);
      if (c - g * bs == bs - 1)  // columns that fill the block up meet zero weights, but they must be finite
        for (int j = 1; j <= a.s.bs_p() - bs; j++) u[j] = to_t<T>(0.f);
      if (!a.seq) {  // decode: the row is its sequence's only one, nobody else reads this history
        for (int j = 0; j < taps - 2; j++) hist[(int64_t)j * w] = hist[(int64_t)(j + 1) * w];
        if (taps > 1) hist[(int64_t)(taps - 2) * w] = now;
      }
    }
  }
  SB_TRACE_END(SB_K_ROPE, 0);
}
// Prompt rows, four channels of CONV_ROWS consecutive rows per thread: the taps slide over registers. Blocks of 8 k channels.
constexpr int CONV_ROWS = 16;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) gated_conv_rows_kernel(GatedArgs a, int64_t rows) {
  const int w = a.s.width, c = ((int)blockIdx.x * 128 + (int)threadIdx.x) * 4;
  const int64_t t0 = (int64_t)blockIdx.y * CONV_ROWS;
  pdl_trigger();
  pdl_wait();
  if (c >= w) return;
  const int n = (int)min((int64_t)CONV_ROWS, rows - t0);
  const float4 xb = *(const float4*)(a.x_bias + c), cb = *(const float4*)(a.conv_bias + c);
  float k[4][TAPS];
#pragma unroll
  for (int j = 0; j < 4; j++)
#pragma unroll
    for (int i = 0; i < TAPS; i++) k[j][i] = a.conv[(int64_t)(c + j) * TAPS + i];
  const float* in = a.p.in + t0 * a.p.ld;
  T* u = (T*)a.u + t0 * a.s.ld_u();
  const int ld = (int)a.p.ld, ld_u = (int)a.s.ld_u();
  auto row = [&](int i) {  // row t0 + i
    const float4 v = *(const float4*)(in + (int64_t)i * ld + w + c);
    return make_float4(v.x + xb.x, v.y + xb.y, v.z + xb.z, v.w + xb.w);
  };
  auto tap = [&](float4& o, int j, const float4& x) {
    o.x = fmaf(k[0][j], x.x, o.x); o.y = fmaf(k[1][j], x.y, o.y); o.z = fmaf(k[2][j], x.z, o.z); o.w = fmaf(k[3][j], x.w, o.w);
  };
  int b = a.seq[t0];
  int li = (int)(t0 - a.qstart[b]);  // rows of the same sequence before t0
  if (n == CONV_ROWS && li >= TAPS - 1 && a.seq[t0 + CONV_ROWS - 1] == b) {  // all of one sequence, and so is what comes before
    float4 x[CONV_ROWS + TAPS - 1];
#pragma unroll
    for (int i = 0; i < CONV_ROWS + TAPS - 1; i++) x[i] = row(i - (TAPS - 1));
#pragma unroll
    for (int i = 0; i < CONV_ROWS; i++) {
      float4 o = cb;
#pragma unroll
      for (int j = 0; j < TAPS; j++) tap(o, j, x[i + j]);
      store4<T>(u + (int64_t)i * ld_u + c, o);
    }
    return;
  }
  float4 win[TAPS];  // the row and the ones before it, oldest first
  for (int i = 0; i < n; i++) {
    if (i > 0) {
      const int b1 = a.seq[t0 + i];
      li = b1 == b ? li + 1 : 0;
      b = b1;
    }
    if (i == 0 || li == 0) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; j++) {
        const int back = TAPS - 1 - j;
        win[j] = back <= li ? row(i - back) : *(const float4*)(a.hist + ((int64_t)b * (TAPS - 1) + TAPS - 1 + li - back) * w + c);
      }
    }
    win[TAPS - 1] = row(i);
    float4 o = cb;
#pragma unroll
    for (int j = 0; j < TAPS; j++) tap(o, j, win[j]);
    store4<T>(u + (int64_t)i * ld_u + c, o);
#pragma unroll
    for (int j = 0; j < TAPS - 1; j++) win[j] = win[j + 1];
  }
}
// the convolution's last inputs after a prompt's rows; grid (channel blocks, nb)
__global__ void __launch_bounds__(256) conv_hist_kernel(GatedArgs a, int64_t rows) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * 256 + threadIdx.x, b = blockIdx.y, w = a.s.width, keep = a.s.taps - 1;
  if (c >= w) return;
  const int n = a.lens[b] - a.past[b];
  float* hist = a.hist + (int64_t)b * keep * w + c;
  for (int j = 0; j < keep; j++) {  // ascending: slot j takes slot j + n, which has not been written yet
    const int from = n + j - keep;  // row of this launch, or (negative) a slot from the end
    hist[(int64_t)j * w] = from >= 0 ? proj(a.p, rows, a.qstart[b] + from, w + c) + a.x_bias[c] : hist[(int64_t)(j + n) * w];
  }
}

// ------------------------------------------------------------------ gated recurrence
struct Step { float a, b; };  // S <- a S + b
// One step of the recurrence, and GELU, in fp32: with the library's functions for fp32 results, and for results that end in bf16
// with exponentials, reciprocals and roots through the approximate instructions (relative error 2^-22 and below), and the series
// of 1 - exp(x) where 1 - a^2 would cancel (x > -1/4; the first term left out is below 2^-23 of the sum).
template <typename T>
__device__ __forceinline__ Step gated_step(float zr, float zi, float u, float decay);
template <>
__device__ __forceinline__ Step gated_step<float>(float zr, float zi, float u, float decay) {
  const float la = decay * sigmoid(zr);
  return Step{expf(la), sqrtf(-expm1f(2.f * la)) * sigmoid(zi) * u};
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float LOG2E = 1.4426950408889634f;
template <>
__device__ __forceinline__ Step gated_step<bf16>(float zr, float zi, float u, float decay) {
  // both sigmoids over one reciprocal; exponents are kept where the product of the denominators is finite
  const float er = 1.f + ex2_approx(fminf(-zr * LOG2E, 60.f)), ei = 1.f + ex2_approx(fminf(-zi * LOG2E, 60.f));
  const float inv = rcp_approx(er * ei), la = decay * (ei * inv), x = 2.f * la;
  const float a = ex2_approx(la * LOG2E);
  const float series = -x * fmaf(x, fmaf(x, fmaf(x, fmaf(x, fmaf(x, 1.f / 720.f, 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f), 1.f);
  float root;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(root) : "f"(x > -0.25f ? series : fmaf(-a, a, 1.f)));
  return Step{a, root * (er * inv) * u};
}
template <typename T>
__device__ __forceinline__ float gelu(float z);
template <>
__device__ __forceinline__ float gelu<float>(float z) { return sb_gelu_tanh(z); }
// 1/2 (1 + tanh(y)) = sigmoid(2 y)
template <>
__device__ __forceinline__ float gelu<bf16>(float z) { return z * rcp_approx(1.f + ex2_approx(-1.5957691216f * LOG2E * fmaf(0.044715f * z * z, z, z))); }
constexpr int SCAN_PER = 8;  // tokens per warp and pass
// grid (ceil(width / 32), nb), SCAN_WARPS warps: lane = channel, warp = run of tokens. Few blocks take many warps, a grid that fills
// the GPU takes small blocks, whose loads and sums overlap each other's.
template <typename T, int SCAN_WARPS>
__global__ void __launch_bounds__(SCAN_WARPS * 32, 32 / SCAN_WARPS) gated_scan_kernel(GatedArgs g, int64_t rows) {
  __shared__ Step fold[SCAN_WARPS][32];
  __shared__ float carry[32];
  SB_TRACE_BEGIN();
  pdl_trigger();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, w = g.s.width;
  const int c = blockIdx.x * 32 + lane, seq = blockIdx.y;
  const bool live = c < w;
  const int bs = g.s.bs(), blk = live ? c / bs : 0, in_blk = live ? c - blk * bs : 0;
  const float rb = live ? g.r_bias[c] : 0.f, ib = live ? g.i_bias[c] : 0.f, decay = live ? g.decay[c] : 0.f, yb = live ? g.y_bias[c] : 0.f;
  pdl_wait();
  SB_TRACE_WAITED();
  const int n = live ? g.lens[seq] - g.past[seq] : 0, n_all = g.lens[seq] - g.past[seq];  // a lane without a channel has no tokens
  const int64_t row0 = g.qstart[seq];
  // the same base for every lane, 32-bit offsets (the host checks that a sequence's rows fit)
  const float* gates = g.gates + row0 * 2 * w;
  const T* us = (const T*)g.u + row0 * g.s.ld_u();
  const float* ys = g.p.in + row0 * g.p.ld;  // a prompt's projection is finished
  T* out = (T*)g.out + row0 * g.ldo;
  const uint32_t ld_g = 2 * (uint32_t)w, ld_u = (uint32_t)g.s.ld_u(), ld_y = (uint32_t)g.p.ld, ldo = (uint32_t)g.ldo;
  const uint32_t og = blk * 2 * bs + in_blk, ou = blk * g.s.bs_p() + in_blk, oc = live ? c : 0;
  if (warp == 0) carry[lane] = live ? g.state[(int64_t)seq * w + c] : 0.f;
  for (int t0 = 0; t0 < n_all; t0 += SCAN_WARPS * SCAN_PER) {
    const int first = t0 + warp * SCAN_PER;
    const uint32_t f = (uint32_t)first;
    Step st[SCAN_PER];
    float y[SCAN_PER];
    if (first + SCAN_PER <= n) {
      float vr[SCAN_PER], vi[SCAN_PER], vu[SCAN_PER];
#pragma unroll
      for (int j = 0; j < SCAN_PER; j++) {
        const uint32_t o = (f + j) * ld_g + og;
        vr[j] = __ldcs(gates + o);
        vi[j] = __ldcs(gates + o + (uint32_t)bs);
        vu[j] = to_f(us[(f + j) * ld_u + ou]);
        y[j] = __ldcs(ys + (f + j) * ld_y + oc);
      }
#pragma unroll
      for (int j = 0; j < SCAN_PER; j++) st[j] = gated_step<T>(vr[j] + rb, vi[j] + ib, vu[j], decay);
    } else {
#pragma unroll
      for (int j = 0; j < SCAN_PER; j++) {
        st[j] = Step{1.f, 0.f};
        y[j] = 0.f;
        if (first + j < n) {
          const uint32_t o = (f + j) * ld_g + og;
          st[j] = gated_step<T>(gates[o] + rb, gates[o + (uint32_t)bs] + ib, to_f(us[(f + j) * ld_u + ou]), decay);
          y[j] = ys[(f + j) * ld_y + oc];
        }
      }
    }
    Step all{1.f, 0.f};
#pragma unroll
    for (int j = 0; j < SCAN_PER; j++) { all.b = fmaf(st[j].a, all.b, st[j].b); all.a *= st[j].a; }
    fold[warp][lane] = all;
    __syncthreads();
    float s = carry[lane];
#pragma unroll 8
    for (int v = 0; v < warp; v++) {
      const Step x = fold[v][lane];
      s = fmaf(x.a, s, x.b);
    }
    __syncthreads();  // everybody has read the state before this pass, and the runs
    if (warp == SCAN_WARPS - 1) carry[lane] = fmaf(all.a, s, all.b);  // read after the next pass's first barrier
#pragma unroll
    for (int j = 0; j < SCAN_PER; j++) {
      s = fmaf(st[j].a, s, st[j].b);
      if (first + j < n) out[(f + j) * ldo + oc] = to_t<T>(s * gelu<T>(y[j] + yb));
    }
  }
  __syncthreads();
  if (warp == 0 && live) g.state[(int64_t)seq * w + c] = carry[lane];
  SB_TRACE_END(SB_K_RECURRENCE, 0);
}
// decode: grid (ceil(width / 256), rows)
template <typename T>
__global__ void __launch_bounds__(256) gated_step_kernel(GatedArgs g, int64_t rows) {
  SB_TRACE_BEGIN();
  pdl_trigger();
  const int c = blockIdx.x * 256 + threadIdx.x, w = g.s.width;
  const int64_t t = blockIdx.y;
  pdl_wait();
  SB_TRACE_WAITED();
  if (c < w) {
    const int bs = g.s.bs(), blk = c / bs, in_blk = c - blk * bs;
    const int64_t gr = (int64_t)blk * 2 * bs + in_blk;
    const float* gates = g.gates + t * 2 * w + gr;
    const float u = to_f(((const T*)g.u)[t * g.s.ld_u() + (int64_t)blk * g.s.bs_p() + in_blk]);
    const Step st = gated_step<T>(gates[0] + g.r_bias[c], gates[bs] + g.i_bias[c], u, g.decay[c]);
    const float s = fmaf(st.a, g.state[t * w + c], st.b);
    g.state[t * w + c] = s;
    ((T*)g.out)[t * g.ldo + c] = to_t<T>(s * gelu<T>(proj(g.p, rows, t, c) + g.y_bias[c]));
  }
  SB_TRACE_END(SB_K_RECURRENCE, 0);
}

// ------------------------------------------------------------------ retention, any widths
// grid (H, sequences), 256 threads. A state element belongs to one thread for the whole launch.
template <typename T>
__global__ void __launch_bounds__(256) retention_any_kernel(RetentionArgs a, int64_t rows) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  pdl_trigger();
  pdl_wait();
  const HeadShape& s = a.s;
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, row = s.row();
  const int n = a.qstart ? a.lens[b] - a.past[b] : 1;
  const int64_t t0 = a.qstart ? a.qstart[b] : b;
  float *qs = sm, *ks = qs + s.dim, *vs = ks + s.dim, *os = vs + s.vdim, *part = os + s.vdim;  // part [256]
  float* S = a.state + ((int64_t)b * s.H + h) * s.dim * s.vdim;
  const float decay = a.decay[h];
  const int parts = s.vdim <= 256 ? 256 / s.vdim : 1;  // threads that share a value column
  const int64_t gcol = (int64_t)s.H * (2 * s.dim + s.vdim) + (int64_t)h * s.vdim;
  for (int i = 0; i < n; i++) {
    const int64_t t = t0 + i, at = (t * s.H + h) * row;
    for (int e = tid; e < s.dim; e += 256) { qs[e] = to_f(((const T*)a.q)[at + e]); ks[e] = to_f(((const T*)a.k)[at + e]); }
    for (int e = tid; e < s.vdim; e += 256) vs[e] = to_f(((const T*)a.v)[at + e]);
    __syncthreads();
    for (int v0 = 0; v0 < s.vdim; v0 += 256) {
      const int v = parts > 1 ? tid % s.vdim : v0 + tid, p = parts > 1 ? tid / s.vdim : 0;
      float acc = 0.f;
      if (v < s.vdim && p < parts) {
        const float vv = vs[v];
#pragma unroll 4
        for (int d = p; d < s.dim; d += parts) {
          const float x = fmaf(decay, S[(int64_t)d * s.vdim + v], ks[d] * vv);
          S[(int64_t)d * s.vdim + v] = x;
          acc = fmaf(qs[d], x, acc);
        }
      }
      if (parts > 1) {
        part[tid] = acc;
        __syncthreads();
        if (p == 0) {
          for (int j = 1; j < parts; j++) acc += part[j * s.vdim + v];
          os[v] = acc;
        }
      } else if (v < s.vdim) {
        os[v] = acc;
      }
    }
    __syncthreads();
    float ss = 0.f;
    for (int v = tid; v < s.vdim; v += 256) ss += os[v] * os[v];
    ss = block_sum(ss, red);
    const float r = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)s.vdim), a.eps)));
    for (int v = tid; v < s.vdim; v += 256) {
      const float g = proj(a.p, rows, t, gcol + v);
      ((T*)a.out)[t * a.ldo + (int64_t)h * s.vdim + v] = to_t<T>(os[v] * r * (g * sigmoid(g)));
    }
    __syncthreads();
  }
}

// ------------------------------------------------------------------ retention, decode
// B * H blocks of one head each, then B * act_blks for the feed-forward's columns; 256 threads. The threads of a block form
// 256 / (vdim / 4) groups; a thread owns four value columns of every group-th state row.
constexpr int RET_UNROLL = 8;
__global__ void __launch_bounds__(256) retention_decode_kernel(RetentionArgs a, int64_t B, int act_blks) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  SB_TRACE_BEGIN();
  pdl_trigger();
  const HeadShape& s = a.s;
  const int tid = threadIdx.x;
  const int64_t heads = B * s.H;
  if (blockIdx.x >= heads) {
    pdl_wait();
    SB_TRACE_WAITED();
    act_block<bf16>(a.act, a.p, B, (blockIdx.x - heads) / act_blks, (int)((blockIdx.x - heads) % act_blks));
    SB_TRACE_END(SB_K_RECURRENCE, 0);
    return;
  }
  const int h = (int)(blockIdx.x % s.H);
  const int64_t b = blockIdx.x / s.H;
  float* S = a.state + (b * s.H + h) * (int64_t)s.dim * s.vdim;
  // the state starts on its way to L2 while the projection still runs (a hint: nothing is read before the wait)
  for (int i = tid * 32; i < s.dim * s.vdim; i += 256 * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(S + i));
  const float decay = a.decay[h];
  pdl_wait();
  SB_TRACE_WAITED();
  float *x = sm, *qs = x + 2 * s.dim, *ks = qs + s.dim, *vs = ks + s.dim, *gs = vs + s.vdim, *po = gs + s.vdim;  // po [groups][vdim]
  const int p = a.cache_lens[b];
  if (p < 0 || p >= a.max_pos) return;
  const int64_t HD = (int64_t)s.H * s.dim;
  const int n4 = (2 * s.dim + 2 * s.vdim) / 4;
  for (int i = tid; i < n4; i += 256) {  // q, k (before rotation), v, g of this head
    int e = i * 4;
    float* dst;
    int64_t col;
    if (e < s.dim) { col = (int64_t)h * s.dim + e; dst = x + e; }
    else if (e < 2 * s.dim) { col = HD + (int64_t)h * s.dim + e - s.dim; dst = x + e; }
    else if (e < 2 * s.dim + s.vdim) { e -= 2 * s.dim; col = 2 * HD + (int64_t)h * s.vdim + e; dst = vs + e; }
    else { e -= 2 * s.dim + s.vdim; col = 2 * HD + (int64_t)(s.H + h) * s.vdim + e; dst = gs + e; }
    *(float4*)dst = proj4(a.p, B, b, col);
  }
  __syncthreads();
  const int half = s.rot / 2;
  for (int e = tid; e < 2 * s.dim; e += 256) {
    const int d = e < s.dim ? e : e - s.dim;
    const float* src = e < s.dim ? x : x + s.dim;
    float v = src[d];
    if (d < s.rot) {
      const int i = d < half ? d : d - half;
      const float c = a.cos_t[(int64_t)p * half + i], n = a.sin_t[(int64_t)p * half + i];
      v = d < half ? src[d] * c - src[d + half] * n : src[d] * c + src[d - half] * n;
    }
    if (e < s.dim) qs[d] = v;
    else ks[d] = v * s.k_scale;
  }
  __syncthreads();
  const int vq = s.vdim / 4, groups = 256 / vq, g = tid / vq, c4 = (tid % vq) * 4;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (g < groups) {
    const float4 v = *(const float4*)(vs + c4);
    for (int d0 = g; d0 < s.dim; d0 += groups * RET_UNROLL) {
      float4 st[RET_UNROLL];
#pragma unroll
      for (int j = 0; j < RET_UNROLL; j++)
        if (d0 + j * groups < s.dim) st[j] = __ldcs((const float4*)(S + (int64_t)(d0 + j * groups) * s.vdim + c4));
#pragma unroll
      for (int j = 0; j < RET_UNROLL; j++) {
        const int d = d0 + j * groups;
        if (d < s.dim) {
          const float k = ks[d], q = qs[d];
          st[j].x = fmaf(decay, st[j].x, k * v.x); st[j].y = fmaf(decay, st[j].y, k * v.y);
          st[j].z = fmaf(decay, st[j].z, k * v.z); st[j].w = fmaf(decay, st[j].w, k * v.w);
          __stcs((float4*)(S + (int64_t)d * s.vdim + c4), st[j]);
          o.x = fmaf(q, st[j].x, o.x); o.y = fmaf(q, st[j].y, o.y); o.z = fmaf(q, st[j].z, o.z); o.w = fmaf(q, st[j].w, o.w);
        }
      }
    }
    *(float4*)(po + g * s.vdim + c4) = o;
  }
  __syncthreads();
  float ss = 0.f;
  for (int v = tid; v < s.vdim; v += 256) {
    float t = 0.f;
    for (int j = 0; j < groups; j++) t += po[j * s.vdim + v];
    po[v] = t;  // this thread's column
    ss += t * t;
  }
  ss = block_sum(ss, red);
  const float r = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)s.vdim), a.eps)));
  for (int v = tid; v < s.vdim; v += 256) ((bf16*)a.out)[b * a.ldo + (int64_t)h * s.vdim + v] = __float2bfloat16_rn(po[v] * r * (gs[v] * sigmoid(gs[v])));
  SB_TRACE_END(SB_K_RECURRENCE, 0);
}
size_t retention_decode_smem(const HeadShape& s) { return (size_t)(4 * s.dim + 2 * s.vdim + 256 / (s.vdim / 4) * s.vdim) * sizeof(float); }

}  // namespace

SB_TRACE_TU(recurrent)

int k_gated_conv(strictb200_ctx* ctx, const GatedArgs& a, int64_t T) {
  const int ch = (a.s.width + 255) / 256, act = act_blocks(a.act);
  if (T * (ch + act) > INT32_MAX || a.p.splits > 8) return sb_fail(STRICTB200_ERR_INVALID_ARG, "gated recurrence: too many rows or partial sums");
  const dim3 grid((unsigned)(T * (ch + act)));
  const GatedShape& s = a.s;
  const bool rows = a.seq && !a.act.kind && a.p.splits == 1 && s.width % 4 == 0 && s.bs() % 8 == 0 && a.p.ld % 4 == 0 && s.taps >= 2 && s.taps <= 4 &&
                    T <= (int64_t)65535 * CONV_ROWS;
  if (rows) {
    const dim3 g((unsigned)((s.width / 4 + 127) / 128), (unsigned)((T + CONV_ROWS - 1) / CONV_ROWS));
    auto go = [&](auto kernel) { return sb_launch(ctx, kernel, g, dim3(128), 0, a, T); };
    if (a.f32) SB_CUDA(s.taps == 2 ? go(gated_conv_rows_kernel<float, 2>) : s.taps == 3 ? go(gated_conv_rows_kernel<float, 3>) : go(gated_conv_rows_kernel<float, 4>));
    else SB_CUDA(s.taps == 2 ? go(gated_conv_rows_kernel<bf16, 2>) : s.taps == 3 ? go(gated_conv_rows_kernel<bf16, 3>) : go(gated_conv_rows_kernel<bf16, 4>));
  } else if (a.f32) SB_CUDA(sb_launch(ctx, gated_conv_kernel<float>, grid, dim3(256), 0, a, T, ch, act));
  else SB_CUDA(sb_launch(ctx, gated_conv_kernel<bf16>, grid, dim3(256), 0, a, T, ch, act));
  ctx->launches++;
  if (!a.seq || a.s.taps < 2) return STRICTB200_OK;
  SB_CUDA(sb_launch(ctx, conv_hist_kernel, dim3((unsigned)ch, (unsigned)a.nb), dim3(256), 0, a, T));
  ctx->launches++;
  return STRICTB200_OK;
}

int k_gated_scan(strictb200_ctx* ctx, const GatedArgs& a, int64_t T) {
  if (!a.seq) {
    const dim3 grid((unsigned)((a.s.width + 255) / 256), (unsigned)T);
    if (a.f32) SB_CUDA(sb_launch(ctx, gated_step_kernel<float>, grid, dim3(256), 0, a, T));
    else SB_CUDA(sb_launch(ctx, gated_step_kernel<bf16>, grid, dim3(256), 0, a, T));
  } else {
    const dim3 grid((unsigned)((a.s.width + 31) / 32), (unsigned)a.nb);
    if ((int64_t)a.max_new * std::max<int64_t>(std::max<int64_t>(2 * a.s.width, a.s.ld_u()), std::max(a.p.ld, a.ldo)) > UINT32_MAX)
      return sb_fail(STRICTB200_ERR_INVALID_ARG, "gated recurrence: too many rows of a sequence in one launch");
    const int64_t blocks = (int64_t)grid.x * grid.y;
    const int warps = blocks > 4 * ctx->sm_count ? 8 : blocks > ctx->sm_count ? 16 : 32;
    auto go = [&](auto kernel) { return sb_launch(ctx, kernel, grid, dim3(warps * 32), 0, a, T); };
    if (a.f32) SB_CUDA(warps == 8 ? go(gated_scan_kernel<float, 8>) : warps == 16 ? go(gated_scan_kernel<float, 16>) : go(gated_scan_kernel<float, 32>));
    else SB_CUDA(warps == 8 ? go(gated_scan_kernel<bf16, 8>) : warps == 16 ? go(gated_scan_kernel<bf16, 16>) : go(gated_scan_kernel<bf16, 32>));
  }
  ctx->launches++;
  return STRICTB200_OK;
}

int k_retention_any(strictb200_ctx* ctx, const RetentionArgs& a) {
  const HeadShape& s = a.s;
  const size_t smem = (size_t)(2 * s.dim + 2 * s.vdim + 256) * sizeof(float);
  if (smem > 40 * 1024) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "retention: heads too wide");
  const dim3 grid((unsigned)s.H, (unsigned)a.nb);
  const int64_t rows = a.qstart ? 0 : a.nb;  // (stride of partial sums; a prompt's projection is one finished array)
  if (a.f32) SB_CUDA(sb_launch(ctx, retention_any_kernel<float>, grid, dim3(256), smem, a, rows));
  else SB_CUDA(sb_launch(ctx, retention_any_kernel<bf16>, grid, dim3(256), smem, a, rows));
  ctx->launches++;
  return STRICTB200_OK;
}

bool sb_retention_decode_fits(const HeadShape& s) {
  return s.dim % 4 == 0 && s.vdim % 4 == 0 && s.vdim <= 1024 && retention_decode_smem(s) <= 40 * 1024;
}
int k_retention_decode(strictb200_ctx* ctx, const RetentionArgs& a, int64_t B) {
  if (!sb_retention_decode_fits(a.s) || a.p.ld % 4 || a.p.splits > 8) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "retention: widths the decode kernel does not take");
  const int act = act_blocks(a.act);
  SB_CUDA(sb_launch(ctx, retention_decode_kernel, dim3((unsigned)(B * (a.s.H + act))), dim3(256), retention_decode_smem(a.s), a, B, act));
  ctx->launches++;
  return STRICTB200_OK;
}
