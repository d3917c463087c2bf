// Retention over prompts on the tcgen05 tensor cores: S <- decay S + k v^T, o = S^T q per head (heads of up to 128 dims), then o
// over its root mean square times silu(g).
// One block owns one head of one sequence and walks its tokens in chunks of 128; with n tokens in the chunk and rows i, j:
//   P = Q K^T                           P_ij *= decay^(i - j) for j <= i, else 0; kept as two bf16 terms (hi + lo)
//   O = P V,  O2 = Q S                  o_i = O_i + decay^(i + 1) O2_i
//   S <- decay^n S + K^T V'             V'_j = decay^(n - 1 - j) v_j
// The state stays in tensor memory in fp32 from the first chunk to the last (lane = query/key dim, column = value dim). As the
// operand of Q S it is written to shared memory as two bf16 terms, and so is V'; q, k and v themselves are bf16, the powers of
// the decay fp32. Tensor memory: P, O, O2 and S, 128 columns each.
//   warps 0..15  rows: thread (row, quarter) owns 32 columns of row `row` of every tile
//   warp 16      one lane issues copies and products
// Few (sequence, head) pairs leave most SMs idle, so a prompt is then cut into segments of whole chunks, in two launches: the first
// walks every segment but the last for its own contribution to the state alone; the second starts each segment from the state
// that the contributions before it add up to.
// A row thread takes its sums of a chunk out of tensor memory, prepares the next chunk's state operand, and only then is the chunk
// finished, while the next one's products run: the sums (bf16) and their sums of squares pass through the tiles of V', which are
// free between two chunks, so that the gates are read and the output written whole rows at a time.
// Every mbarrier wait is bounded: on expiry the block records an error word in host-visible memory, stops, frees its tensor
// memory and returns.
#include <algorithm>

#include "mixers.cuh"
#include "tcgen05.cuh"

using namespace tc;

namespace {

constexpr int CHUNK = 128;
constexpr int ROW_THREADS = 4 * CHUNK;
constexpr int RT_THREADS = ROW_THREADS + 32;

struct RtArgs {
  int H, dim, vdim;
  const int32_t *lens, *past, *qstart;
  const float* decay;
  float* state;
  const float* g;   // first gate column of the projection
  int64_t ld_g;
  float eps;
  bf16* out;
  int64_t ldo;
  int* status;
  // segments: chunks of each, how many there are, and per segment [nb, H, dim, vdim] of scratch: the state that a segment leaves
  // (segment 0 with what came before it); the last one holds a copy of the state before the launch
  int seg_chunks, segs;
  float* seg_state;
};

// two bf16 terms by truncation: hi = the upper 16 bits, lo = the upper 16 bits of the exact remainder
__device__ __forceinline__ void split2(float p0, float p1, uint32_t& hi, uint32_t& lo) {
  const uint32_t b0 = __float_as_uint(p0), b1 = __float_as_uint(p1);
  hi = __byte_perm(b0, b1, 0x7632);
  lo = __byte_perm(__float_as_uint(p0 - __uint_as_float(b0 & 0xFFFF0000u)), __float_as_uint(p1 - __uint_as_float(b1 & 0xFFFF0000u)), 0x7632);
}
__device__ __forceinline__ void arrive(uint64_t* bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory"); }
// 16 bytes `chunk` of row `row` of a swizzled box
__device__ __forceinline__ uint32_t box_off(int row, int chunk) { return (uint32_t)(row * 128 + ((chunk ^ (row & 7)) << 4)); }

// STATE: the first launch of a prompt in segments. grid (H, nb, segments)
template <bool STATE>
__global__ void __launch_bounds__(RT_THREADS) retention_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                                                      const __grid_constant__ CUtensorMap map_v, RtArgs a) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t bar_qk, bar_v, bar_s, bar_o, bar_state, s_ready, vp_ready, p_ready;
  __shared__ uint32_t tmem_base_slot;
  __shared__ float pw[CHUNK + 1], pw_seg;

  const int h = blockIdx.x, b = blockIdx.y, seg = blockIdx.z;
  const int first = seg * a.seg_chunks * CHUNK, n_seq = a.lens[b] - a.past[b];
  if (first >= n_seq) return;  // whole block, before anything is allocated
  const bool last = first + a.seg_chunks * CHUNK >= n_seq;
  if (STATE && last) return;   // nobody starts from the state the last segment leaves
  const int n_all = last ? n_seq - first : a.seg_chunks * CHUNK, chunks = (n_all + CHUNK - 1) / CHUNK;
  const int64_t row0 = a.qstart[b] + first;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  uint8_t *bQ = smem, *bK = bQ + TILE_BYTES, *bV = bK + TILE_BYTES, *bVh = bV + TILE_BYTES, *bVl = bVh + TILE_BYTES, *bSh = bVl + TILE_BYTES, *bSl = bSh + TILE_BYTES;
  const uint32_t sQ = smem_u32(bQ), sK = smem_u32(bK), sV = smem_u32(bV), sVh = smem_u32(bVh), sVl = smem_u32(bVl), sSh = smem_u32(bSh), sSl = smem_u32(bSl);
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&bar_qk), 1); mbar_init(smem_u32(&bar_v), 1);
    mbar_init(smem_u32(&bar_s), 1); mbar_init(smem_u32(&bar_o), 1); mbar_init(smem_u32(&bar_state), 1);
    mbar_init(smem_u32(&s_ready), ROW_THREADS); mbar_init(smem_u32(&vp_ready), ROW_THREADS); mbar_init(smem_u32(&p_ready), ROW_THREADS);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (threadIdx.x == CHUNK + 1) pw_seg = (float)pow((double)a.decay[h], (double)(a.seg_chunks * CHUNK));
  if (threadIdx.x <= CHUNK) pw[threadIdx.x] = (float)pow((double)a.decay[h], (double)threadIdx.x);
  if (warp == 16) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_slot)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tP = tmem_base_slot, tO = tP + 128, tO2 = tP + 256, tS = tP + 384;
  // D = F32, A = B = bf16, M = N = 128; bit 15: A is MN-major (its rows are the reduction), bit 16: B is
  constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(128 >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
  constexpr uint32_t idesc_b = idesc | (1u << 16), idesc_ab = idesc_b | (1u << 15);

  if (warp == 16) {
    if (lane == 0) {
      auto load = [&](int c) {
        const int row = (int)row0 + c * CHUNK;
        mbar_expect_tx(smem_u32(&bar_qk), (STATE ? 1 : 2) * TILE_BYTES);
        for (int i = 0; i < 2; i++) {
          if (!STATE) tma_load_3d(sQ + i * HALF_BYTES, &map_q, i * 64, h, row, smem_u32(&bar_qk));
          tma_load_3d(sK + i * HALF_BYTES, &map_k, i * 64, h, row, smem_u32(&bar_qk));
        }
        mbar_expect_tx(smem_u32(&bar_v), TILE_BYTES);
        for (int i = 0; i < 2; i++) tma_load_3d(sV + i * HALF_BYTES, &map_v, i * 64, h, row, smem_u32(&bar_v));
      };
      load(0);
      bool good = true;
      for (int c = 0; c < chunks && good; c++) {
        const uint32_t ph = (uint32_t)(c & 1);
        if (c + 1 < chunks) {  // the next chunk's rows on their way to L2
          const int row = (int)row0 + (c + 1) * CHUNK;
          for (int i = 0; i < 2; i++) {
            if (!STATE) tma_prefetch_3d(&map_q, i * 64, h, row);
            tma_prefetch_3d(&map_k, i * 64, h, row);
            tma_prefetch_3d(&map_v, i * 64, h, row);
          }
        }
        good = mbar_wait(smem_u32(&bar_qk), ph) && mbar_wait(smem_u32(&s_ready), ph);
        if (!good) break;
        tc_fence_after();
        if (!STATE) {
#pragma unroll
          for (int s = 0; s < 8; s++) {
            const uint32_t off = (uint32_t)((s >> 2) * HALF_BYTES + (s & 3) * 32);
            tc_mma_ss(tP, desc_kmajor(sQ + off), desc_kmajor(sK + off), idesc, s ? 1u : 0u);
          }
          tc_commit(smem_u32(&bar_s));
#pragma unroll
          for (int s = 0; s < 8; s++) {
            const uint64_t dq = desc_kmajor(sQ + (uint32_t)((s >> 2) * HALF_BYTES + (s & 3) * 32));
            tc_mma_ss(tO2, dq, desc_mnmajor(sSh + (uint32_t)(s * 2048)), idesc_b, s ? 1u : 0u);
            tc_mma_ss(tO2, dq, desc_mnmajor(sSl + (uint32_t)(s * 2048)), idesc_b, 1u);
          }
          good = mbar_wait(smem_u32(&p_ready), ph) && mbar_wait(smem_u32(&bar_v), ph);
          if (!good) break;
          tc_fence_after();
#pragma unroll
          for (int s = 0; s < 8; s++) {
            const uint64_t dv = desc_mnmajor(sV + (uint32_t)(s * 2048));
            const uint32_t pcol = (uint32_t)((s >> 1) * 32 + (s & 1) * 8);
            tc_mma_ts(tO, tP + pcol, dv, idesc_b, s ? 1u : 0u);
            tc_mma_ts(tO, tP + pcol + 16, dv, idesc_b, 1u);
          }
          tc_commit(smem_u32(&bar_o));
        }
        good = mbar_wait(smem_u32(&vp_ready), ph);
        if (!good) break;
        tc_fence_after();
#pragma unroll
        for (int s = 0; s < 8; s++) {
          const uint64_t dk = desc_mnmajor(sK + (uint32_t)(s * 2048));
          tc_mma_ss(tS, dk, desc_mnmajor(sVh + (uint32_t)(s * 2048)), idesc_ab, 1u);
          tc_mma_ss(tS, dk, desc_mnmajor(sVl + (uint32_t)(s * 2048)), idesc_ab, 1u);
        }
        tc_commit(smem_u32(&bar_state));
        if (c + 1 < chunks) {
          good = mbar_wait(smem_u32(&bar_state), ph);  // every product of the chunk has read its tiles, every row its part of V
          if (good) load(c + 1);
        }
      }
      if (!good) set_status(a.status, 17);
    }
  } else {
    const int row = (int)threadIdx.x & (CHUNK - 1), quarter = (int)threadIdx.x >> 7;
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    const int c0 = quarter * 32;  // first of this thread's columns, in every tile
    const uint32_t box = (uint32_t)((quarter >> 1) * HALF_BYTES);
    const int chunk0 = (quarter & 1) * 4;  // first of its 16-byte chunks in the box's row
    auto rows_sync = [&]() { asm volatile("bar.sync 1, 512;" ::: "memory"); };
    const int64_t head = ((int64_t)b * a.H + h) * a.dim * a.vdim, per_seg = (int64_t)gridDim.y * a.H * a.dim * a.vdim, mine = (int64_t)row * a.vdim + c0;
    // this thread's part of a state (where it exists): what the segment begins with, and where it leaves its own
    const float* S_in = (STATE || (seg == 0 && last) || a.segs == 1 ? a.state : a.seg_state + (seg ? 0 : a.segs - 1) * per_seg) + head + mine;
    float* S_out = (STATE ? a.seg_state + seg * per_seg : a.state) + head + mine;
    const bool s_vec = (a.vdim & 3) == 0;
    const bool vec = ((a.vdim | (int)(a.ld_g & 3) | (int)(a.ldo & 3)) & 3) == 0 && ((uintptr_t)a.g & 15) == 0 && ((uintptr_t)a.out & 7) == 0;
    float* sums = (float*)bVl;  // [4][CHUNK] while the tile is free

    // A chunk of n tokens: the state before it (in tensor memory) as two bf16 tiles, and decay^n times it back to tensor memory.
    auto state_operand = [&](int c) {
      const int n = min(CHUNK, n_all - c * CHUNK);
      const float dn = pw[n];
#pragma unroll
      for (int q = 0; q < 2; q++) {
        uint32_t r[16];
        tc_ld16(tS + lane_base + (uint32_t)(c0 + q * 16), r);
        tc_wait_ld();
#pragma unroll
        for (int j = 0; j < 2 && !STATE; j++) {
          uint4 hi, lo;
          split2(__uint_as_float(r[8 * j]), __uint_as_float(r[8 * j + 1]), hi.x, lo.x);
          split2(__uint_as_float(r[8 * j + 2]), __uint_as_float(r[8 * j + 3]), hi.y, lo.y);
          split2(__uint_as_float(r[8 * j + 4]), __uint_as_float(r[8 * j + 5]), hi.z, lo.z);
          split2(__uint_as_float(r[8 * j + 6]), __uint_as_float(r[8 * j + 7]), hi.w, lo.w);
          const uint32_t off = box + box_off(row, chunk0 + q * 2 + j);
          *(uint4*)(bSh + off) = hi;
          *(uint4*)(bSl + off) = lo;
        }
#pragma unroll
        for (int j = 0; j < 16; j++) r[j] = __float_as_uint(__uint_as_float(r[j]) * dn);
        tc_st16(tS + lane_base + (uint32_t)(c0 + q * 16), r);
      }
      tc_wait_st();
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      tc_fence_before();
      arrive(&s_ready);
    };
    // The values under their powers of the decay at the chunk's end.
    auto value_operand = [&](int c) -> bool {
      const int n = min(CHUNK, n_all - c * CHUNK);
      if (!mbar_wait(smem_u32(&bar_v), (uint32_t)(c & 1))) return false;
      const float wv = row < n ? pw[n - 1 - row] : 0.f;
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const uint32_t off = box + box_off(row, chunk0 + j);
        const uint4 v = *(const uint4*)(bV + off);
        uint4 hi, lo;
        auto both = [&](uint32_t x, uint32_t& o_hi, uint32_t& o_lo) {
          split2(__uint_as_float(x << 16) * wv, __uint_as_float(x & 0xFFFF0000u) * wv, o_hi, o_lo);
        };
        both(v.x, hi.x, lo.x); both(v.y, hi.y, lo.y); both(v.z, hi.z, lo.z); both(v.w, hi.w, lo.w);
        *(uint4*)(bVh + off) = hi;
        *(uint4*)(bVl + off) = lo;
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      arrive(&vp_ready);
      return true;
    };

    auto read_state = [&](const float* S, float* r) {
#pragma unroll
      for (int j = 0; j < 8; j++) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (row < a.dim && c0 + 4 * j < a.vdim) {
          if (s_vec) x = *(const float4*)(S + 4 * j);
          else {
            x.x = S[4 * j];
            if (c0 + 4 * j + 1 < a.vdim) x.y = S[4 * j + 1];
            if (c0 + 4 * j + 2 < a.vdim) x.z = S[4 * j + 2];
            if (c0 + 4 * j + 3 < a.vdim) x.w = S[4 * j + 3];
          }
        }
        r[4 * j] = x.x; r[4 * j + 1] = x.y; r[4 * j + 2] = x.z; r[4 * j + 3] = x.w;
      }
    };
    auto write_state = [&](float* S, const uint32_t* r) {
#pragma unroll
      for (int j = 0; j < 8; j++) {
        if (row >= a.dim || c0 + 4 * j >= a.vdim) continue;
        if (s_vec) *(uint4*)(S + 4 * j) = make_uint4(r[4 * j], r[4 * j + 1], r[4 * j + 2], r[4 * j + 3]);
        else
#pragma unroll
          for (int i = 0; i < 4; i++)
            if (c0 + 4 * j + i < a.vdim) S[4 * j + i] = __uint_as_float(r[4 * j + i]);
      }
    };
    bool ok = true;
    {
      float x[32];
      uint32_t r[32];
      if (STATE && seg > 0) {
#pragma unroll
        for (int j = 0; j < 32; j++) x[j] = 0.f;
      } else {
        read_state(S_in, x);
      }
      if (!STATE && seg > 0) {  // segment 0 left a whole state, the others what they add
        for (int i = 1; i < seg; i++) {
          float y[32];
          read_state(a.seg_state + i * per_seg + head + mine, y);
#pragma unroll
          for (int j = 0; j < 32; j++) x[j] = fmaf(pw_seg, x[j], y[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < 32; j++) r[j] = __float_as_uint(x[j]);
      if (STATE && seg == 0) write_state(a.seg_state + (a.segs - 1) * per_seg + head + mine, r);
      tc_st32(tS + lane_base + (uint32_t)c0, r);
      tc_wait_st();
      state_operand(0);
      ok = value_operand(0);
    }
    if constexpr (STATE) {
      for (int c = 0; c < chunks && ok; c++) {
        if (!mbar_wait(smem_u32(&bar_state), (uint32_t)(c & 1))) { ok = false; break; }
        tc_fence_after();
        if (c + 1 < chunks) {
          state_operand(c + 1);
          ok = value_operand(c + 1);
          continue;
        }
        uint32_t r[32];
        tc_ld32(tS + lane_base + (uint32_t)c0, r);
        tc_wait_ld();
        write_state(S_out, r);
      }
    } else
    for (int c = 0; c < chunks && ok; c++) {
      const uint32_t ph = (uint32_t)(c & 1);
      const int n = min(CHUNK, n_all - c * CHUNK);
      // ---- the chunk's gates on their way to L2: 128 bytes per thread
      {
        const int r = (int)threadIdx.x >> 2, col = ((int)threadIdx.x & 3) * 32;
        if (r < n && col < a.vdim) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.g + (row0 + c * CHUNK + r) * a.ld_g + (int64_t)h * a.vdim + col));
      }
      // ---- P under the decay
      if (!mbar_wait(smem_u32(&bar_s), ph)) { ok = false; break; }
      tc_fence_after();
      {
        uint32_t r[32], hi[16], lo[16];
        tc_ld32(tP + lane_base + (uint32_t)c0, r);
        tc_wait_ld();
#pragma unroll
        for (int j = 0; j < 16; j++) {
          const int k = c0 + 2 * j;
          const float p0 = k <= row ? __uint_as_float(r[2 * j]) * pw[row - k] : 0.f;
          const float p1 = k + 1 <= row ? __uint_as_float(r[2 * j + 1]) * pw[row - k - 1] : 0.f;
          split2(p0, p1, hi[j], lo[j]);
        }
        tc_st16(tP + lane_base + (uint32_t)c0, hi);
        tc_st16(tP + lane_base + (uint32_t)(c0 + 16), lo);
      }
      tc_wait_st();
      tc_fence_before();
      arrive(&p_ready);
      // ---- sums of the chunk
      if (!mbar_wait(smem_u32(&bar_o), ph)) { ok = false; break; }
      tc_fence_after();
      const float d1 = pw[min(row + 1, CHUNK)];
      uint32_t o[16];  // bf16 pairs
      float ss = 0.f;
#pragma unroll
      for (int q = 0; q < 2; q++) {
        uint32_t r[16], r2[16];
        tc_ld16(tO + lane_base + (uint32_t)(c0 + q * 16), r);
        tc_ld16(tO2 + lane_base + (uint32_t)(c0 + q * 16), r2);
        tc_wait_ld();
#pragma unroll
        for (int j = 0; j < 16; j += 2) {
          const float u = fmaf(d1, __uint_as_float(r2[j]), __uint_as_float(r[j])), v = fmaf(d1, __uint_as_float(r2[j + 1]), __uint_as_float(r[j + 1]));
          o[q * 8 + j / 2] = mix::pack_bf16(u, v);
          ss = fmaf(u, u, fmaf(v, v, ss));  // columns beyond vdim are zero
        }
      }
      if (!mbar_wait(smem_u32(&bar_state), ph)) { ok = false; break; }
      tc_fence_after();
      sums[quarter * CHUNK + row] = ss;
#pragma unroll
      for (int j = 0; j < 4; j++) *(uint4*)(bVh + box + box_off(row, chunk0 + j)) = make_uint4(o[4 * j], o[4 * j + 1], o[4 * j + 2], o[4 * j + 3]);
      if (c + 1 < chunks) {
        state_operand(c + 1);
      } else if (last) {
        uint32_t r[32];
        tc_ld32(tS + lane_base + (uint32_t)c0, r);
        tc_wait_ld();
        write_state(S_out, r);
      }
      // ---- norm, gate, store: warp w finishes rows 8 w.., four columns per lane
      const int col = 4 * lane;
      const int64_t t0 = row0 + c * CHUNK + 8 * warp;
      const float* g = a.g + t0 * a.ld_g + (int64_t)h * a.vdim + col;
      float4 z[8];
#pragma unroll
      for (int i = 0; i < 8; i++) {
        z[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (8 * warp + i < n && col < a.vdim) {
          const float* p = g + i * a.ld_g;
          if (vec) z[i] = __ldcs((const float4*)p);
          else {
            z[i].x = p[0];
            if (col + 1 < a.vdim) z[i].y = p[1];
            if (col + 2 < a.vdim) z[i].z = p[2];
            if (col + 3 < a.vdim) z[i].w = p[3];
          }
        }
      }
      rows_sync();
      // silu of a pair over one reciprocal; the exponents are kept where the product of the denominators is finite
      auto silu2 = [](float u, float v, float& su, float& sv) {
        float eu, ev, inv;
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(eu) : "f"(fminf(u * -1.4426950408889634f, 60.f)));
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(ev) : "f"(fminf(v * -1.4426950408889634f, 60.f)));
        eu += 1.f;
        ev += 1.f;
        asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(inv) : "f"(eu * ev));
        su = u * (ev * inv);
        sv = v * (eu * inv);
      };
      const float per_dim = 1.0f / (float)a.vdim;
#pragma unroll
      for (int i = 0; i < 8; i++) {
        const int r = 8 * warp + i;
        if (r >= n || col >= a.vdim) continue;
        const float total = sums[r] + sums[CHUNK + r] + sums[2 * CHUNK + r] + sums[3 * CHUNK + r];
        const float rn = rsqrtf(fmaf(total, per_dim, a.eps));
        float s0, s1, s2, s3;
        silu2(z[i].x, z[i].y, s0, s1);
        silu2(z[i].z, z[i].w, s2, s3);
        const uint2 w = *(const uint2*)(bVh + (lane >> 4) * HALF_BYTES + box_off(r, (lane & 15) >> 1) + (lane & 1) * 8);
        const float y0 = __uint_as_float(w.x << 16) * rn * s0, y1 = __uint_as_float(w.x & 0xFFFF0000u) * rn * s1;
        const float y2 = __uint_as_float(w.y << 16) * rn * s2, y3 = __uint_as_float(w.y & 0xFFFF0000u) * rn * s3;
        bf16* dst = a.out + (t0 + i) * a.ldo + (int64_t)h * a.vdim + col;
        if (vec) *(uint2*)dst = make_uint2(mix::pack_bf16(y0, y1), mix::pack_bf16(y2, y3));
        else {
          dst[0] = __float2bfloat16_rn(y0);
          if (col + 1 < a.vdim) dst[1] = __float2bfloat16_rn(y1);
          if (col + 2 < a.vdim) dst[2] = __float2bfloat16_rn(y2);
          if (col + 3 < a.vdim) dst[3] = __float2bfloat16_rn(y3);
        }
      }
      rows_sync();  // the tiles are free again
      if (c + 1 < chunks) ok = value_operand(c + 1);
    }
    if (!ok && row == 0) set_status(a.status, 18);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 16) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tP), "r"(512u) : "memory");
  }
}

}  // namespace

bool sb_retention_prefill_fits(const HeadShape& s) { return s.dim <= 128 && s.vdim <= 128; }

// Segments a prompt is cut into: as many as the SMs take at once (one block per SM), of at least two chunks each.
int sb_retention_segments(strictb200_ctx* ctx, const HeadShape& s, int nb, int max_new) {
  const int chunks = (max_new + CHUNK - 1) / CHUNK;
  int segs = std::min((int)(ctx->sm_count / std::max<int64_t>((int64_t)s.H * nb, 1)), chunks / 2);
  if (segs < 2) return 1;
  const int per = (chunks + segs - 1) / segs;
  return (chunks + per - 1) / per;
}

int k_retention_prefill(strictb200_ctx* ctx, const RetentionArgs& p, int64_t T) {
  const HeadShape& s = p.s;
  if (!sb_retention_prefill_fits(s) || p.f32 || p.p.splits != 1) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "retention: heads the tensor-core kernel does not take");
  if (s.H > INT32_MAX / 2 || p.nb > 65535 || T > INT32_MAX) return sb_fail(STRICTB200_ERR_INVALID_ARG, "retention: too many sequences or rows");
  const int segs = sb_retention_segments(ctx, s, p.nb, p.max_new), chunks = (p.max_new + CHUNK - 1) / CHUNK;
  if (segs > 1 && !p.seg_state) return sb_fail(STRICTB200_ERR_INVALID_ARG, "retention: segments need scratch");
  RtArgs a{s.H, s.dim, s.vdim, p.lens, p.past, p.qstart, p.decay, p.state, p.p.in + (int64_t)s.H * (2 * s.dim + s.vdim), p.p.ld, p.eps, (bf16*)p.out, p.ldo, ctx->d_status,
           (chunks + segs - 1) / segs, segs, p.seg_state};
  const int row = s.row();
  CUtensorMap mq, mk, mv;
  SB_TRY(make_map3(&mq, p.q, row, s.H, T, row, (int64_t)s.H * row));
  SB_TRY(make_map3(&mk, p.k, row, s.H, T, row, (int64_t)s.H * row));
  SB_TRY(make_map3(&mv, p.v, row, s.H, T, row, (int64_t)s.H * row));
  const size_t smem = 7 * TILE_BYTES + 1024;
  static SbDeviceOnce once;
  SB_CUDA(once.run(ctx->device, [&] {
    const cudaError_t e = cudaFuncSetAttribute(retention_prefill_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return e != cudaSuccess ? e : cudaFuncSetAttribute(retention_prefill_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  }));
  if (segs > 1) {
    retention_prefill_kernel<true><<<dim3((unsigned)s.H, (unsigned)p.nb, (unsigned)segs - 1), RT_THREADS, smem, ctx->stream>>>(mq, mk, mv, a);
    SB_LAUNCHED(ctx);
  }
  retention_prefill_kernel<false><<<dim3((unsigned)s.H, (unsigned)p.nb, (unsigned)segs), RT_THREADS, smem, ctx->stream>>>(mq, mk, mv, a);
  SB_LAUNCHED(ctx);
  return STRICTB200_OK;
}
