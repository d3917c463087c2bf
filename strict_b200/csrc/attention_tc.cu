// Causal GQA prefill attention on the tcgen05 tensor cores (head_dim 128, bf16).
// One block = 128 query positions of one head, 128 threads: thread r owns query row r, which is
// also lane r of tensor memory, so the softmax needs no shuffles.
// Per 128-key tile:
//   S = Q K^T        tcgen05.mma kind::f16, A = Q tile and B = K tile in shared memory (both
//                    K-major, two 64-dim halves of 128-byte-swizzled rows written by TMA),
//                    fp32 accumulator in tensor memory (128 columns)
//   softmax          every thread reads its row of S with tcgen05.ld (twice: maximum, then
//                    exponentials), keeps running maximum and sum, and writes P as TWO bf16
//                    terms (hi + lo by truncation, so that P.V matches an exact-softmax oracle
//                    to 2^-16)
//                    back to tensor memory with tcgen05.st (2 x 64 columns)
//   O += P V        tcgen05.mma with A = P from tensor memory and B = the V tile in shared
//                    memory, read MN-major (its rows are keys = the K dimension of this product),
//                    accumulating into the running output, which stays in tensor memory (128
//                    columns) for the whole block. P overwrites S in place (32 fp32 columns of a
//                    chunk become 16 columns of P hi and 16 of P lo), so a block needs 256 columns.
//   rescaling        the running output follows the running maximum lazily: a row is rescaled
//                    (read-modify-write of its 128 columns) only when its maximum grew by more
//                    than 2^8; otherwise it keeps the older reference maximum
// The K tile of the next step is requested as soon as S is complete, the V tile as soon as
// the previous P.V is complete, so the copies run under the softmax. Two blocks fit
// an SM (96 KB of shared memory, 256 tensor-memory columns each) and fill each other's gaps.
// Every mbarrier wait is bounded: on expiry the block records an error word in host-visible
// memory, stops, frees its tensor memory and returns.
#include <cstdlib>

#include "tcgen05.cuh"

using namespace tc;

namespace {

constexpr int D = 128;
constexpr int BQ = 128;   // query rows per block
constexpr int BKV = 128;  // keys per tile
constexpr float LOG2E = 1.4426950408889634f;

struct TcAttnArgs {
  const int32_t* lens;
  const int32_t* past;
  const int32_t* qstart;
  int S, Hq, Hkv, maxlen;
  float scale_log2;
  bf16* out;
  int* status;
  // keys of a layer with per-head keys rebuilt from latents (LatentPrefillArgs); unused by the GQA form
  const int32_t* koff;   // [B] row of the sequence's first key in the key and value arrays
  const int32_t* kpos0;  // [B] position of that key
  int window;            // keys a row sees, itself included
  int nks_q, nks_r;      // 16-wide reduction steps of the unrotated and of the rotated part
  int dv;                // value width
  int64_t ldo;           // row stride of out
  // heads with a sink and an output gate
  int sink;              // 1: the softmax denominator counts one more key, of score 0 and without a value
  const float* gate;     // [rows, Hq] factor of a head's output; may be null
};

__global__ void __launch_bounds__(128) attn_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                                              const __grid_constant__ CUtensorMap map_v, TcAttnArgs a) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t bar_q, bar_k, bar_v, bar_s, bar_o;
  __shared__ uint32_t tmem_base_slot;
  __shared__ int abort_flag;

  const int b = blockIdx.z, h = blockIdx.y, q0 = blockIdx.x * BQ;
  const int len = a.lens[b], pst = a.past ? a.past[b] : 0;
  const int n_new = len - pst;
  if (q0 >= n_new) return;  // whole block, before anything is allocated
  const int64_t row0 = a.qstart ? a.qstart[b] : (int64_t)b * a.S;
  const int hk = h / (a.Hq / a.Hkv);
  const int warp = threadIdx.x >> 5;
  const int kv_end = min(len, pst + q0 + BQ);  // last key any row of this block may see, exclusive
  const int ntiles = (kv_end + BKV - 1) / BKV;
  const int kv_row0 = (b * a.Hkv + hk) * a.maxlen;

  const uint32_t sQ = smem_u32(smem), sK = sQ + TILE_BYTES, sV = sK + TILE_BYTES;
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&bar_q), 1);
    mbar_init(smem_u32(&bar_k), 1);
    mbar_init(smem_u32(&bar_v), 1);
    mbar_init(smem_u32(&bar_s), 1);
    mbar_init(smem_u32(&bar_o), 1);
    abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_slot)), "r"(256u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_base_slot;
  const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
  const uint32_t tS = tmem, tO = tmem + 128;  // columns: S (then P hi/lo in place) and the running output

  if (threadIdx.x == 0) {
    mbar_expect_tx(smem_u32(&bar_q), TILE_BYTES);
    tma_load_2d(sQ, &map_q, h * D, (int)(row0 + q0), smem_u32(&bar_q));
    tma_load_2d(sQ + HALF_BYTES, &map_q, h * D + 64, (int)(row0 + q0), smem_u32(&bar_q));
    mbar_expect_tx(smem_u32(&bar_k), TILE_BYTES);
    tma_load_2d(sK, &map_k, 0, kv_row0, smem_u32(&bar_k));
    tma_load_2d(sK + HALF_BYTES, &map_k, 64, kv_row0, smem_u32(&bar_k));
    mbar_expect_tx(smem_u32(&bar_v), TILE_BYTES);
    tma_load_2d(sV, &map_v, 0, kv_row0, smem_u32(&bar_v));
    tma_load_2d(sV + HALF_BYTES, &map_v, 64, kv_row0, smem_u32(&bar_v));
  }

  // instruction descriptors: D = F32, A = B = BF16, M = 128, N = 128; B of P.V is MN-major
  constexpr uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(128 >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
  constexpr uint32_t idesc_pv = idesc_s | (1u << 16);

  float m_run = -INFINITY, l_run = 0.f;
  const int qpos = pst + q0 + (int)threadIdx.x;  // position of this thread's query row
  bool ok = true;

  for (int t = 0; t < ntiles; t++) {
    const uint32_t ph = (uint32_t)(t & 1);
    // ---- S = Q K^T (after the previous P.V has finished reading P and the V tile)
    if (threadIdx.x == 0) {
      bool good = true;
      if (t > 0) {
        good = mbar_wait(smem_u32(&bar_o), ph ^ 1);
        if (good) {
          mbar_expect_tx(smem_u32(&bar_v), TILE_BYTES);
          tma_load_2d(sV, &map_v, 0, kv_row0 + t * BKV, smem_u32(&bar_v));
          tma_load_2d(sV + HALF_BYTES, &map_v, 64, kv_row0 + t * BKV, smem_u32(&bar_v));
        }
      } else {
        good = mbar_wait(smem_u32(&bar_q), 0);
      }
      good = good && mbar_wait(smem_u32(&bar_k), ph);
      if (!good) { set_status(a.status, 7); abort_flag = 1; }
      else {
        tc_fence_after();
#pragma unroll
        for (int s = 0; s < 8; s++) {
          const uint32_t off = (uint32_t)((s >> 2) * HALF_BYTES + (s & 3) * 32);  // 16 dims = 32 bytes inside the 64-dim half
          tc_mma_ss(tS, desc_kmajor(sQ + off), desc_kmajor(sK + off), idesc_s, s ? 1u : 0u);
        }
        tc_commit(smem_u32(&bar_s));
      }
    }
    __syncthreads();
    if (*(volatile int*)&abort_flag) { ok = false; break; }
    if (!mbar_wait(smem_u32(&bar_s), ph)) { if (threadIdx.x == 0) set_status(a.status, 8); ok = false; break; }
    tc_fence_after();
    // the K tile is free: request the next one
    if (threadIdx.x == 0 && t + 1 < ntiles) {
      mbar_expect_tx(smem_u32(&bar_k), TILE_BYTES);
      tma_load_2d(sK, &map_k, 0, kv_row0 + (t + 1) * BKV, smem_u32(&bar_k));
      tma_load_2d(sK + HALF_BYTES, &map_k, 64, kv_row0 + (t + 1) * BKV, smem_u32(&bar_k));
    }
    // ---- softmax of this thread's row
    const int k0 = t * BKV;
    const int k_lim = min(len, qpos + 1) - k0;  // keys [0, k_lim) of the tile are visible to this row
    const bool full = k0 + BKV <= min(len, pst + q0 + 1);  // every row of the block sees the whole tile (block-uniform)
    float m_tile = -INFINITY;
#pragma unroll 1
    for (int c = 0; c < 4; c++) {
      uint32_t r[32];
      tc_ld32(tS + lane_base + (uint32_t)(c * 32), r);
      tc_wait_ld();
      if (full) {
#pragma unroll
        for (int j = 0; j < 32; j++) m_tile = fmaxf(m_tile, __uint_as_float(r[j]));
      } else {
#pragma unroll
        for (int j = 0; j < 32; j++)
          if (c * 32 + j < k_lim) m_tile = fmaxf(m_tile, __uint_as_float(r[j]));
      }
    }
    m_tile *= a.scale_log2;  // the scale is positive: the maximum commutes with it
    // The running output lives in tensor memory, so following the maximum costs a read-modify-write
    // of the row. It is only done when the maximum grew by more than 2^8 (the exponentials then
    // stay below 256, harmless for the two-term bf16 P and the fp32 sums); otherwise the row keeps
    // its older reference maximum, and the final division by the running sum is unchanged.
    const bool grow = m_tile > m_run + 8.0f;  // also true for the first tile (m_run = -inf)
    const float m_use = grow ? m_tile : m_run;
    const float corr = grow ? exp2f(m_run - m_use) : 1.0f;  // 0 for the first tile
    m_run = m_use;
    if (t > 0 && __any_sync(0xffffffffu, grow)) {
#pragma unroll 1
      for (int c = 0; c < 4; c++) {
        uint32_t r[32];
        tc_ld32(tO + lane_base + (uint32_t)(c * 32), r);
        tc_wait_ld();
#pragma unroll
        for (int j = 0; j < 32; j++) r[j] = __float_as_uint(__uint_as_float(r[j]) * corr);
        tc_st32(tO + lane_base + (uint32_t)(c * 32), r);
      }
    }
    float row_sum = 0.f;
#pragma unroll 1
    for (int c = 0; c < 4; c++) {
      uint32_t r[32];
      tc_ld32(tS + lane_base + (uint32_t)(c * 32), r);
      tc_wait_ld();
      uint32_t hi[16], lo[16];
#pragma unroll
      for (int j = 0; j < 16; j++) {
        const int kk = c * 32 + 2 * j;
        float p0 = ex2_approx(fmaf(__uint_as_float(r[2 * j]), a.scale_log2, -m_use));
        float p1 = ex2_approx(fmaf(__uint_as_float(r[2 * j + 1]), a.scale_log2, -m_use));
        if (!full) {
          if (kk >= k_lim) p0 = 0.f;
          if (kk + 1 >= k_lim) p1 = 0.f;
        }
        row_sum += p0 + p1;
        // two-term split by truncation: hi = the upper 16 bits of p, lo = the upper 16 bits of the
        // (exact) remainder; p - hi - lo < 2^-16 p, and no conversion instruction is needed
        const uint32_t b0 = __float_as_uint(p0), b1 = __float_as_uint(p1);
        hi[j] = __byte_perm(b0, b1, 0x7632);
        const uint32_t l0 = __float_as_uint(p0 - __uint_as_float(b0 & 0xFFFF0000u)), l1 = __float_as_uint(p1 - __uint_as_float(b1 & 0xFFFF0000u));
        lo[j] = __byte_perm(l0, l1, 0x7632);
      }
      // in place: the 32 fp32 columns of this chunk become 16 columns of P hi and 16 of P lo
      tc_st16(tS + lane_base + (uint32_t)(c * 32), hi);
      tc_st16(tS + lane_base + (uint32_t)(c * 32 + 16), lo);
    }
    tc_wait_st();
    l_run = l_run * corr + row_sum;
    tc_fence_before();
    __syncthreads();  // P of all rows is in tensor memory (and the rescaled O, if any)
    // ---- O += P V
    if (threadIdx.x == 0) {
      if (!mbar_wait(smem_u32(&bar_v), ph)) { set_status(a.status, 9); abort_flag = 1; }
      else {
        tc_fence_after();
#pragma unroll
        for (int s = 0; s < 8; s++) {
          // 16 keys = 16 rows of 128 bytes = 2048 bytes of the V tile = 8 packed columns of P hi (and of P lo)
          const uint64_t dv = desc_mnmajor(sV + (uint32_t)(s * 2048));
          const uint32_t pcol = (uint32_t)((s >> 1) * 32 + (s & 1) * 8);
          tc_mma_ts(tO, tS + pcol, dv, idesc_pv, (t | s) ? 1u : 0u);
          tc_mma_ts(tO, tS + pcol + 16, dv, idesc_pv, 1u);
        }
        tc_commit(smem_u32(&bar_o));
      }
    }
  }

  __syncthreads();
  if (*(volatile int*)&abort_flag) ok = false;
  if (ok && !mbar_wait(smem_u32(&bar_o), (uint32_t)((ntiles - 1) & 1))) { if (threadIdx.x == 0) set_status(a.status, 10); ok = false; }
  tc_fence_after();
  if (ok) {
    const bool live = q0 + (int)threadIdx.x < n_new;
    const float inv = 1.0f / l_run;
    bf16* dst = a.out + ((row0 + q0 + threadIdx.x) * a.Hq + h) * D;
#pragma unroll 1
    for (int c = 0; c < 4; c++) {
      uint32_t r[32];
      tc_ld32(tO + lane_base + (uint32_t)(c * 32), r);
      tc_wait_ld();
      if (live) {
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          uint4 w;
          w.x = f32_to_bf16_bits(__uint_as_float(r[i]) * inv) | (f32_to_bf16_bits(__uint_as_float(r[i + 1]) * inv) << 16);
          w.y = f32_to_bf16_bits(__uint_as_float(r[i + 2]) * inv) | (f32_to_bf16_bits(__uint_as_float(r[i + 3]) * inv) << 16);
          w.z = f32_to_bf16_bits(__uint_as_float(r[i + 4]) * inv) | (f32_to_bf16_bits(__uint_as_float(r[i + 5]) * inv) << 16);
          w.w = f32_to_bf16_bits(__uint_as_float(r[i + 6]) * inv) | (f32_to_bf16_bits(__uint_as_float(r[i + 7]) * inv) << 16);
          *(uint4*)(dst + c * 32 + i) = w;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(256u) : "memory");
  }
}

// ------------------------------------------------------------------ two query tiles per block
// The kernel above runs S -> softmax -> PV of a block strictly one after the other, so the tensor
// pipe idles during the softmax and the softmax threads idle during the MMAs (two blocks per SM
// hide part of it). Here one block owns TWO tiles of 128 query rows (A and B, 256 consecutive
// positions of one head) that share every K/V tile, with separate roles:
//   warps 0..7   softmax of tile A (its own 256 tensor-memory columns: S/P and O); row r = lane r is
//                served by two threads (warps 0..3 and 4..7) that own 64 of the 128 columns each
//                and exchange only the row maximum, so two warps per scheduler hide each
//                other's tensor-memory and exp2 latencies
//   warps 8..15  softmax of tile B (the other 256 columns), same split
//   warp 16      one lane issues all MMAs in ping-pong order (PV_A(t) S_A(t+1) PV_B(t) S_B(t+1)):
//                while the A threads run their softmax the tensor pipe works on tile B, and so on
//   warp 17      one lane issues the TMA copies into two-stage K and V rings
// The whole tensor memory (512 columns) and 193 KB of shared memory: one block per SM.
//
// The tile shapes are parameters: a query/key row is QA 64-dim atoms of its own head followed by RA
// atoms that all heads share on the key side (the rotated part of latent attention; its own array
// and copy), a value row VA atoms. Head widths that do not fill their last atom are cut by the
// tensor maps (dims x heads x rows), which fill with zeros; reduction steps beyond the width are not
// issued. KST = stages of the K ring. WIN adds a sliding window: the walk over the key tiles begins
// at the first tile any row of the block sees, and rows drop keys below their own window.
//
// PLAIN: grouped heads of 128 dims, output rows [Hq, 128]. Otherwise the output goes to rows of ldo with heads of dv dims, and
// without a shared part (RA = 0: grouped heads over cache rows of 64 * QA dims) the sink and the gate of TcAttnArgs apply.
constexpr int TC2_THREADS = 576;  // 16 softmax warps + MMA warp + TMA warp

template <int QA, int RA, int VA, int KST>
constexpr int tc2_tile_bytes() { return (2 * (QA + RA) + KST * (QA + RA) + 2 * VA) * HALF_BYTES; }

template <int QA, int RA, int VA, int KST, bool WIN, bool PLAIN>
__global__ void __launch_bounds__(TC2_THREADS) attn_prefill_tc2_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_qr,
                                                                      const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_kr,
                                                                      const __grid_constant__ CUtensorMap map_v, TcAttnArgs a) {
  constexpr int QK_BYTES = (QA + RA) * HALF_BYTES, V_BYTES = VA * HALF_BYTES;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t bar_q, k_full[KST], k_empty[KST], v_full[2], v_empty[2], bar_s[2], bar_p[2], bar_o[2];
  __shared__ uint32_t tmem_base_slot;
  __shared__ float x_max[2][2][BQ], x_sum[2][BQ];  // [tile][column half][row]: exchange between the two threads of a row

  const int b = blockIdx.z, h = blockIdx.y, q0 = blockIdx.x * 2 * BQ;
  const int len = a.lens[b], pst = a.past ? a.past[b] : 0;
  const int n_new = len - pst;
  if (q0 >= n_new) return;  // whole block, before anything is allocated
  const int64_t row0 = a.qstart ? a.qstart[b] : (int64_t)b * a.S;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // position and row of the first key of the walk, and the head coordinate of the keys
  int kp0 = 0, kv_row0, kh = 0;
  if (RA) {
    kh = h;
    kp0 = a.kpos0[b];
    if (WIN) kp0 += max(0, pst + q0 - a.window + 1 - kp0) / BKV * BKV;
    kv_row0 = a.koff[b] + kp0 - a.kpos0[b];
  } else {
    kv_row0 = (b * a.Hkv + h / (a.Hq / a.Hkv)) * a.maxlen;
  }
  // K/V tiles each query tile needs (tile B is empty when the sequence ends inside tile A)
  int nt[2];
  nt[0] = (min(len, pst + q0 + BQ) - kp0 + BKV - 1) / BKV;
  nt[1] = q0 + BQ < n_new ? (min(len, pst + q0 + 2 * BQ) - kp0 + BKV - 1) / BKV : 0;
  const int ntiles = max(nt[0], nt[1]);

  const uint32_t sQ = smem_u32(smem), sK = sQ + 2 * QK_BYTES, sV = sK + KST * QK_BYTES;
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&bar_q), 1);
    for (int i = 0; i < 2; i++) {
      if (i < KST) { mbar_init(smem_u32(&k_full[i]), 1); mbar_init(smem_u32(&k_empty[i]), 1); }
      mbar_init(smem_u32(&v_full[i]), 1); mbar_init(smem_u32(&v_empty[i]), 1);
      mbar_init(smem_u32(&bar_s[i]), 1); mbar_init(smem_u32(&bar_p[i]), 2 * BQ); mbar_init(smem_u32(&bar_o[i]), 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 16) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_slot)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_base_slot;
  constexpr uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(128 >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
  constexpr uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(VA * 64 >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);

  if (warp == 17) {
    // ---- TMA producer
    if (lane == 0) {
      mbar_expect_tx(smem_u32(&bar_q), (nt[1] ? 2 : 1) * QK_BYTES);
      for (int w = 0; w < (nt[1] ? 2 : 1); w++) {
        for (int i = 0; i < QA; i++) tma_load_3d(sQ + w * QK_BYTES + i * HALF_BYTES, &map_q, i * 64, h, (int)(row0 + q0 + w * BQ), smem_u32(&bar_q));
        for (int i = 0; i < RA; i++) tma_load_3d(sQ + w * QK_BYTES + (QA + i) * HALF_BYTES, &map_qr, i * 64, h, (int)(row0 + q0 + w * BQ), smem_u32(&bar_q));
      }
      for (int t = 0; t < ntiles; t++) {
        const int kst = t % KST, vst = t & 1;
        const int row = kv_row0 + t * BKV;
        if (t >= KST && !mbar_wait(smem_u32(&k_empty[kst]), (uint32_t)((t / KST) & 1) ^ 1)) { set_status(a.status, 11); break; }
        mbar_expect_tx(smem_u32(&k_full[kst]), QK_BYTES);
        for (int i = 0; i < QA; i++) tma_load_3d(sK + kst * QK_BYTES + i * HALF_BYTES, &map_k, i * 64, kh, row, smem_u32(&k_full[kst]));
        for (int i = 0; i < RA; i++) tma_load_3d(sK + kst * QK_BYTES + (QA + i) * HALF_BYTES, &map_kr, i * 64, 0, row, smem_u32(&k_full[kst]));
        if (t >= 2 && !mbar_wait(smem_u32(&v_empty[vst]), (uint32_t)((t >> 1) & 1) ^ 1)) { set_status(a.status, 12); break; }
        mbar_expect_tx(smem_u32(&v_full[vst]), V_BYTES);
        for (int i = 0; i < VA; i++) tma_load_3d(sV + vst * V_BYTES + i * HALF_BYTES, &map_v, i * 64, kh, row, smem_u32(&v_full[vst]));
      }
    }
  } else if (warp == 16) {
    // ---- MMA issue, ping-pong between the two query tiles: S_A(0) S_B(0), then per K/V tile
    // PV_A(t) S_A(t+1) PV_B(t) S_B(t+1). The tensor pipe runs them in program order, so while
    // the A threads are in the softmax of step t+1 the pipe works on tile B, and vice versa.
    if (lane == 0) {
      auto issue_s = [&](int w, int t) {
        const int st = t % KST;
        const uint32_t tS = tmem + (uint32_t)(w * 256);
#pragma unroll
        for (int s = 0; s < 4 * (QA + RA); s++) {
          if (RA && (s < 4 * QA ? s >= a.nks_q : s - 4 * QA >= a.nks_r)) continue;  // beyond the head's width
          const uint32_t off = (uint32_t)((s >> 2) * HALF_BYTES + (s & 3) * 32);
          tc_mma_ss(tS, desc_kmajor(sQ + w * QK_BYTES + off), desc_kmajor(sK + st * QK_BYTES + off), idesc_s, s ? 1u : 0u);
        }
        tc_commit(smem_u32(&bar_s[w]));
      };
      bool good = mbar_wait(smem_u32(&bar_q), 0) && mbar_wait(smem_u32(&k_full[0]), 0);
      if (good) {
        tc_fence_after();
        for (int w = 0; w < 2; w++)
          if (nt[w] > 0) issue_s(w, 0);
        tc_commit(smem_u32(&k_empty[0]));
      }
      for (int t = 0; t < ntiles && good; t++) {
        const int st = t & 1;
        const uint32_t rph = (uint32_t)((t >> 1) & 1), ph = (uint32_t)(t & 1);
        good = mbar_wait(smem_u32(&v_full[st]), rph);
        bool k_next_ready = false;
        for (int w = 0; w < 2 && good; w++) {
          if (t < nt[w]) {
            good = mbar_wait(smem_u32(&bar_p[w]), ph);  // P (and the rescaled O) of this step are in tensor memory
            if (!good) break;
            tc_fence_after();
            const uint32_t tS = tmem + (uint32_t)(w * 256), tO = tS + 128;
#pragma unroll
            for (int s = 0; s < 8; s++) {
              const uint64_t dv = desc_mnmajor(sV + st * V_BYTES + (uint32_t)(s * 2048));
              const uint32_t pcol = (uint32_t)((s >> 1) * 32 + (s & 1) * 8);
              tc_mma_ts(tO, tS + pcol, dv, idesc_pv, (t | s) ? 1u : 0u);
              tc_mma_ts(tO, tS + pcol + 16, dv, idesc_pv, 1u);
            }
            tc_commit(smem_u32(&bar_o[w]));
          }
          if (t + 1 < nt[w]) {
            if (!k_next_ready) {
              good = mbar_wait(smem_u32(&k_full[(t + 1) % KST]), (uint32_t)(((t + 1) / KST) & 1));
              if (!good) break;
              tc_fence_after();
              k_next_ready = true;
            }
            issue_s(w, t + 1);
          }
        }
        if (!good) break;
        tc_commit(smem_u32(&v_empty[st]));                               // both PV products have read the V tile
        if (t + 1 < ntiles) tc_commit(smem_u32(&k_empty[(t + 1) % KST]));  // both S products of the next step have read its K tile
      }
      if (!good) set_status(a.status, 13);
    }
  } else {
    // ---- softmax warpgroups: w = 0 (tile A) or 1 (tile B)
    const int w = warp >> 3, half = (warp >> 2) & 1, row = (int)threadIdx.x & (BQ - 1);
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    auto wg_sync = [&]() { asm volatile("bar.sync %0, 256;" ::"r"(1 + w) : "memory"); };  // the 256 threads of this tile
    const uint32_t tS = tmem + (uint32_t)(w * 256), tO = tS + 128;
    const int qw = q0 + w * BQ;           // first query row of this tile
    const int qpos = pst + qw + row;
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int t = 0; t < nt[w]; t++) {
      const uint32_t ph = (uint32_t)(t & 1);
      if (!mbar_wait(smem_u32(&bar_s[w]), ph)) { if (row == 0) set_status(a.status, 14); ok = false; break; }
      tc_fence_after();
      const int k0 = kp0 + t * BKV;
      const int k_lim = min(len, qpos + 1) - k0;
      const int k_low = WIN ? qpos - a.window + 1 - k0 : 0;  // keys [k_low, k_lim) of the tile are visible to this row
      const bool full = k0 + BKV <= min(len, pst + qw + 1) && (!WIN || pst + qw + BQ - a.window <= k0);
      float m_tile = -INFINITY;
#pragma unroll 1
      for (int c = 2 * half; c < 2 * half + 2; c++) {
        uint32_t r[32];
        tc_ld32(tS + lane_base + (uint32_t)(c * 32), r);
        tc_wait_ld();
        if (full) {
#pragma unroll
          for (int j = 0; j < 32; j++) m_tile = fmaxf(m_tile, __uint_as_float(r[j]));
        } else {
#pragma unroll
          for (int j = 0; j < 32; j++)
            if (c * 32 + j < k_lim && (!WIN || c * 32 + j >= k_low)) m_tile = fmaxf(m_tile, __uint_as_float(r[j]));
        }
      }
      x_max[w][half][row] = m_tile;
      wg_sync();
      m_tile = fmaxf(x_max[w][0][row], x_max[w][1][row]) * a.scale_log2;
      const bool grow = m_tile > m_run + 8.0f;  // lazy rescaling, as in the kernel above
      const float m_use = grow ? m_tile : m_run;
      const float corr = grow ? exp2f(m_run - m_use) : 1.0f;
      m_run = m_use;
      if (t > 0 && __any_sync(0xffffffffu, grow)) {
        // the previous PV of this tile must have finished writing O
        if (!mbar_wait(smem_u32(&bar_o[w]), ph ^ 1)) { if (row == 0) set_status(a.status, 15); ok = false; break; }
        tc_fence_after();
#pragma unroll 1
        for (int c = VA * half; c < VA * half + VA; c++) {
          uint32_t r[32];
          tc_ld32(tO + lane_base + (uint32_t)(c * 32), r);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; j++) r[j] = __float_as_uint(__uint_as_float(r[j]) * corr);
          tc_st32(tO + lane_base + (uint32_t)(c * 32), r);
        }
      }
      float row_sum = 0.f;
#pragma unroll 1
      for (int c = 2 * half; c < 2 * half + 2; c++) {
        uint32_t r[32];
        tc_ld32(tS + lane_base + (uint32_t)(c * 32), r);
        tc_wait_ld();
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int j = 0; j < 16; j++) {
          const int kk = c * 32 + 2 * j;
          float p0 = ex2_approx(fmaf(__uint_as_float(r[2 * j]), a.scale_log2, -m_use));
          float p1 = ex2_approx(fmaf(__uint_as_float(r[2 * j + 1]), a.scale_log2, -m_use));
          if (!full) {
            if (kk >= k_lim || (WIN && kk < k_low)) p0 = 0.f;
            if (kk + 1 >= k_lim || (WIN && kk + 1 < k_low)) p1 = 0.f;
          }
          row_sum += p0 + p1;
          const uint32_t b0 = __float_as_uint(p0), b1 = __float_as_uint(p1);
          hi[j] = __byte_perm(b0, b1, 0x7632);
          const uint32_t l0 = __float_as_uint(p0 - __uint_as_float(b0 & 0xFFFF0000u)), l1 = __float_as_uint(p1 - __uint_as_float(b1 & 0xFFFF0000u));
          lo[j] = __byte_perm(l0, l1, 0x7632);
        }
        tc_st16(tS + lane_base + (uint32_t)(c * 32), hi);
        tc_st16(tS + lane_base + (uint32_t)(c * 32 + 16), lo);
      }
      tc_wait_st();
      l_run = l_run * corr + row_sum;
      tc_fence_before();
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&bar_p[w])) : "memory");
      wg_sync();  // x_max is rewritten in the next step
    }
    if (ok && nt[w] > 0) {
      if (!mbar_wait(smem_u32(&bar_o[w]), (uint32_t)((nt[w] - 1) & 1))) { if (row == 0) set_status(a.status, 16); ok = false; }
      tc_fence_after();
    }
    if (half) x_sum[w][row] = l_run;  // the two threads of a row saw the same maxima: their sums add
    wg_sync();
    if (!half) x_sum[w][row] += l_run;
    wg_sync();
    if (ok && nt[w] > 0) {
      const bool live = qw + row < n_new;
      float inv;
      if constexpr (!PLAIN && !RA) {
        inv = 1.0f / (x_sum[w][row] + (a.sink ? exp2f(-m_run) : 0.f));  // the sums are relative to 2^m_run
        if (a.gate && live) inv *= a.gate[(row0 + qw + row) * a.Hq + h];
      } else {
        inv = 1.0f / x_sum[w][row];
      }
      bf16* dst = !PLAIN ? a.out + (row0 + qw + row) * a.ldo + (int64_t)h * a.dv : a.out + ((row0 + qw + row) * a.Hq + h) * D;
      const bool whole = PLAIN || (((a.dv & 7) == 0) && ((a.ldo & 7) == 0));
#pragma unroll 1
      for (int c = VA * half; c < VA * half + VA; c++) {
        uint32_t r[32];
        tc_ld32(tO + lane_base + (uint32_t)(c * 32), r);
        tc_wait_ld();
        if (live && !whole) {
#pragma unroll
          for (int i = 0; i < 32; i++)
            if (c * 32 + i < a.dv) dst[c * 32 + i] = __float2bfloat16_rn(__uint_as_float(r[i]) * inv);
        } else if (live) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (!PLAIN && c * 32 + i >= a.dv) break;
            uint4 wv;
            wv.x = f32_to_bf16_bits(__uint_as_float(r[i]) * inv) | (f32_to_bf16_bits(__uint_as_float(r[i + 1]) * inv) << 16);
            wv.y = f32_to_bf16_bits(__uint_as_float(r[i + 2]) * inv) | (f32_to_bf16_bits(__uint_as_float(r[i + 3]) * inv) << 16);
            wv.z = f32_to_bf16_bits(__uint_as_float(r[i + 4]) * inv) | (f32_to_bf16_bits(__uint_as_float(r[i + 5]) * inv) << 16);
            wv.w = f32_to_bf16_bits(__uint_as_float(r[i + 6]) * inv) | (f32_to_bf16_bits(__uint_as_float(r[i + 7]) * inv) << 16);
            *(uint4*)(dst + c * 32 + i) = wv;
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 16) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
  }
}

template <int QA, int RA, int VA, int KST, bool WIN, bool PLAIN>
int launch_tc2(strictb200_ctx* ctx, const CUtensorMap* m, const TcAttnArgs& a, int B, int S) {
  const size_t smem = tc2_tile_bytes<QA, RA, VA, KST>() + 1024;
  static SbDeviceOnce once;  // one per instantiation
  SB_CUDA(once.run(ctx->device, [&] { return cudaFuncSetAttribute(attn_prefill_tc2_kernel<QA, RA, VA, KST, WIN, PLAIN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); }));
  dim3 grid((unsigned)((S + 2 * BQ - 1) / (2 * BQ)), (unsigned)a.Hq, (unsigned)B);
  attn_prefill_tc2_kernel<QA, RA, VA, KST, WIN, PLAIN><<<grid, TC2_THREADS, smem, ctx->stream>>>(m[0], m[1], m[2], m[3], m[4], a);
  SB_LAUNCHED(ctx);
  return STRICTB200_OK;
}

}  // namespace

// q, out: [q_rows, Hq, 128]; caches [B, Hkv, maxlen, 128]. ERR_UNSUPPORTED for shapes this kernel does not take.
int k_attn_prefill_tc(strictb200_ctx* ctx, const bf16* q, const bf16* kc, const bf16* vc, const int32_t* lens, const int32_t* past,
                      const int32_t* qstart, int B, int S, int64_t q_rows, int Hq, int Hkv, int maxlen, float scale, bf16* out) {
  if (Hq > 65535 || B > 65535 || Hq % Hkv) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "attention: too many heads or sequences");
  if ((int64_t)B * Hkv * maxlen > INT32_MAX || q_rows > INT32_MAX) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "attention: cache too large for 32-bit tile coordinates");
  if (((uintptr_t)q | (uintptr_t)kc | (uintptr_t)vc) & 15) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "attention: operands must be 16-byte aligned");
  TcAttnArgs a{lens, past, qstart, S, Hq, Hkv, maxlen, scale * LOG2E, out, ctx->d_status, nullptr, nullptr, 0, 0, 0, D, (int64_t)Hq * D, 0, nullptr};
  // two query tiles per block (ping-pong) from 256 new tokens per sequence on; the attn_tc option (1 / 2) forces a kernel
  const int forced = ctx->opt.attn_tc;
  if (forced == 2 || (forced != 1 && S >= 2 * BQ)) {
    CUtensorMap m[5];
    SB_TRY(make_map3(&m[0], q, D, Hq, q_rows, D, (int64_t)Hq * D));
    SB_TRY(make_map3(&m[2], kc, D, 1, (int64_t)B * Hkv * maxlen, D, D));
    SB_TRY(make_map3(&m[4], vc, D, 1, (int64_t)B * Hkv * maxlen, D, D));
    m[1] = m[0]; m[3] = m[2];
    return launch_tc2<2, 0, 2, 2, false, true>(ctx, m, a, B, S);
  }
  CUtensorMap mq, mk, mv;
  SB_TRY(make_map(&mq, q, q_rows, (int64_t)Hq * D, (int64_t)Hq * D));
  SB_TRY(make_map(&mk, kc, (int64_t)B * Hkv * maxlen, D, D));
  SB_TRY(make_map(&mv, vc, (int64_t)B * Hkv * maxlen, D, D));
  const size_t smem = 3 * TILE_BYTES + 1024;
  static SbDeviceOnce once;
  SB_CUDA(once.run(ctx->device, [&] { return cudaFuncSetAttribute(attn_prefill_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); }));
  dim3 grid((unsigned)((S + BQ - 1) / BQ), (unsigned)Hq, (unsigned)B);
  attn_prefill_tc_kernel<<<grid, 128, smem, ctx->stream>>>(mq, mk, mv, a);
  SB_LAUNCHED(ctx);
  return STRICTB200_OK;
}

// Grouped heads over cache rows of row_dims = 64 or 128 dims (narrower heads are filled up with zeros), values of vdim dims.
int k_attn_prefill_heads(strictb200_ctx* ctx, const HeadPrefillArgs& p) {
  const int HD = p.row_dims;
  if (HD != 64 && HD != 128) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "prefill attention: rows of 64 or 128 dims");
  if (p.H > 65535 || p.B > 65535 || p.H % p.Hkv || p.q_rows > INT32_MAX || (int64_t)p.B * p.Hkv * p.maxlen > INT32_MAX)
    return sb_fail(STRICTB200_ERR_UNSUPPORTED, "prefill attention: too many heads, sequences or rows");
  TcAttnArgs a{};
  a.lens = p.lens; a.past = p.past; a.qstart = p.qstart; a.S = p.S; a.Hq = p.H; a.Hkv = p.Hkv; a.maxlen = p.maxlen;
  a.scale_log2 = p.scale * LOG2E; a.out = p.out; a.status = ctx->d_status; a.dv = p.vdim; a.ldo = p.ldo; a.sink = p.sink; a.gate = p.gate;
  CUtensorMap m[5];
  SB_TRY(make_map3(&m[0], p.q, HD, p.H, p.q_rows, HD, (int64_t)p.H * HD));
  SB_TRY(make_map3(&m[2], p.k, HD, 1, (int64_t)p.B * p.Hkv * p.maxlen, HD, HD));
  SB_TRY(make_map3(&m[4], p.v, HD, 1, (int64_t)p.B * p.Hkv * p.maxlen, HD, HD));
  m[1] = m[0]; m[3] = m[2];
  return HD == 64 ? launch_tc2<1, 0, 1, 2, false, false>(ctx, m, a, p.B, p.S) : launch_tc2<2, 0, 2, 2, false, false>(ctx, m, a, p.B, p.S);
}

bool sb_latent_prefill_fits(int dim, int rot, int vdim) { return dim <= 128 && rot <= 64 && vdim <= 128; }

int k_attn_prefill_latent(strictb200_ctx* ctx, const LatentPrefillArgs& p) {
  if (!sb_latent_prefill_fits(p.dim, p.rot, p.vdim)) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "latent prefill attention: head too wide for the tensor-core kernel");
  if (p.H > 65535 || p.B > 65535 || p.q_rows > INT32_MAX || p.k_rows > INT32_MAX)
    return sb_fail(STRICTB200_ERR_UNSUPPORTED, "latent prefill attention: too many heads, sequences or rows");
  TcAttnArgs a{};
  a.lens = p.lens; a.past = p.past; a.qstart = p.qstart; a.S = p.S; a.Hq = p.H; a.Hkv = p.H;
  a.scale_log2 = p.scale * LOG2E; a.out = p.out; a.status = ctx->d_status;
  a.koff = p.koff; a.kpos0 = p.kpos0; a.window = p.window; a.nks_q = (p.dim + 15) / 16; a.nks_r = (p.rot + 15) / 16; a.dv = p.vdim; a.ldo = p.ldo;
  CUtensorMap m[5];
  SB_TRY(make_map3(&m[0], p.q, p.dim, p.H, p.q_rows, p.q_head, p.q_head * p.H));
  SB_TRY(make_map3(&m[1], p.q + p.q_rot, p.rot, p.H, p.q_rows, p.q_head, p.q_head * p.H));
  SB_TRY(make_map3(&m[2], p.k, p.dim, p.H, p.k_rows, p.k_head, p.ldk));
  SB_TRY(make_map3(&m[3], p.k_rot, p.rot, 1, p.k_rows, p.ld_rot, p.ld_rot));
  SB_TRY(make_map3(&m[4], p.v, p.vdim, p.H, p.k_rows, p.v_head, p.ldk));
  const int S = p.S, B = p.B;
#define LATENT_TC2(QA, VA, KST) return p.window > 0 ? launch_tc2<QA, 1, VA, KST, true, false>(ctx, m, a, B, S) : launch_tc2<QA, 1, VA, KST, false, false>(ctx, m, a, B, S)
  if (p.dim <= 64) {
    if (p.vdim <= 64) LATENT_TC2(1, 1, 2);
    LATENT_TC2(1, 2, 2);
  }
  if (p.vdim <= 64) LATENT_TC2(2, 1, 1);
  LATENT_TC2(2, 2, 1);  // three 64-dim atoms per query and key row: one stage of keys is what shared memory leaves
#undef LATENT_TC2
}
