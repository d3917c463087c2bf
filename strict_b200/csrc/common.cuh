// Internal declarations shared by the translation units of libstrictb200.so.
#pragma once
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_fp8.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <mutex>
#include <string>
#include <utility>

#include "../../include/strictb200.h"

struct TpState;     // tp.cpp

// All-reduce over peer memory (tp.cpp): every rank owns a buffer that all ranks of the box map
// (CUDA IPC). Passed to kernels by value. Two exchanges use it:
//   row-granular (the decode step's default): the row kernel that consumes the sum pushes each of
//     its values into the peers' buffers as one word whose two lowest mantissa bits carry the row's
//     epoch modulo 4, and polls its own buffer until the words of every peer carry the current tag
//     (row_data, row_epoch); sums are taken over the values with those two bits cleared;
//   whole-result (shapes the row exchange does not take): a publish kernel writes the rank's fp32
//     partial result into its own buffer and raises an epoch flag in every peer's buffer; the
//     consumer waits for all flags and adds the ranks' data in rank order with plain peer loads
//     (data, flags, epoch, done).
// Every wait is bounded by wait_limit polls; on expiry the kernel sets *status and goes on.
struct TpCommDev {
  float* data[8];   // rank r's data area, two epoch parities of max_elems floats each
  int* flags[8];    // rank r's flag area: flags[parity * 8 + source rank] = last epoch published
  int* epoch;       // this rank's epoch counter (device memory, advanced by the publish kernel)
  unsigned* done;   // this rank's block counter of the publish kernel
  int* status;      // host-visible error word
  int world, rank;
  long long max_elems;
  // Row-granular variant (the row kernel itself exchanges the sums): every value is pushed into
  // the peers' buffers as a word that carries its epoch tag, so a word validates itself and
  // neither fences nor separate flags are needed.
  float* row_data[8];   // rank r's packet area: [parity][source rank] areas of 2 * row_elems words (the first row_elems in use)
  int* row_epoch;       // this rank's per-row epoch counters (device memory, one writer per row)
  long long row_elems;  // values per (parity, source rank)
  int max_rows;
  unsigned wait_limit;  // polls before a wait gives up (the context's wait_limit option, copied at launch)
};
struct SbProfiler;  // model.cu
void sb_prof_split(strictb200_ctx*, int cls);  // model.cu: inside a profiled call, the following launches count for class `cls`

// Switches of a context. Each is read once from the environment (STRICTB200_<NAME IN CAPITALS>)
// when the context is created and can be changed afterwards with strictb200_set_option; no
// launch path reads the environment. -1 stands for the library's own choice.
struct SbOptions {
  int pdl = 1;                 // launch the decode-path kernels with programmatic dependent launch
  int attn_tc = -1;            // prefill attention: 0 mma.sync, 1 tcgen05 one query tile per block, 2 two tiles per block
  int gemm_pair = 1;           // many-token GEMM on SM pairs (0: the one-SM persistent kernel)
  int prefetch = 1;            // GEMMs request their first ring of weight tiles before the dependency wait
  int deep_ring = 1;           // few-token GEMM: a ring that fills the SM when the grid is one block per SM
  int attn_blocks_per_sm = 0;  // >0: size decode-attention key chunks for that many blocks per SM
  int split_target = 0;        // >0: blocks a few-token GEMM's K splits aim at
  int tp_two_shot = -1;        // fused all-reduce: 0 one shot, 1 two shots
  int wait_limit = 1 << 22;    // polls of a cross-rank wait before the kernel gives up and sets the error word
  int prefill_chunk = 16384;   // token rows per prefill chunk
  int fuse_rope = 0;           // decode step: QK-norm, RoPE and the cache append inside the attention kernel (bit-identical; measured no faster)
  int row_cluster = 4;         // blocks (one cluster) per row of the decode row kernels, where the row has 1024 columns per block; 0 or 1 = one block per row
  int attn_prefetch = 1;       // decode attention starts to load its first key/value tiles before the dependency wait
  int blur_rows = 0;           // rows of the image per block of the blur kernel; 0 = chosen from the image and the grid
  int host_timeout_ms = 0;     // >0: a synchronising call gives up after this long, aborts the NCCL communicator and returns ERR_TIMEOUT
};

// One-time set-up that belongs to a device (function attributes are set per device): run(device, f)
// calls f the first time it is reached for that device, under a lock, and again on a later call
// if it failed. Contexts on different devices, driven from different threads, each get their turn.
struct SbDeviceOnce {
  std::mutex mu;
  bool done[64] = {};
  template <typename F>
  cudaError_t run(int device, F&& f) {
    if (device < 0 || device >= 64) return f();
    std::lock_guard<std::mutex> lock(mu);
    if (done[device]) return cudaSuccess;
    cudaError_t e = f();
    if (e == cudaSuccess) done[device] = true;
    return e;
  }
};

struct strictb200_ctx {
  int device = 0;
  int sm_count = 148;
  cudaStream_t stream = nullptr;
  cudaEvent_t ev0 = nullptr, ev1 = nullptr;
  uint64_t launches = 0;
  // scratch for op-level entry points (quantised activations, split partials)
  void* ws = nullptr;
  size_t ws_bytes = 0;
  uint64_t rec_launches0 = 0;  // launch counter when a recording began
  void* ws2 = nullptr;  // second scratch (split-K partial results of the stand-alone GEMM entry)
  size_t ws2_bytes = 0;
  void* flush_buf = nullptr;
  size_t flush_bytes = 0;
  int tp_world = 1, tp_rank = 0;
  TpState* tp = nullptr;
  SbProfiler* prof = nullptr;
  int* h_status = nullptr;  // pinned, device-visible error word written by kernels whose bounded waits expired
  int* d_status = nullptr;
  void* gemm_ws = nullptr;  // stream-K tile counters + partial tiles of the tensor-memory GEMM
  size_t gemm_count_bytes = 0, gemm_part_bytes = 0;
  SbOptions opt;
  unsigned long long* trace_rec = nullptr;  // armed trace (strictb200_trace_begin): records, counter, capacity
  unsigned int* trace_count = nullptr;
  unsigned int trace_capacity = 0;
  // scratch of the prefill chunks (activations of up to opt.prefill_chunk token rows), grow-only
  void* prefill_ws = nullptr;
  size_t prefill_ws_bytes = 0;
  uint64_t ws_generation = 0;  // advanced whenever a scratch buffer is re-allocated (recorded sequences check it)
};

void sb_set_error(const std::string& msg);
int sb_fail(int code, const std::string& msg);
// Waits for the context's stream. Under tensor parallelism it also polls NCCL's asynchronous error
// state (a failed peer or link) and, with the host_timeout_ms option, gives up after that long; in
// both cases the communicator is aborted so that its kernels leave the GPU, and the call returns
// ERR_NCCL / ERR_TIMEOUT instead of hanging.
int sb_sync(strictb200_ctx* ctx, const char* what);
int sb_check_status(strictb200_ctx* ctx, const char* what);  // after a stream synchronise: ERR_TIMEOUT if a kernel's wait expired
int sb_ws(strictb200_ctx* ctx, size_t bytes, void** out);  // grow-only context scratch
int sb_ws2(strictb200_ctx* ctx, size_t bytes, void** out);  // a second one, for calls that already hold the first

#define SB_CUDA(expr)                                                                          \
  do {                                                                                         \
    cudaError_t _e = (expr);                                                                   \
    if (_e != cudaSuccess)                                                                     \
      return sb_fail(_e == cudaErrorMemoryAllocation ? STRICTB200_ERR_OOM : STRICTB200_ERR_CUDA, \
                     std::string(#expr) + ": " + cudaGetErrorString(_e));                      \
  } while (0)
#define SB_TRY(expr)            \
  do {                          \
    int _s = (expr);            \
    if (_s != STRICTB200_OK) return _s; \
  } while (0)
#define SB_REQUIRE(cond, msg) \
  do {                        \
    if (!(cond)) return sb_fail(STRICTB200_ERR_INVALID_ARG, std::string(msg) + " (" #cond ")"); \
  } while (0)
#define SB_ENTER(ctx)                                                  \
  do {                                                                 \
    if (!(ctx)) return sb_fail(STRICTB200_ERR_INVALID_ARG, "null context"); \
    SB_CUDA(cudaSetDevice((ctx)->device));                             \
  } while (0)
// after a kernel launch
#define SB_LAUNCHED(ctx)          \
  do {                            \
    (ctx)->launches++;            \
    SB_CUDA(cudaGetLastError());  \
  } while (0)

// ------------------------------------------------------------------ launchers (internal API)
// Every launcher enqueues on ctx->stream and returns a status.
typedef __nv_bfloat16 bf16;

// elementwise.cu
int k_ew_binary(strictb200_ctx*, int op, const float* a, const float* b, float* out, int64_t n);
int k_ew_program(strictb200_ctx*, const int32_t* h_code, int n_instr, const float* const* h_arrays, int n_arrays,
                 const float* h_scalars, int n_scalars, const float* h_consts, int n_consts, float* out, int64_t n);
int k_ew_program2(strictb200_ctx*, const int32_t* h_code, int n_instr, const float* const* h_arrays, int n_arrays,
                  const float* h_scalars, int n_scalars, const float* h_consts, int n_consts, float* out, int64_t n);
// gen.cu
int k_gen_normal_f32(strictb200_ctx*, uint64_t key, int64_t first, int64_t count, float std_, float* out);
int k_gen_normal_bf16(strictb200_ctx*, uint64_t key, int64_t first, int64_t count, float std_, bf16* out);
int k_gen_tokens(strictb200_ctx*, uint64_t key, int64_t count, uint32_t range, int32_t* out);
int k_gen_weight_e4m3(strictb200_ctx*, uint64_t key, int64_t row0, int64_t rows, int64_t K, int64_t col0, int64_t cols,
                      float std_, uint8_t* q, int64_t ldq, float* scale);
uint64_t sb_stream_key(uint64_t seed, uint64_t tensor);
// norm.cu
// Activations enter the FP8 GEMMs as two E4M3 terms, x = s*(hi + lo/16) with s a power of two.
// Row layout of the split buffer: tokens in groups of 8; group g occupies rows [16g, 16g+16):
// 8 hi rows then 8 lo rows, so that the hi and lo accumulators of a token land in the same
// thread (mma.sync n-tile pairs) / adjacent accumulator columns (tensor memory).
inline int64_t sb_qrows(int64_t M) { return 16 * ((M + 7) / 8); }
int k_quantize_rows(strictb200_ctx*, const bf16* x, int64_t M, int64_t K, int64_t ldx, uint8_t* q, float* scale);
// Single-term absmax/448 quantisation of weight rows (the tied LM head).
int k_quantize_weight_rows(strictb200_ctx*, const bf16* x, int64_t M, int64_t K, int64_t ldx, uint8_t* q, float* scale);
// Row op of the residual stream. For every token row:
//   y_in  = part ? sum over groups g of (sum over splits s of part[g][s][row]) * sx[g][row] * sw[col]   (fp32)
//         : x_f32 ? x_f32 : x_in (bf16)
//   resid = residual_f32 ? residual_f32 + y_in (fp32, stored back)
//         : residual ? bf16(residual + y_in) (stored back) : y_in
//   n     = bf16((resid * r) * gain) ; written as bf16 (y) and/or as the two-term E4M3 split (q, qscale)
struct RowNormArgs {
  const float* x_f32 = nullptr;      // [M,d] fp32 input (e.g. after an all-reduce)
  const bf16* x_in = nullptr;        // [M,d] (used when part and x_f32 are null)
  const float* part = nullptr;       // [groups][splits][M,d] fp32 raw accumulators
  int groups = 1, splits = 1;
  const float* sx = nullptr;         // [groups][M]
  const float* sw = nullptr;         // [d]
  const TpCommDev* comm = nullptr;   // input = sum over ranks of the published partial results (fused all-reduce)
  float* residual_f32 = nullptr;     // [M,d] fp32 residual stream, in/out, may be null
  bf16* residual = nullptr;          // [M,d] bf16 residual, in/out, may be null
  const float* gain = nullptr;       // [d]; null: only the residual update is done
  float eps = 1e-6f;
  bf16* y = nullptr;                 // [M,d] normalised bf16 output, may be null
  uint8_t* q = nullptr;              // split output [sb_qrows(M), d], may be null
  float* qscale = nullptr;           // [M]
};
int k_rownorm(strictb200_ctx*, const RowNormArgs& a, int64_t M, int64_t d);
int k_reduce_scale(strictb200_ctx*, const float* part, int splits, const float* sx, const float* sw, int64_t M, int64_t N, float* out,
                   bf16* out_bf16 = nullptr);
// Grouped RMS norm of the residual stream, one or two gains over one normalisation:
//   x += sum over splits of part (when given); every group of d / groups consecutive columns is divided by its own root mean
//   square; y1 = x_n * g1 and, with g2, y2 = x_n * g2, as bf16 or fp32 rows
struct GroupNormArgs {
  float* x = nullptr;            // [M, ldx] fp32 residual stream, in/out
  int64_t ldx = 0;
  const float* part = nullptr;   // [splits][M, ldp] raw sums of the projections that feed the residual, may be null
  int64_t ldp = 0;
  int splits = 1;
  const float *g1 = nullptr, *g2 = nullptr;  // [d]; g1 null: only the residual update
  float eps = 1e-5f;
  int groups = 1;
  void *y1 = nullptr, *y2 = nullptr;
  int64_t ldy = 0;
  bool f32 = false;              // y in fp32
  // Two sublayers that feed the residual under scales of their own: the first splits0 partial sums belong to the first one;
  // x += mult * (scale0 * (sum of those) + scale1 * (sum of the rest)). Scales are [d], null: 1.
  int splits0 = 8;
  const float *scale0 = nullptr, *scale1 = nullptr;
  float mult = 1.f;
  float out_scale = 1.f;         // factor on y1 and y2
};
int k_group_norm(strictb200_ctx*, const GroupNormArgs& a, int64_t M, int64_t d);
void sb_xielu_coefficients(float p, float q, float* pos, float* neg);
int k_layernorm(strictb200_ctx*, const float* x, const float* g, const float* b, float eps, int64_t M, int64_t d, float* y);
int k_add_f32(strictb200_ctx*, float* x, const float* y, int64_t n);
int k_swiglu(strictb200_ctx*, const bf16* gate_up, const float* gate_up_f32, int64_t M, int64_t I, bf16* y, uint8_t* q, float* qscale);
// gate_up as split-K partials [splits][M][2I] + scales -> two-term split of silu(gate)*up
int k_swiglu_part(strictb200_ctx*, const float* part, int splits, const float* sx, const float* sw, int64_t M, int64_t I, uint8_t* q,
                  float* qscale);
int k_gelu_tanh(strictb200_ctx*, const float* x, int64_t n, float* y);
#ifdef __CUDACC__
// xIELU for results that are rounded to bf16: exp through ex2, and the series of exp(z) - 1 - z where that would cancel
__device__ __forceinline__ float sb_xielu_bf16(float z, float pos, float neg) {
  const float zz = z * z;
  const float series = zz * fmaf(z, fmaf(z, 0.041666667f, 0.16666667f), 0.5f);
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(z * 1.4426950408889634f));
  const float t = z > -0.0625f ? series : e - 1.0f - z;
  return fmaf(z > 0.f ? pos : neg, z > 0.f ? zz : t, 0.5f * z);
}
// tanh-approximated GELU in fp32 with the operation order of the element-wise kernel
__device__ __forceinline__ float sb_gelu_tanh(float v) {
  const float u = __fmul_rn(0.797884583f, __fadd_rn(v, __fmul_rn(0.044715f, __fmul_rn(__fmul_rn(v, v), v))));
  return __fmul_rn(__fmul_rn(0.5f, v), __fadd_rn(1.0f, tanhf(u)));
}
// xIELU: pos * z^2 + z/2 above zero, neg * (exp(z) - 1 - z) + z/2 below; pos = softplus(p), neg = 1/2 + softplus(q)
__device__ __forceinline__ float sb_xielu(float z, float pos, float neg) {
  return z > 0.f ? fmaf(pos * z, z, 0.5f * z) : fmaf(neg, expm1f(z) - z, 0.5f * z);
}
#endif
// rope.cu
struct RopeArgs {
  const bf16* qkv = nullptr;      // [T, nqkv] bf16 (used when part and qkv_f32 are null)
  const float* qkv_f32 = nullptr; // [T, nqkv] fp32 projection result
  const float* part = nullptr;    // [splits][T, nqkv] raw accumulators
  int splits = 1;
  const float* sx = nullptr;      // [T]
  const float* sw = nullptr;      // [nqkv]
  const int32_t* seq = nullptr;   // [T] sequence of each row (null: row t is sequence t)
  const int32_t* pos = nullptr;   // [T] position of each row (null: pos = lens[seq])
  const int32_t* lens = nullptr;  // [B] current lengths (decode)
  const float* cos_t = nullptr;   // [max_pos, D/2]
  const float* sin_t = nullptr;
  const float* qgain = nullptr;
  const float* kgain = nullptr;
  float eps = 1e-6f;
  int Hq = 0, Hkv = 0, D = 128, maxlen = 0, max_pos = 0;
  bf16* q_out = nullptr;          // [T,Hq,D]
  bf16* kcache = nullptr;         // [B,Hkv,maxlen,D]
  bf16* vcache = nullptr;
};
int k_rope_qknorm_kvappend(strictb200_ctx*, const RopeArgs& a, int64_t T);
// Frequencies stretched for longer contexts (YaRN): a pair that turns more than `fast` times within `original` positions
// keeps its frequency, one that turns less than `slow` times has it divided by `factor`, a linear ramp in between; cos and
// sin are multiplied by 0.1 ln(factor) + 1. factor 0: none.
struct RopeScaling {
  double factor = 0, original = 0, fast = 0, slow = 0;
  bool operator==(const RopeScaling& o) const { return factor == o.factor && original == o.original && fast == o.fast && slow == o.slow; }
};
int sb_rope_table(strictb200_ctx*, int max_pos, int D, double theta, float** d_cos, float** d_sin, const RopeScaling& scaling = RopeScaling());
// gemm_fp8.cu
struct GemmArgs {
  int64_t M = 0, N = 0, K = 0;
  const uint8_t* xq = nullptr;  // split activations [sb_qrows(M), K], row stride ldx
  int64_t ldx = 0;
  const float* sx = nullptr;    // [M]
  const uint8_t* wq = nullptr;  // [N,K], row stride ldw
  int64_t ldw = 0;
  const float* sw = nullptr;    // [N]
  void* out = nullptr;          // [M,N] bf16 or fp32 (when splits == 1)
  int out_f32 = 0;
  float* part = nullptr;        // [splits][M,N] raw accumulators (when splits > 1 or raw)
  int splits = 1;
  int raw = 0;                  // 1: always write raw accumulators to part, even for splits == 1
  int kernel = 0;               // 0 auto, 1 skinny, 2 mma.sync tiles, 3 tcgen05
  int i8 = 0;                   // 1: int8 weights and two int8 activation terms (gemm_int8.cu); part then holds int32 sums [splits][2][M,N]
};
int k_gemm_fp8(strictb200_ctx*, const GemmArgs& a);
int sb_gemm_pick_splits(strictb200_ctx*, int64_t M, int64_t N, int64_t K);
int sb_pick_splits_kb(strictb200_ctx*, int64_t M, int64_t N, int64_t nkb);  // the same rule for nkb K blocks of 128 bytes
// gemm_bf16.cu: Y[M,N] = X[M,K] . W[N,K]^T, bf16 operands on the kernels of the E4M3 path (tcgen05 kind::f16), fp32 accumulation.
// Where a finished value goes. Columns from n_switch on (0 = none) belong to a second product of the same launch: its
// operand rows are x_row_off + m, and with act_out set the value leaves through the activation.
struct Bf16Epilogue {
  float* out_f32 = nullptr;   // [M, ldo]
  bf16* out_bf16 = nullptr;   // [M, ldo] (used when out_f32 is null)
  int64_t ldo = 0;
  int accumulate = 0;         // out_f32 += value (the residual stream), times alpha * col_scale[n] when col_scale is given
  const float* col_scale = nullptr;
  float alpha = 1.f;
  int n_switch = 0, x_row_off = 0;
  bf16* act_out = nullptr;    // [M, ld_act], column n - n_switch
  int64_t ld_act = 0;
  float act_pos = 0.f, act_neg = 0.f;  // xIELU coefficients (sb_xielu)
  int glu = 0;                // 1: from n_switch on columns are (gate, up) pairs; act_out column (n - n_switch) / 2 = relu(gate) * up
};
struct GemmBf16Args {
  int64_t M = 0, N = 0, K = 0;  // K in elements; rows may end inside a 64-element block (the copies fill with zeros)
  const bf16* x = nullptr;
  int64_t ldx = 0, x_rows = 0;  // rows of x that exist (0 = M)
  const bf16* w = nullptr;
  int64_t ldw = 0;
  float* part = nullptr;        // [splits][M,N] raw sums instead of an epilogue
  int splits = 1;
  int64_t k_switch = 0;         // > 0 (a multiple of 64, with part): the first splits0 splits share the columns of K before it, the others those after it
  int splits0 = 0;
  int group_n = 0;              // > 0: block-diagonal product, columns [g * group_n, (g + 1) * group_n) read x from its column g * group_k on
  int64_t group_k = 0;          // (group_n must be a multiple of the kernel's channel tile: 128 up to 128 tokens, 256 beyond)
  Bf16Epilogue e;
};
int k_gemm_bf16(strictb200_ctx*, const GemmBf16Args& g);
int sb_gemm_bf16_splits(strictb200_ctx*, int64_t M, int64_t N, int64_t K);
// gemm_f32.cu
int k_gemm_f32(strictb200_ctx*, int64_t M, int64_t N, int64_t K, const float* x, const float* w, const float* bias, float* y,
               int accumulate);
struct GemmF32Args {
  int64_t M = 0, N = 0, K = 0;
  const float* x = nullptr;
  int64_t ldx = 0;
  const float* w = nullptr;
  int64_t ldw = 0;
  const float* bias = nullptr;
  float* y = nullptr;
  int64_t ldy = 0;
  int mode = 0;  // 0 store, 1 add to y, 2 GELU, 3 xIELU, 4 add alpha * col_scale[n] * value to y (col_scale null: 1)
  float act_pos = 0.f, act_neg = 0.f;
  const float* col_scale = nullptr;
  float alpha = 1.f;
};
int k_gemm_f32(strictb200_ctx*, const GemmF32Args& g);
// attention.cu
int k_attn_prefill(strictb200_ctx*, const bf16* q, const bf16* kc, const bf16* vc, const int32_t* lens, const int32_t* past,
                   const int32_t* qstart, int B, int S, int64_t q_rows, int Hq, int Hkv, int D, int maxlen, float scale, bf16* out);
// attention_tc.cu: prompt rows of a latent-attention layer over keys and values rebuilt per head (kv_expand) and the shared rotated key part
struct LatentPrefillArgs {
  const bf16* q = nullptr;      // [q_rows, H, q_head]: the unrotated dims first, the rotated ones from q_rot on
  int64_t q_rows = 0, q_head = 0, q_rot = 0;
  const bf16* k = nullptr;      // row r, head h: k + r * ldk + h * k_head
  const bf16* v = nullptr;      // row r, head h: v + r * ldk + h * v_head
  int64_t k_rows = 0, ldk = 0, k_head = 0, v_head = 0;
  const bf16* k_rot = nullptr;  // row r: k_rot + r * ld_rot
  int64_t ld_rot = 0;
  const int32_t *lens = nullptr, *past = nullptr, *qstart = nullptr;  // [B]
  const int32_t *koff = nullptr, *kpos0 = nullptr;                    // [B] row and position of the first key of a sequence
  int B = 0, S = 0, H = 0, dim = 0, rot = 0, vdim = 0;
  int window = 0;               // 0: every earlier key
  float scale = 1.f;
  bf16* out = nullptr;          // row t, head h: out + t * ldo + h * vdim
  int64_t ldo = 0;
};
// the same kernel over grouped heads straight from the cache, with a sink and a gate per head
struct HeadPrefillArgs {
  const bf16* q = nullptr;      // [q_rows, H, row_dims]
  int64_t q_rows = 0;
  const bf16 *k = nullptr, *v = nullptr;  // [B, Hkv, maxlen, row_dims]
  const int32_t *lens = nullptr, *past = nullptr, *qstart = nullptr;  // [B]
  int B = 0, S = 0, H = 0, Hkv = 0, maxlen = 0, row_dims = 128, vdim = 128;
  float scale = 1.f;
  int sink = 0;
  const float* gate = nullptr;  // [q_rows, H]
  bf16* out = nullptr;          // row t, head h: out + t * ldo + h * vdim
  int64_t ldo = 0;
};
int k_attn_prefill_heads(strictb200_ctx*, const HeadPrefillArgs& a);
bool sb_latent_prefill_fits(int dim, int rot, int vdim);
int k_attn_prefill_latent(strictb200_ctx*, const LatentPrefillArgs& a);
// latent.cu: latent attention (one low-rank vector and one rotated key part per position instead of keys and values per head)
#ifdef __CUDACC__
#define SB_HD __host__ __device__
#else
#define SB_HD
#endif
struct LatentShape {
  int H = 0, dim = 0, rot = 0, vdim = 0, rank = 0;
  int window = 0;                  // keys a position sees, itself included; 0 = every earlier one
  float scale = 1.f;
  SB_HD int dim_p() const { return (dim + 7) & ~7; }
  SB_HD int kv_head() const { return ((dim > vdim ? dim : vdim) + 7) & ~7; }  // head stride of the rebuilt keys and values, one for both
  SB_HD int rot8() const { return (rot + 7) & ~7; }
  SB_HD int q_head() const { return dim_p() + rot8(); }   // head stride of the query buffer; the rotated part begins at dim_p
  SB_HD int rank_p() const { return (rank + 15) & ~15; }  // a cache row: latent, rotated key part, each padded with zeros
  SB_HD int row() const { return rank_p() + ((rot + 15) & ~15); }
  SB_HD int n_q() const { return H * (dim + rot); }
  SB_HD int n_kv() const { return 2 * H * kv_head(); }    // rows of the [uk | uv] matrix, ld = rank_p
};
// The projection's output becomes queries (rotated) and, for a layer with latents of its own, a cache row.
struct LatentSplitArgs {
  LatentShape s;
  const float* in = nullptr;       // [splits][T, ld_in]: queries head by head, then latent and rotated key part
  int64_t ld_in = 0;
  int splits = 1;
  const int32_t *seq = nullptr, *pos = nullptr, *lens = nullptr;  // row t: sequence seq[t] (null: t) at pos[t] (null: lens[seq])
  const float *cos_t = nullptr, *sin_t = nullptr;                 // [max_pos, rot/2]
  int max_pos = 0, maxlen = 0;
  const float* norm_w = nullptr;   // [rank]
  float eps = 1e-5f;
  void* q_out = nullptr;           // [T, H, q_head]
  void* cache = nullptr;           // [B, maxlen, row]; null: the layer reads another layer's latents
  bool f32 = false;
};
int k_latent_split(strictb200_ctx*, const LatentSplitArgs& a, int64_t T);
// The decode step's form: the same, with the queries carried into latent space (q . W_uk per head), and the feed-forward
// half of the projection through its activation.
struct LatentDecodeInArgs {
  LatentSplitArgs a;
  const bf16* wkv = nullptr;       // [n_kv, rank_p]
  bf16* q_abs = nullptr;           // [B, H, row]
  int act_col = 0, n_act = 0;      // columns [act_col, act_col + n_act) of `in` through xIELU to act[b * ld_act + i]
  float act_pos = 0.f, act_neg = 0.f;
  bf16* act = nullptr;
  int64_t ld_act = 0;
};
bool sb_latent_decode_fits(const LatentShape& s);
int k_latent_decode_in(strictb200_ctx*, const LatentDecodeInArgs& a, int64_t B);
// Split-key attention of one new token per sequence over the latents of its window (the key chunks of a sequence are merged
// inside a cluster), then the value projection of every head. len_plan: lengths the chunks are planned for.
int sb_latent_decode_chunk(strictb200_ctx*, const LatentShape& s, int B, int len_plan);
size_t sb_latent_decode_scratch(const LatentShape& s, int B);
int k_latent_attn_decode(strictb200_ctx*, const LatentShape& s, const bf16* q_abs, const bf16* cache, const int32_t* lens, int B, int maxlen, int chunk,
                         int nsplit, bf16* scratch, const bf16* wkv, bf16* out, int64_t ldo);
// Any widths, bf16 or fp32, prompt rows and decode rows: one block per row and head, straight from the cache.
int k_latent_attn_any(strictb200_ctx*, const LatentShape& s, bool f32, const void* q, const void* cache, const void* wkv, const int32_t* seq,
                      const int32_t* pos, const int32_t* lens, int64_t T, int maxlen, void* out, int64_t ldo);
// rows of the cache of several sequences one after the other: dst row koff[j] + i = cache row kpos0[j] + i of sequence j, i < n[j]
int k_latent_gather(strictb200_ctx*, const bf16* cache, int64_t maxlen, int row, const int32_t* koff, const int32_t* kpos0, const int32_t* lens, int nb,
                    int max_n, bf16* dst);
// heads.cu: softmax attention over grouped heads of any width (optional RMS norm of the rotated queries and keys, sink, output
// gate per head), and the projection rows of every mixer that has rotated heads
struct HeadShape {
  int H = 0, G = 0, dim = 0, vdim = 0, rot = 0;  // query heads, key/value heads, query/key and value dims, rotated dims (first ones, i with i + rot/2)
  float scale = 1.f;
  float k_scale = 1.f;  // factor on the rotated keys
  int qk_norm = 0;      // 1: rotated queries and keys divided by their root mean square
  int sink = 0;         // 1: one more key in the softmax denominator, score 0, no value
  int gate = 0;         // 1: a column per head; its sigmoid multiplies the head's output
  SB_HD int row() const {  // dims of a query, key or value row in memory (zeros beyond dim or vdim)
    const int m = dim > vdim ? dim : vdim;
    return m <= 64 ? 64 : m <= 128 ? 128 : (m + 7) & ~7;
  }
  SB_HD int n_in() const { return H * dim + G * (dim + vdim) + (gate ? H : 0); }
};
// The feed-forward's columns of a projection, finished: kind 1 xIELU of columns [col, col + n), kind 2 relu(gate) * up of
// the n column pairs from col on. out[t * ld + i], bf16 or fp32 like the rest of the launch.
struct ActArgs {
  int kind = 0, col = 0, n = 0;
  float pos = 0.f, neg = 0.f;
  void* out = nullptr;
  int64_t ld = 0;
};
// Rows of a projection: column c of row t is the sum over splits of in[(split * T + t) * ld + c].
struct ProjRows {
  const float* in = nullptr;
  int64_t ld = 0;
  int splits = 1;  // at most 8
};
// Columns [q heads | k heads | v heads | gates] become rotated rows.
struct HeadSplitArgs {
  HeadShape s;
  ProjRows p;
  const int32_t *seq = nullptr, *pos = nullptr, *lens = nullptr;  // row t: sequence seq[t] (null: t) at pos[t] (null: lens[seq])
  const float *cos_t = nullptr, *sin_t = nullptr;                 // [max_pos, rot/2]
  int max_pos = 0, maxlen = 0;
  float eps = 1e-5f;
  void* q_out = nullptr;               // [T, H, row]
  void *k_out = nullptr, *v_out = nullptr;  // caches [B, G, maxlen, row], or [T, G, row] with dense
  bool dense = false;
  float* gate_out = nullptr;           // [T, H]
  bool f32 = false;
  ActArgs act;
};
int k_head_split(strictb200_ctx*, const HeadSplitArgs& a, int64_t T);
// one block per row and head, straight from the cache; prompt rows (seq, pos) and decode rows (lens)
int k_head_attn_any(strictb200_ctx*, const HeadShape& s, bool f32, const void* q, const void* kc, const void* vc, const float* gate, const int32_t* seq,
                    const int32_t* pos, const int32_t* lens, int64_t T, int maxlen, void* out, int64_t ldo);
// merge of the key chunks of k_attn_decode_chunks
int k_head_combine(strictb200_ctx*, const HeadShape& s, const float* o_part, const float* ml_part, const float* gate, const int32_t* lens, int B, int maxlen,
                   int chunk, int nsplit, bf16* out, int64_t ldo);
int k_act_rows(strictb200_ctx*, const ProjRows& p, const ActArgs& a, bool f32, int64_t T);
// recurrent.cu: layers with a state per sequence instead of a cache (all states fp32)
// Real-gated linear recurrence behind a causal convolution per channel. Projection columns [y | x], `width` each.
struct GatedShape {
  int width = 0, taps = 1, blocks = 1;
  SB_HD int bs() const { return width / blocks; }
  SB_HD int bs_p() const { return (bs() + 7) & ~7; }       // columns of a block in the convolution's output, which the gate product reads
  SB_HD int64_t ld_u() const { return (int64_t)blocks * bs_p(); }
};
struct GatedArgs {
  GatedShape s;
  ProjRows p;
  const float *y_bias = nullptr, *x_bias = nullptr;          // [width]
  const float *conv = nullptr, *conv_bias = nullptr;         // [width, taps], [width]
  const float *r_bias = nullptr, *i_bias = nullptr;          // [width]
  const float* decay = nullptr;                              // [width] -8 softplus(lam)
  float* hist = nullptr;                                     // [B, taps - 1, width] the convolution's last inputs
  float* state = nullptr;                                    // [B, width]
  const int32_t *seq = nullptr, *qstart = nullptr, *lens = nullptr, *past = nullptr;  // prompt rows; null: row t is the next token of sequence t
  int nb = 0, max_new = 0;
  void* u = nullptr;                                         // [T, ld_u]
  const float* gates = nullptr;                              // [T, 2 width]: block by block, its bs values for r, then those for i
  void* out = nullptr;                                       // [T, ldo]
  int64_t ldo = 0;
  bool f32 = false;
  ActArgs act;
};
int k_gated_conv(strictb200_ctx*, const GatedArgs& a, int64_t T);   // u, and the new hist; with act, the feed-forward's columns too
int k_gated_scan(strictb200_ctx*, const GatedArgs& a, int64_t T);   // the recurrence and out = S * gelu(y)
// Retention: S <- decay S + k v^T, o = S^T q, per head; o over its root mean square, times silu(g). Projection columns [q | k | v | g].
struct RetentionArgs {
  HeadShape s;
  ProjRows p;
  const float* decay = nullptr;  // [H]
  float* state = nullptr;        // [B, H, dim, vdim]
  const void *q = nullptr, *k = nullptr, *v = nullptr;  // [T, H, row] (k_head_split, dense)
  const int32_t *qstart = nullptr, *lens = nullptr, *past = nullptr;  // prompt rows of nb sequences; null: row t is the next token of sequence t
  int nb = 0, max_new = 0;
  float eps = 1e-5f;
  void* out = nullptr;
  int64_t ldo = 0;
  bool f32 = false;
  float* seg_state = nullptr;  // k_retention_prefill: scratch [sb_retention_segments, nb, H, dim, vdim] when that is more than one
  // k_retention_decode: straight from the projection
  const float *cos_t = nullptr, *sin_t = nullptr;
  const int32_t* cache_lens = nullptr;  // [B] positions of the new tokens
  int max_pos = 0;
  ActArgs act;
};
int k_retention_any(strictb200_ctx*, const RetentionArgs& a);            // any widths, token by token
bool sb_retention_prefill_fits(const HeadShape& s);
int k_retention_prefill(strictb200_ctx*, const RetentionArgs& a, int64_t T);  // retention_tc.cu: chunks of 128 tokens
int sb_retention_segments(strictb200_ctx*, const HeadShape& s, int nb, int max_new);
bool sb_retention_decode_fits(const HeadShape& s);
int k_retention_decode(strictb200_ctx*, const RetentionArgs& a, int64_t B);
size_t sb_attn_decode_scratch(int B, int Hq, int D, int nsplit);
int sb_attn_decode_splits(strictb200_ctx*, int B, int Hkv, int maxlen);
int sb_attn_decode_chunk(strictb200_ctx*, int B, int Hkv, int maxlen, int len_plan);  // keys per block for sequences of about len_plan keys (at most 8 chunks cover maxlen)
// rope != null: the queries and the new token's key/value rows are computed inside the attention kernel from the qkv
// projection's partial results (what k_rope_qknorm_kvappend would do in a kernel of its own); q is then unused
int k_attn_decode(strictb200_ctx*, const bf16* q, const bf16* kc, const bf16* vc, const int32_t* lens, int len_add, int B, int Hq,
                  int Hkv, int D, int maxlen, float scale, int nsplit, float* scratch, bf16* out, uint8_t* q_out, float* qscale_out,
                  const RopeArgs* rope = nullptr, int chunk = 0);
int k_attn_decode_chunks(strictb200_ctx*, int HD, const bf16* q, const bf16* kc, const bf16* vc, const int32_t* lens, int B, int Hq, int Hkv, int maxlen,
                         float scale, int nsplit, int chunk, float* o_part, float* ml_part);
int k_attn_f32(strictb200_ctx*, const float* qkv, float* kc, float* vc, const int32_t* seq, const int32_t* pos, const int32_t* lens,
               int64_t T, int H, int D, int maxlen, float scale, float* out);
// sampling.cu
int k_embedding_bf16(strictb200_ctx*, const bf16* table, const int32_t* ids, int64_t T, int64_t d, int64_t vocab, bf16* out);
int k_embedding_bf16_f32(strictb200_ctx*, const bf16* table, const int32_t* ids, int64_t T, int64_t d, int64_t vocab, float* out);
int k_embedding_f32(strictb200_ctx*, const float* wte, const float* wpe, const int32_t* ids, const int32_t* pos, const int32_t* lens,
                    int64_t T, int64_t d, int64_t vocab, int max_pos, float* out);
int k_argmax(strictb200_ctx*, const float* x, int64_t M, int64_t N, int64_t ldx, int32_t* out, float* val_out, void* scratch);
size_t sb_argmax_scratch(int64_t M, int64_t N);  // bytes of chunk winners for the two-stage pick
int k_gather_rows(strictb200_ctx*, const void* src, const int32_t* rows, int64_t n_rows, int64_t row_bytes, void* dst);
int k_add_i32(strictb200_ctx*, int32_t* x, const int32_t* inc, int32_t c, int64_t n);
int k_f32_to_bf16(strictb200_ctx*, const float* x, int64_t n, bf16* y);
int k_bf16_to_f32(strictb200_ctx*, const bf16* x, int64_t n, float* y);
// tp.cpp
const TpCommDev* sb_tp_comm(strictb200_ctx*);  // null unless the peer buffers were opened
bool sb_tp_comm_fits(strictb200_ctx*, int64_t M, int64_t d);  // the peer-memory all-reduce takes an [M,d] result
bool sb_tp_row_exchange_ok(strictb200_ctx*, int64_t M, int64_t d, int two_shot);  // ... with the row-granular exchange (one row width per context)
// out[m,n] = (sum_s part[s][m,n]) * sx[m] * sw[n] written to this rank's peer buffer, then published
int k_tp_publish(strictb200_ctx*, const float* part, int splits, const float* sx, const float* sw, int64_t M, int64_t N);
int sb_tp_allreduce_f32(strictb200_ctx*, float* buf, int64_t count);
int sb_tp_allgather(strictb200_ctx*, const void* send, void* recv, int64_t bytes_per_rank);
void sb_tp_destroy(strictb200_ctx*);
int sb_tp_async_error(strictb200_ctx*);  // 0 = none; else the NCCL result code of the communicator's asynchronous error
void sb_tp_abort(strictb200_ctx*);       // ncclCommAbort: stops the communicator's kernels; the communicator is unusable afterwards

// ------------------------------------------------------------------ device helpers
#ifdef __CUDACC__
__device__ __forceinline__ uint32_t f32_to_bf16_bits(float f);
// Sixteen tokens m0.. of one output channel n per lane (channels of a warp are consecutive, the first one even, all on the
// same side of n_switch). bf16 rows: neighbouring lanes trade tokens so that each stores two channels at a time.
__device__ __forceinline__ void sb_bf16_store16(const Bf16Epilogue& e, int M, int N, int m0, int n, const uint32_t* r) {
  const bool act = e.act_out && n >= e.n_switch;
  if (act && e.glu) {
    // The lanes of a pair hold the gate and the up value of one channel. Each takes eight tokens, then the lanes of two
    // neighbouring channels trade so that each stores both channels of four tokens.
    const int odd = n & 1, second = (n >> 1) & 1, j = (n - e.n_switch) >> 1, nf = (N - e.n_switch) >> 1;
    float p[8];
#pragma unroll
    for (int i = 0; i < 8; i++) {
      const float got = __uint_as_float(__shfl_xor_sync(0xffffffffu, odd ? r[i] : r[8 + i], 1));
      const float gate = odd ? got : __uint_as_float(r[i]), up = odd ? __uint_as_float(r[8 + i]) : got;
      p[i] = fmaxf(gate, 0.f) * up;
    }
    bf16* o = e.act_out + (int64_t)(m0 + odd * 8 + second * 4) * e.ld_act + (j - second);
#pragma unroll
    for (int i = 0; i < 4; i++, o += e.ld_act) {
      const float got = __shfl_xor_sync(0xffffffffu, second ? p[i] : p[4 + i], 2);
      const float lo = second ? got : p[i], hi = second ? p[4 + i] : got;
      if (m0 + odd * 8 + second * 4 + i < M && j - second < nf) {
        if (j - second + 1 < nf) *(uint32_t*)o = f32_to_bf16_bits(lo) | (f32_to_bf16_bits(hi) << 16);
        else *o = __float2bfloat16_rn(lo);
      }
    }
    return;
  }
  if (!act && e.out_f32) {
    if (n >= N) return;
    const float cs = e.col_scale ? e.alpha * e.col_scale[n] : e.alpha;
    float* o = e.out_f32 + (int64_t)m0 * e.ldo + n;
    float old[16];  // all read before the first store, so that the sixteen reads overlap
    if (e.accumulate) {
#pragma unroll
      for (int j = 0; j < 16; j++) old[j] = m0 + j < M ? o[j * e.ldo] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 16; j++, o += e.ldo)
      if (m0 + j < M) *o = e.accumulate ? fmaf(cs, __uint_as_float(r[j]), old[j]) : __uint_as_float(r[j]);
    return;
  }
  const int64_t ld = act ? e.ld_act : e.ldo;
  bf16* o = act ? e.act_out + (n - e.n_switch) : e.out_bf16 + n;
  float v[16];
#pragma unroll
  for (int j = 0; j < 16; j++) v[j] = __uint_as_float(r[j]);
  if (act) {
#pragma unroll
    for (int j = 0; j < 16; j++) v[j] = sb_xielu_bf16(v[j], e.act_pos, e.act_neg);
  }
  if ((ld & 1) == 0 && (N & 1) == 0 && ((uintptr_t)(act ? e.act_out : e.out_bf16) & 3) == 0) {  // the same for every lane
    const bool odd = n & 1;
    o += (int64_t)(m0 + (odd ? 8 : 0)) * ld - (odd ? 1 : 0);
#pragma unroll
    for (int j = 0; j < 8; j++, o += ld) {
      const float got = __shfl_xor_sync(0xffffffffu, odd ? v[j] : v[8 + j], 1);
      const float lo = odd ? got : v[j], hi = odd ? v[8 + j] : got;
      if (m0 + j + (odd ? 8 : 0) < M && n < N) *(uint32_t*)o = f32_to_bf16_bits(lo) | (f32_to_bf16_bits(hi) << 16);
    }
  } else if (n < N) {
    o += (int64_t)m0 * ld;
#pragma unroll
    for (int j = 0; j < 16; j++, o += ld)
      if (m0 + j < M) *o = __float2bfloat16_rn(v[j]);
  }
}
// Programmatic dependent launch. A kernel launched through sb_launch may begin while its
// predecessor in the stream is still running: pdl_trigger() lets the successor start launching,
// pdl_wait() blocks until the predecessor has completed and its writes are visible. Every such
// kernel calls pdl_wait() before it reads or writes anything another kernel touches (so the
// ordering stays transitive along the stream); only reads of constants (weights) may precede it.
// Without the launch attribute both are no-ops.
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
// Diagnostics: per-block time stamps of the decode step's kernels. While a trace is armed
// (strictb200_trace_begin) thread 0 of every block of an instrumented kernel records the global
// timer at block start, after the dependency wait and at block end, with the SM it ran on; the
// host reads the records back (strictb200_trace_end). The pointer lives in a device variable of
// each translation unit (read at run time, so a recorded CUDA graph can be traced as it is); when
// it is null a block pays one cached load.
struct SbTraceDev {
  unsigned long long* rec;  // [capacity][8]: start, after the wait, end, kernel id | tag << 8 | SM << 48, three optional marks inside the kernel, 0
  unsigned int* count;
  unsigned int capacity;
};
static __device__ SbTraceDev sb_trace_dev;
#define SB_TRACE_TU(name) \
  int sb_trace_set_##name(const SbTraceDev& t) { return cudaMemcpyToSymbol(sb_trace_dev, &t, sizeof t) == cudaSuccess ? 0 : 1; }
enum { SB_K_GEMM = 1, SB_K_ROWNORM = 2, SB_K_ROPE = 3, SB_K_ATTN = 4, SB_K_COMBINE = 5, SB_K_SWIGLU = 6, SB_K_ROWNORM_TP = 7, SB_K_RECURRENCE = 8 };
__device__ __forceinline__ unsigned long long sb_globaltimer() {
  unsigned long long t;
  asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
  return t;
}
__device__ __forceinline__ void sb_trace_emit(int kid, uint32_t tag, const unsigned long long* marks) {
  if (!marks[0]) return;
  const unsigned long long t2 = sb_globaltimer();
  unsigned int smid;
  asm volatile("mov.u32 %0, %%smid;" : "=r"(smid));
  const unsigned int i = atomicAdd(sb_trace_dev.count, 1u);
  if (i < sb_trace_dev.capacity) {
    unsigned long long* r = sb_trace_dev.rec + (size_t)i * 8;
    r[0] = marks[0]; r[1] = marks[1]; r[2] = t2;
    r[3] = (unsigned long long)kid | ((unsigned long long)tag << 8) | ((unsigned long long)smid << 48);
    r[4] = marks[2]; r[5] = marks[3]; r[6] = marks[4]; r[7] = 0;
  }
}
// In a kernel: SB_TRACE_BEGIN() first, SB_TRACE_WAITED() by thread 0 right after its pdl_wait(), SB_TRACE_END(id, tag) last;
// SB_TRACE_MARK(0..2) stamps a point in between (as thread 0 reaches it).
#define SB_TRACE_BEGIN()                                 \
  __shared__ unsigned long long sb_tr_[5];               \
  if (threadIdx.x == 0) {                                \
    sb_tr_[0] = sb_trace_dev.rec ? sb_globaltimer() : 0; \
    sb_tr_[1] = sb_tr_[2] = sb_tr_[3] = sb_tr_[4] = 0;   \
  }
#define SB_TRACE_WAITED() \
  if (threadIdx.x == 0 && sb_tr_[0]) sb_tr_[1] = sb_globaltimer();
#define SB_TRACE_MARK(i) \
  if (threadIdx.x == 0 && sb_tr_[0]) sb_tr_[2 + (i)] = sb_globaltimer();
#define SB_TRACE_END(kid, tag) \
  if (threadIdx.x == 0) sb_trace_emit(kid, (uint32_t)(tag), sb_tr_);
// L2 eviction policy for data that is read exactly once per step (weights, the KV cache): such
// lines are the first to be replaced, so the 126 MB L2 keeps the small tensors the kernels hand
// to each other, the scale/gain vectors and the kernels' own instructions resident.
__device__ __forceinline__ uint64_t l2_evict_first_policy() {
  uint64_t p;
  asm volatile("createpolicy.fractional.L2::evict_first.b64 %0, 1.0;" : "=l"(p));
  return p;
}
template <typename... KArgs, typename... Args>
inline cudaError_t sb_launch(strictb200_ctx* ctx, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = ctx->stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = ctx->opt.pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}
// Same, as thread-block clusters of `cluster` blocks (the grid must be a multiple of it).
template <typename... KArgs, typename... Args>
inline cudaError_t sb_launch_cluster(strictb200_ctx* ctx, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, dim3 cluster, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = ctx->stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cluster.x;
  attr[0].val.clusterDim.y = cluster.y;
  attr[0].val.clusterDim.z = cluster.z;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = ctx->opt.pdl ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}
// One-value-per-block exchange inside a thread-block cluster of at most 8 blocks: every block
// pushes its value into the others' shared memory with st.async, which also completes bytes on
// the receiver's mbarrier, so a block waits only for the values it needs and nobody reads a
// block that may already have left (measured about 0.4 us, against 0.9 us for a cluster
// barrier plus remote reads plus a second barrier before exit).
struct ClusterExchange {
  float slot[2][8];
  unsigned long long bar[2];  // one barrier per exchange: a fast block's second value must not count for a slow block's first wait
};
// All threads of all blocks call this once at kernel start (before any long wait).
__device__ __forceinline__ void cluster_exchange_init(ClusterExchange* x) {
  if (threadIdx.x == 0) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"((uint32_t)__cvta_generic_to_shared(&x->bar[0])));
    asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"((uint32_t)__cvta_generic_to_shared(&x->bar[1])));
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
}
// All threads of all blocks call this with a block-uniform value, at most once per `which` (0,
// then 1); returns false if the other blocks' values did not arrive within the spin limit
// (slot[which][] is then incomplete). Afterwards slot[which][r] holds block r's value in every block.
__device__ __forceinline__ bool cluster_exchange(ClusterExchange* x, float v, uint32_t nblocks, uint32_t rank, int which = 0) {
  const uint32_t bar = (uint32_t)__cvta_generic_to_shared(&x->bar[which]);
  if (threadIdx.x == 0) {
    x->slot[which][rank] = v;
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(4u * (nblocks - 1)) : "memory");
  }
  if (which == 0) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");  // every block's barriers are initialised
  if (threadIdx.x < nblocks && threadIdx.x != rank) {
    uint32_t rslot, rbar;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(rslot) : "r"((uint32_t)__cvta_generic_to_shared(&x->slot[which][rank])), "r"(threadIdx.x));
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(rbar) : "r"(bar), "r"(threadIdx.x));
    asm volatile("st.async.weak.shared::cluster.mbarrier::complete_tx::bytes.b32 [%0], %1, [%2];" ::"r"(rslot), "r"(__float_as_uint(v)), "r"(rbar) : "memory");
  }
  uint32_t done = 0;
  for (uint32_t spins = 0; !done && spins < (1u << 20); spins++)
    asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}" : "=r"(done) : "r"(bar), "r"(0u) : "memory");
  return done != 0;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Block-wide reductions over blockDim.x threads (multiple of 32, <= 1024). `red` holds 32 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = l < nw ? red[l] : 0.f;
  return warp_sum(t);
}
__device__ __forceinline__ float block_max(float v, float* red) {
  v = warp_max(v);
  int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = l < nw ? red[l] : -INFINITY;
  return warp_max(t);
}
__device__ __forceinline__ float bf16_bits_to_f32(uint32_t h) { return __uint_as_float(h << 16); }
__device__ __forceinline__ uint32_t f32_to_bf16_bits(float f) { return (uint32_t)__bfloat16_as_ushort(__float2bfloat16_rn(f)); }
__device__ __forceinline__ float round_bf16(float f) { return __bfloat162float(__float2bfloat16_rn(f)); }
// E4M3 encode, round-to-nearest-even, saturating to +-448 (cvt.rn.satfinite.e4m3x2.f32).
__device__ __forceinline__ uint32_t f32x2_to_e4m3x2(float lo, float hi) {
  uint16_t r;
  asm("cvt.rn.satfinite.e4m3x2.f32 %0, %2, %1;" : "=h"(r) : "f"(lo), "f"(hi));
  return (uint32_t)r;
}
__device__ __forceinline__ uint32_t f32x4_to_e4m3x4(float a, float b, float c, float d) {
  return f32x2_to_e4m3x2(a, b) | (f32x2_to_e4m3x2(c, d) << 16);
}
// E4M3 pair -> two floats (exact; through f16x2).
__device__ __forceinline__ float2 e4m3x2_to_f32x2(uint32_t pair) {
  uint32_t h2;
  asm("cvt.rn.f16x2.e4m3x2 %0, %1;" : "=r"(h2) : "h"((uint16_t)pair));
  return __half22float2(*reinterpret_cast<__half2*>(&h2));
}
// Exponent e of the power-of-two row scale: the smallest 2^e with amax/2^e <= 448.
__device__ __forceinline__ int sb_scale_exponent(float amax) {
  if (!(amax >= 7.888609e-31f)) return 0;
  uint32_t b = __float_as_uint(amax);
  int E = (int)((b >> 23) & 255) - 126;
  return (b & 0x7FFFFFu) <= 0x600000u ? E - 9 : E - 8;
}
__device__ __forceinline__ float sb_pow2(int e) { return __uint_as_float((uint32_t)(e + 127) << 23); }
// Two-term split of 8 values already divided by the row scale: hi = e4m3(v), lo = e4m3(16*(v-hi)).
__device__ __forceinline__ void sb_split8(const float* v, uint2* hi, uint2* lo) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; i++) {
    h[i] = f32x2_to_e4m3x2(v[2 * i], v[2 * i + 1]);
    float2 hv = e4m3x2_to_f32x2(h[i]);
    l[i] = f32x2_to_e4m3x2(__fmul_rn(16.0f, __fsub_rn(v[2 * i], hv.x)), __fmul_rn(16.0f, __fsub_rn(v[2 * i + 1], hv.y)));
  }
  *hi = make_uint2(h[0] | (h[1] << 16), h[2] | (h[3] << 16));
  *lo = make_uint2(l[0] | (l[1] << 16), l[2] | (l[3] << 16));
}
// Store the split of 8 consecutive columns of token row m into the split buffer q [*, K].
__device__ __forceinline__ void sb_store_split8(uint8_t* q, int64_t K, int64_t m, int64_t k, const float* v, float inv) {
  float t[8];
#pragma unroll
  for (int i = 0; i < 8; i++) t[i] = __fmul_rn(v[i], inv);
  uint2 hi, lo;
  sb_split8(t, &hi, &lo);
  int64_t row = 16 * (m >> 3) + (m & 7);
  *(uint2*)(q + row * K + k) = hi;
  *(uint2*)(q + (row + 8) * K + k) = lo;
}
// The same for 4 consecutive columns.
__device__ __forceinline__ void sb_store_split4(uint8_t* q, int64_t K, int64_t m, int64_t k, const float* v, float inv) {
  uint32_t h[2], l[2];
#pragma unroll
  for (int i = 0; i < 2; i++) {
    float a = __fmul_rn(v[2 * i], inv), b = __fmul_rn(v[2 * i + 1], inv);
    h[i] = f32x2_to_e4m3x2(a, b);
    float2 hv = e4m3x2_to_f32x2(h[i]);
    l[i] = f32x2_to_e4m3x2(__fmul_rn(16.0f, __fsub_rn(a, hv.x)), __fmul_rn(16.0f, __fsub_rn(b, hv.y)));
  }
  int64_t row = 16 * (m >> 3) + (m & 7);
  *(uint32_t*)(q + row * K + k) = h[0] | (h[1] << 16);
  *(uint32_t*)(q + (row + 8) * K + k) = l[0] | (l[1] << 16);
}
#endif
