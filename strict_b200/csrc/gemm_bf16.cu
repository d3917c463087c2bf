// bf16 linear layers on the tcgen05 kernels of the E4M3 path: up to 128 tokens (and every launch that leaves K splits to its
// consumer) the split-K tile kernel, beyond that the 256 x 256 tile on SM pairs. The two kernels stage 128-byte rows of K
// whatever the element type; with kind::f16 such a row is 64 bf16 elements and an operand row is one token.
#include "common.cuh"

int k_gemm_bf16_tmem_split(strictb200_ctx* ctx, const GemmBf16Args& g);  // gemm_tmem_split.cu
int k_gemm_bf16_tmem_pair(strictb200_ctx* ctx, const GemmBf16Args& g);   // gemm_tmem_pair.cu

int sb_gemm_bf16_splits(strictb200_ctx* ctx, int64_t M, int64_t N, int64_t K) {
  if (M > 128) return 1;
  return sb_pick_splits_kb(ctx, M, N, (K + 63) / 64);
}

int k_gemm_bf16(strictb200_ctx* ctx, const GemmBf16Args& g) {
  if (g.M <= 0 || g.N <= 0 || g.K <= 0 || g.M > INT32_MAX || g.N > INT32_MAX || g.K > INT32_MAX / 2)
    return sb_fail(STRICTB200_ERR_INVALID_ARG, "gemm_bf16: bad shape");
  if (((uintptr_t)g.x | (uintptr_t)g.w | (uintptr_t)(2 * g.ldx) | (uintptr_t)(2 * g.ldw)) & 15)
    return sb_fail(STRICTB200_ERR_INVALID_ARG, "gemm_bf16: operands and row strides must be 16-byte aligned");
  if (g.e.n_switch % 256) return sb_fail(STRICTB200_ERR_INVALID_ARG, "gemm_bf16: the second product must begin at a multiple of 256 columns");
  if (g.M <= 128 || (g.part && g.M <= 256)) return k_gemm_bf16_tmem_split(ctx, g);
  if (!g.part) return k_gemm_bf16_tmem_pair(ctx, g);
  if (g.splits != 1) return sb_fail(STRICTB200_ERR_INVALID_ARG, "gemm_bf16: K splits are for at most 256 tokens");
  GemmBf16Args f = g;  // one "split" of many tokens is the finished product
  f.part = nullptr;
  f.e.out_f32 = g.part; f.e.ldo = g.N; f.e.accumulate = 0; f.e.act_out = nullptr;
  return k_gemm_bf16_tmem_pair(ctx, f);
}

extern "C" int strictb200_gemm_bf16(strictb200_ctx* ctx, int64_t M, int64_t N, int64_t K, const uint16_t* d_x, const uint16_t* d_w, void* d_y,
                                    int out_dtype) {
  SB_ENTER(ctx);
  SB_REQUIRE(M >= 0 && N > 0 && K > 0 && K % 8 == 0, "bad shape (K must be a multiple of 8)");
  SB_REQUIRE(out_dtype == 0 || out_dtype == 1, "out_dtype: 0 bf16, 1 fp32");
  if (!M) return STRICTB200_OK;
  SB_REQUIRE(d_x && d_w && d_y, "null pointer");
  GemmBf16Args g;
  g.M = M; g.N = N; g.K = K; g.x = (const bf16*)d_x; g.ldx = K; g.w = (const bf16*)d_w; g.ldw = K;
  if (out_dtype) g.e.out_f32 = (float*)d_y;
  else g.e.out_bf16 = (bf16*)d_y;
  g.e.ldo = N;
  return k_gemm_bf16(ctx, g);
}
