// Models described layer by layer: every layer names its mixer and feed-forward with their sizes; all layers share the width and
// the parallel form
//     x <- x + m (ls1 * mixer(norm1(x)) + ls2 * ff(norm2(x))),   both norms of the same x,
// where the two norms may be one, and the scales per channel (ls1, ls2) and m may be absent. Mixers: latent attention
// (latent.cu), softmax attention over grouped heads (heads.cu), a gated linear recurrence and retention (recurrent.cu).
// Weights and activations are bf16 (fp32 residual, norms, scores, softmax, recurrences), or everything is fp32.
//
// The parallel form leaves two matrix products per layer on the residual path:
//   w_in  [the mixer's projections | zero rows to a multiple of 256 | the feed-forward's]   one launch; with two norms its first
//         part multiplies norm1(x), the rest norm2(x) (two operand row ranges of one buffer, which one row kernel writes). The
//         rows of a gated feed-forward alternate gate and up, so that an epilogue holds both values of a channel.
//   w_out [o | down] side by side along K, over the row [mixer output | activation]: one product adds both; where each has a
//         scale of its own the K splits of a decode step do not cross the seam, and a prompt multiplies the parts in turn.
// Latent attention adds [uk | uv] per head (rows of a head padded to one multiple of 8), K = the latent; the gated recurrence its
// block-diagonal gate matrices, [r | i] of a block one after the other.
//
// Cache: one array, layer after layer: latent attention rows [B, maxlen, latent | rotated key part] for the layers with latents
// of their own, softmax attention keys then values [B, kv heads, maxlen, row]. States are a second array, fp32: the gated
// recurrence's [B, width] and its convolution's last inputs [B, taps - 1, width], retention's [B, heads, dim, vdim].
#include "model.cuh"

namespace {

enum { T_DKV = 2, T_UK = 3, T_UV = 4, T_G = 5, T_CONV = 11, T_RA = 12, T_RI = 13 };  // besides T_Q, T_K, T_V, T_O, T_GATE, T_UP, T_DOWN

struct StackLayer {
  int kind = STRICTB200_MIXER_LATENT, mlp = STRICTB200_MLP_NONE;
  LatentShape s;          // latent attention
  HeadShape hs;           // softmax attention and retention
  GatedShape gs;          // gated recurrence
  int src = 0;            // layer whose latents this layer reads
  bool own = true;        // ... which is this one
  int ff = 0;             // 0: no feed-forward
  double base = 0;
  RopeScaling scaling;
  int rot = 0;            // rotated dims
  int64_t n0 = 0;         // rows of w_in that multiply norm1(x)
  int64_t n_switch = 0;   // first row of the feed-forward's part (0: none)
  int64_t n_in = 0;       // all rows of w_in
  int64_t ko_p = 0, ldo = 0;  // columns of w_out before the feed-forward's part, and all of them
  void *w_in = nullptr, *w_kv = nullptr, *w_out = nullptr;
  float *norm1 = nullptr, *norm2 = nullptr, *dkv_norm = nullptr;
  float act[2] = {0.f, 0.f}, act_pos = 0.f, act_neg = 0.f;
  float *cos_t = nullptr, *sin_t = nullptr;
  float *ls1 = nullptr, *ls2 = nullptr;  // scales per channel of the mixer's and the feed-forward's result
  void* w_gate = nullptr;                // gated recurrence: [blocks * 2 * bs, bs_p]
  float *y_bias = nullptr, *x_bias = nullptr, *conv = nullptr, *conv_bias = nullptr, *r_bias = nullptr, *i_bias = nullptr, *lam = nullptr;
  float* decay = nullptr;                // gated recurrence: -8 softplus(lam) per channel; retention: per head
  size_t state = 0;                      // floats of state per sequence
  bool glu() const { return mlp == STRICTB200_MLP_RELU_GLU; }
  int64_t n_out() const { return kind == STRICTB200_MIXER_LATENT ? (int64_t)s.H * s.vdim : kind == STRICTB200_MIXER_GATED ? gs.width : (int64_t)hs.H * hs.vdim; }
  bool fast_prefill = false, fast_decode = false;
};

int64_t pad8(int64_t n) { return (n + 7) / 8 * 8; }
int64_t pad64(int64_t n) { return (n + 63) / 64 * 64; }

}  // namespace

struct SbStack {
  bool f32 = false;
  int groups = 1;
  bool shared_norm = false, layer_scale = false;
  float mult = 1.f, logit_scale = 1.f;
  int64_t dp = 0;  // row stride of everything d_model wide
  void *embed = nullptr, *head = nullptr;
  float* normf = nullptr;
  std::vector<StackLayer> L;
  bool pads = false;      // some row of the [attention | activation] buffer or of the norm outputs has padding columns
  uint64_t version = 1;   // advanced when a constant that launches carry by value changes
  size_t esz() const { return f32 ? 4 : 2; }
};

namespace {

int zalloc(strictb200_model* m, void** p, size_t bytes) {
  char* c;
  SB_TRY(dalloc(m, &c, bytes));
  SB_CUDA(cudaMemsetAsync(c, 0, bytes, m->ctx->stream));
  *p = c;
  return STRICTB200_OK;
}

// ------------------------------------------------------------------ named tensors
struct Slot {
  void* dev = nullptr;
  bool dev_f32 = false;
  int64_t rows = 0, cols = 0, ld = 0;
  int64_t per_group = 0, group_stride = 0;  // row r lives at row (r / per_group) * group_stride + r % per_group
  float* host = nullptr;                    // values kept on the host
  StackLayer* lam = nullptr;                // the layer whose decay follows from this tensor
};

template <typename S, typename D>
__device__ __forceinline__ D conv(S v);
template <> __device__ __forceinline__ float conv<float, float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 conv<float, bf16>(float v) { return __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ float conv<bf16, float>(bf16 v) { return __bfloat162float(v); }
template <> __device__ __forceinline__ bf16 conv<bf16, bf16>(bf16 v) { return v; }

// dense [rows, cols] <-> the tensor's place; to_dense: the other way
template <typename S, typename D>
__global__ void place_kernel(S* __restrict__ dense, D* __restrict__ dev, int64_t rows, int64_t cols, int64_t ld, int64_t per_group, int64_t group_stride,
                             int to_dense) {
  const int64_t n = rows * cols, step = (int64_t)gridDim.x * blockDim.x;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += step) {
    const int64_t r = i / cols, c = i - r * cols;
    D* d = dev + ((r / per_group) * group_stride + r % per_group) * ld + c;
    if (to_dense) dense[i] = conv<D, S>(*d);
    else *d = conv<S, D>(dense[i]);
  }
}
int place(strictb200_ctx* ctx, const Slot& s, void* dense, bool dense_f32, bool to_dense) {
  const int64_t n = s.rows * s.cols;
  const unsigned grid = (unsigned)std::min<int64_t>((n + 255) / 256, (int64_t)ctx->sm_count * 16);
#define PLACE(S, D) place_kernel<S, D><<<grid, 256, 0, ctx->stream>>>((S*)dense, (D*)s.dev, s.rows, s.cols, s.ld, s.per_group, s.group_stride, to_dense)
  if (dense_f32) {
    if (s.dev_f32) PLACE(float, float); else PLACE(float, bf16);
  } else {
    if (s.dev_f32) PLACE(bf16, float); else PLACE(bf16, bf16);
  }
#undef PLACE
  SB_LAUNCHED(ctx);
  return STRICTB200_OK;
}

// Names as a checkpoint of such a model has them: embed, head, final.norm, l<i>.norm1/.norm2/.ls1/.ls2, l<i>.mlp.{gate,up,down,act},
// and l<i>.mix. {q,dkv,dkv.norm,uk,uv,o} (latent attention), {q,k,v,g,o} (softmax attention, retention),
// {y,y.b,x,x.b,conv,conv.b,ra,ra.b,ri,ri.b,lam,o} (gated recurrence).
bool find_slot(strictb200_model* m, const std::string& name, Slot* o) {
  SbStack& st = *m->stack;
  const int64_t d = m->c.d_model;
  auto set = [&](void* dev, bool f32, int64_t rows, int64_t cols, int64_t ld) {
    o->dev = dev; o->dev_f32 = f32; o->rows = rows; o->cols = cols; o->ld = ld;
    o->per_group = rows; o->group_stride = rows;
    return dev != nullptr;
  };
  auto at = [&](void* base, int64_t elements) -> void* { return base ? (char*)base + elements * (int64_t)st.esz() : nullptr; };
  if (name == "embed") return set(st.embed, st.f32, m->c.vocab, d, st.dp);
  if (name == "head") return set(st.head, st.f32, m->c.vocab, d, st.dp);
  if (name == "final.norm") return set(st.normf, true, 1, d, d);
  if (name.size() < 4 || name[0] != 'l') return false;
  const size_t dot = name.find('.');
  if (dot == std::string::npos || dot < 2) return false;
  for (size_t i = 1; i < dot; i++)
    if (name[i] < '0' || name[i] > '9') return false;
  if (dot > 8) return false;
  const int l = atoi(name.substr(1, dot - 1).c_str());
  if (l >= (int)st.L.size()) return false;
  StackLayer& w = st.L[l];
  const LatentShape& s = w.s;
  const std::string k = name.substr(dot + 1);
  if (k == "norm1") return set(w.norm1, true, 1, d, d);
  if (k == "norm2") return w.norm2 && set(w.norm2, true, 1, d, d);
  if (k == "ls1") return set(w.ls1, true, 1, d, d);
  if (k == "ls2") return w.ff && set(w.ls2, true, 1, d, d);
  if (k == "mix.o") return set(w.w_out, st.f32, d, w.n_out(), w.ldo);
  if (k.compare(0, 4, "mix.") == 0 && w.kind != STRICTB200_MIXER_LATENT) {
    auto rows = [&](int64_t first, int64_t n) { return set(at(w.w_in, first * st.dp), st.f32, n, d, st.dp); };
    if (w.kind == STRICTB200_MIXER_GATED) {
      const GatedShape& g = w.gs;
      const int64_t bs = g.bs();
      if (k == "mix.y") return rows(0, g.width);
      if (k == "mix.x") return rows(g.width, g.width);
      if (k == "mix.y.b") return set(w.y_bias, true, 1, g.width, g.width);
      if (k == "mix.x.b") return set(w.x_bias, true, 1, g.width, g.width);
      if (k == "mix.conv") return set(w.conv, true, g.width, g.taps, g.taps);
      if (k == "mix.conv.b") return set(w.conv_bias, true, 1, g.width, g.width);
      if (k == "mix.ra.b") return set(w.r_bias, true, 1, g.width, g.width);
      if (k == "mix.ri.b") return set(w.i_bias, true, 1, g.width, g.width);
      if (k == "mix.lam") { o->lam = &w; return set(w.lam, true, 1, g.width, g.width); }
      if (k == "mix.ra" || k == "mix.ri") {
        const bool ok = set(at(w.w_gate, k == "mix.ri" ? bs * g.bs_p() : 0), st.f32, g.width, bs, g.bs_p());
        o->per_group = bs; o->group_stride = 2 * bs;
        return ok;
      }
      return false;
    }
    const HeadShape& q = w.hs;
    const int64_t nq = (int64_t)q.H * q.dim, nk = (int64_t)q.G * q.dim, nv = (int64_t)q.G * q.vdim;
    if (k == "mix.q") return rows(0, nq);
    if (k == "mix.k") return rows(nq, nk);
    if (k == "mix.v") return rows(nq + nk, nv);
    if (k == "mix.g") return w.n0 > nq + nk + nv && rows(nq + nk + nv, w.n0 - nq - nk - nv);
    return false;
  }
  if (k == "mix.q") return set(w.w_in, st.f32, s.n_q(), d, st.dp);
  if (k == "mix.dkv") return w.own && set(at(w.w_in, s.n_q() * st.dp), st.f32, s.rank + s.rot, d, st.dp);
  if (k == "mix.dkv.norm") return w.own && set(w.dkv_norm, true, 1, s.rank, s.rank);
  if (k == "mix.uk" || k == "mix.uv") {
    const bool v = k == "mix.uv";
    const int64_t n = v ? s.vdim : s.dim;
    const bool ok = set(at(w.w_kv, v ? (int64_t)s.H * s.kv_head() * s.rank_p() : 0), st.f32, s.H * n, s.rank, s.rank_p());
    o->per_group = n; o->group_stride = s.kv_head();
    return ok;
  }
  if (!w.ff) return false;
  if (k == "mlp.up" || (k == "mlp.gate" && w.glu())) {
    const bool ok = set(at(w.w_in, (w.n_switch + (w.glu() && k == "mlp.up" ? 1 : 0)) * st.dp), st.f32, w.ff, d, st.dp);
    if (w.glu()) { o->per_group = 1; o->group_stride = 2; }
    return ok;
  }
  if (k == "mlp.down") return set(at(w.w_out, w.ko_p), st.f32, d, w.ff, w.ldo);
  if (k == "mlp.act" && w.mlp == STRICTB200_MLP_XIELU) {
    o->host = w.act; o->rows = 1; o->cols = 2;
    return true;
  }
  return false;
}

// decay = -8 softplus(lam)
__global__ void gated_decay_kernel(const float* __restrict__ lam, int n, float* __restrict__ decay) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const double z = lam[i];
  decay[i] = (float)(-8.0 * (log1p(exp(-fabs(z))) + (z > 0 ? z : 0.0)));
}
int set_decay(strictb200_ctx* ctx, const StackLayer& w) {
  gated_decay_kernel<<<(w.gs.width + 255) / 256, 256, 0, ctx->stream>>>(w.lam, w.gs.width, w.decay);
  SB_LAUNCHED(ctx);
  return STRICTB200_OK;
}

void set_act(StackLayer& w) { sb_xielu_coefficients(w.act[0], w.act[1], &w.act_pos, &w.act_neg); }

// ------------------------------------------------------------------ pieces both schedules use
// y = x . w^T of one matrix that is no part of a combined launch (the LM head)
int head_rows(strictb200_model* m, int64_t M, void* h, float* logits) {
  SbStack& st = *m->stack;
  if (st.f32) {
    GemmF32Args g;
    g.M = M; g.N = m->c.vocab; g.K = st.dp; g.x = (const float*)h; g.ldx = st.dp; g.w = (const float*)st.head; g.ldw = st.dp; g.y = logits; g.ldy = m->c.vocab;
    return k_gemm_f32(m->ctx, g);
  }
  GemmBf16Args g;
  g.M = M; g.N = m->c.vocab; g.K = m->c.d_model; g.x = (const bf16*)h; g.ldx = st.dp; g.w = (const bf16*)st.head; g.ldw = st.dp;
  g.e.out_f32 = logits; g.e.ldo = m->c.vocab;
  return k_gemm_bf16(m->ctx, g);
}

GemmBf16Args gemm_in_args(const SbStack& st, const StackLayer& w, int64_t d, int64_t M, void* h) {
  GemmBf16Args g;
  g.M = M; g.N = w.n_in; g.K = d; g.x = (const bf16*)h; g.ldx = st.dp; g.w = (const bf16*)w.w_in; g.ldw = st.dp;
  g.e.n_switch = (int)w.n_switch;
  if (!st.shared_norm) { g.x_rows = 2 * M; g.e.x_row_off = (int)M; }
  return g;
}

// row stride of a finished projection: the mixer's columns, and in fp32 those of a gated feed-forward too
int64_t ld_in_of(const SbStack& st, const StackLayer& w) { return !w.ff || (st.f32 && w.glu()) ? w.n_in : w.n_switch; }

// the feed-forward's columns of a projection of all columns
ActArgs act_args(const StackLayer& w, void* oa, size_t esz) {
  ActArgs a;
  if (!w.ff) return a;
  a.kind = w.glu() ? 2 : 1; a.col = (int)w.n_switch; a.n = w.ff; a.pos = w.act_pos; a.neg = w.act_neg;
  a.out = (char*)oa + w.ko_p * esz; a.ld = w.ldo;
  return a;
}

// The projection of M rows, finished: the mixer's columns in fp32 to `in` (row stride ld_in), the activation to its place in `oa`.
int project_in(strictb200_model* m, const StackLayer& w, int64_t M, void* h, float* in, int64_t ld_in, void* oa) {
  SbStack& st = *m->stack;
  if (st.f32) {
    GemmF32Args g;
    g.M = M; g.N = w.n0; g.K = st.dp; g.x = (const float*)h; g.ldx = st.dp; g.w = (const float*)w.w_in; g.ldw = st.dp; g.y = in; g.ldy = ld_in;
    SB_TRY(k_gemm_f32(m->ctx, g));
    if (!w.ff) return STRICTB200_OK;
    g.w = (const float*)w.w_in + w.n_switch * st.dp;
    if (!st.shared_norm) g.x = (const float*)h + M * st.dp;
    if (w.glu()) {
      g.N = 2 * w.ff; g.y = in + w.n_switch;
      SB_TRY(k_gemm_f32(m->ctx, g));
      return k_act_rows(m->ctx, ProjRows{in, ld_in, 1}, act_args(w, oa, 4), true, M);
    }
    g.N = w.ff; g.y = (float*)oa + w.ko_p; g.ldy = w.ldo; g.mode = 3; g.act_pos = w.act_pos; g.act_neg = w.act_neg;
    return k_gemm_f32(m->ctx, g);
  }
  GemmBf16Args g = gemm_in_args(st, w, m->c.d_model, M, h);
  g.e.out_f32 = in; g.e.ldo = ld_in;
  if (w.ff) { g.e.act_out = (bf16*)oa + w.ko_p; g.e.ld_act = w.ldo; g.e.act_pos = w.act_pos; g.e.act_neg = w.act_neg; g.e.glu = w.glu(); }
  return k_gemm_bf16(m->ctx, g);
}

// x += m (ls1 * (mixer output . o^T) + ls2 * (activation . down^T)); without scales one product over both
int project_out(strictb200_model* m, const StackLayer& w, int64_t M, void* oa, float* x) {
  SbStack& st = *m->stack;
  const bool seam = st.layer_scale && w.ff;
  for (int part = 0; part < (seam ? 2 : 1); part++) {
    const int64_t k0 = part ? w.ko_p : 0, k1 = seam && !part ? w.ko_p : w.ldo;
    const float* scale = part ? w.ls2 : w.ls1;
    if (st.f32) {
      GemmF32Args g;
      g.M = M; g.N = m->c.d_model; g.K = k1 - k0; g.x = (const float*)oa + k0; g.ldx = w.ldo; g.w = (const float*)w.w_out + k0; g.ldw = w.ldo; g.y = x; g.ldy = st.dp;
      g.mode = 4; g.col_scale = scale; g.alpha = st.mult;
      SB_TRY(k_gemm_f32(m->ctx, g));
      continue;
    }
    GemmBf16Args g;
    g.M = M; g.N = m->c.d_model; g.K = k1 - k0; g.x = (const bf16*)oa + k0; g.ldx = w.ldo; g.w = (const bf16*)w.w_out + k0; g.ldw = w.ldo;
    g.e.out_f32 = x; g.e.ldo = st.dp; g.e.accumulate = 1; g.e.col_scale = scale; g.e.alpha = st.mult;
    SB_TRY(k_gemm_bf16(m->ctx, g));
  }
  return STRICTB200_OK;
}

// K splits of the decode step's output product: those of the mixer's columns, and all of them
void out_splits(strictb200_ctx* ctx, const SbStack& st, const StackLayer& w, int64_t B, int64_t d, int* first, int* all) {
  *all = sb_gemm_bf16_splits(ctx, B, d, w.ldo);
  *first = *all;
  if (!st.layer_scale || !w.ff) return;
  const int n0 = (int)(w.ko_p / 64), n1 = (int)((w.ldo - w.ko_p + 63) / 64);
  const int want = *all < 2 ? 2 : *all;
  *first = std::min(std::max((int)((double)want * n0 / (n0 + n1) + 0.5), 1), std::min(want - 1, n0));
  *all = *first + std::min(want - *first, n1);
}

// Sums of a layer's output product that the next norm adds to the residual
struct Pending {
  const StackLayer* from = nullptr;
  const float* part = nullptr;
  int splits = 1, splits0 = 1;
};
int out_parts(strictb200_model* m, const StackLayer& w, int64_t B, const void* oa, float* part, Pending* p) {
  const SbStack& st = *m->stack;
  GemmBf16Args o;
  o.M = B; o.N = m->c.d_model; o.K = w.ldo; o.x = (const bf16*)oa; o.ldx = w.ldo; o.w = (const bf16*)w.w_out; o.ldw = w.ldo; o.part = part;
  out_splits(m->ctx, st, w, B, o.N, &o.splits0, &o.splits);
  if (o.splits0 < o.splits) o.k_switch = w.ko_p;
  p->from = &w; p->part = part; p->splits = o.splits; p->splits0 = o.splits0;
  return k_gemm_bf16(m->ctx, o);
}
int norm_rows(strictb200_model* m, const StackLayer* w, int64_t M, float* x, const Pending& p, void* h) {
  SbStack& st = *m->stack;
  GroupNormArgs a;
  a.x = x; a.ldx = st.dp; a.part = p.part; a.ldp = m->c.d_model; a.splits = p.splits;
  a.splits0 = p.splits0; a.mult = st.mult;
  if (p.from) { a.scale0 = p.from->ls1; a.scale1 = p.from->ls2; }
  if (!w) a.out_scale = st.logit_scale;
  a.g1 = w ? w->norm1 : st.normf; a.g2 = w ? w->norm2 : nullptr;
  a.eps = m->c.eps; a.groups = st.groups; a.y1 = h; a.y2 = (char*)h + M * st.dp * st.esz(); a.ldy = st.dp; a.f32 = st.f32;
  return k_group_norm(m->ctx, a, M, m->c.d_model);
}

int embed_rows(strictb200_model* m, const int32_t* ids, int64_t M, float* x) {
  SbStack& st = *m->stack;
  if (st.f32) return k_embedding_f32(m->ctx, (const float*)st.embed, nullptr, ids, nullptr, nullptr, M, st.dp, m->c.vocab, 0, x);
  return k_embedding_bf16_f32(m->ctx, (const bf16*)st.embed, ids, M, st.dp, m->c.vocab, x);
}

LatentSplitArgs split_args(strictb200_model* m, strictb200_kv* kv, int l, int b0) {
  SbStack& st = *m->stack;
  const StackLayer& w = st.L[l];
  LatentSplitArgs a;
  a.s = w.s; a.cos_t = w.cos_t; a.sin_t = w.sin_t; a.max_pos = m->c.max_pos; a.maxlen = kv->maxlen; a.norm_w = w.dkv_norm; a.eps = m->c.eps; a.f32 = st.f32;
  a.cache = w.own ? (char*)kv->k + (kv->layer_off[l] + (size_t)b0 * kv->maxlen * w.s.row()) * st.esz() : nullptr;
  return a;
}
const char* latents(strictb200_model* m, strictb200_kv* kv, int l, int b0) {
  const SbStack& st = *m->stack;
  return (const char*)kv->k + (kv->layer_off[st.L[l].src] + (size_t)b0 * kv->maxlen * st.L[l].s.row()) * st.esz();
}

// ------------------------------------------------------------------ mixers with heads or states
// The rows of a launch: those of a prompt chunk, or one next token for every sequence of the cache.
struct MixRows {
  int64_t T = 0;
  int b0 = 0, nb = 0, max_new = 0;
  const int32_t *seq = nullptr, *pos = nullptr, *qstart = nullptr, *past = nullptr;  // prompts only
  const int32_t* lens = nullptr;  // lengths after a prompt's rows, or before the next tokens
  bool prompt() const { return seq != nullptr; }
};
struct MixBufs {
  char *q = nullptr, *k = nullptr, *v = nullptr, *u = nullptr;
  float *gate = nullptr, *gates = nullptr, *o_part = nullptr, *ml_part = nullptr, *seg_state = nullptr;
};
void carve_mix(strictb200_model* m, const StackLayer& w, int64_t T, bool prompt, int nb, int max_new, char* base, MixBufs* o, size_t* total) {
  const size_t esz = m->stack->esz();
  Carver cv{base};
  if (w.kind == STRICTB200_MIXER_GATED) {
    o->u = cv.take<char>(T * w.gs.ld_u() * esz);
    o->gates = cv.take<float>(T * 2 * w.gs.width);
  } else if (w.kind != STRICTB200_MIXER_LATENT) {
    const size_t rows = (size_t)T * w.hs.H * w.hs.row();
    o->q = cv.take<char>(rows * esz);
    if (w.kind == STRICTB200_MIXER_RETENTION) {
      o->k = cv.take<char>(rows * esz);
      o->v = cv.take<char>(rows * esz);
      const int segs = prompt && !m->stack->f32 && sb_retention_prefill_fits(w.hs) ? sb_retention_segments(m->ctx, w.hs, nb, max_new) : 1;
      if (segs > 1) o->seg_state = cv.take<float>((size_t)segs * nb * w.state);
    } else {
      o->gate = cv.take<float>((size_t)T * w.hs.H);
      if (!prompt && w.fast_decode) {
        o->o_part = cv.take<float>(rows * 8);
        o->ml_part = cv.take<float>((size_t)T * w.hs.H * 8 * 2);
      }
    }
  }
  *total = cv.off;
}

// gates [T, 2 width] = u times the block-diagonal [r | i] matrices
int gate_product(strictb200_model* m, const StackLayer& w, int64_t T, const void* u, float* gates) {
  const GatedShape& g = w.gs;
  const int64_t bs = g.bs(), bp = g.bs_p(), n = 2 * bs;
  const bool f32 = m->stack->f32;
  const bool one = !f32 && n % (T <= 128 ? 128 : 256) == 0;  // every channel tile inside one block: a single launch
  for (int b = 0; b < (one ? 1 : g.blocks); b++) {
    if (f32) {
      GemmF32Args a;
      a.M = T; a.N = n; a.K = bp; a.x = (const float*)u + b * bp; a.ldx = g.ld_u(); a.w = (const float*)w.w_gate + b * n * bp; a.ldw = bp;
      a.y = gates + b * n; a.ldy = 2 * g.width;
      SB_TRY(k_gemm_f32(m->ctx, a));
      continue;
    }
    GemmBf16Args a;
    a.M = T; a.N = one ? 2 * g.width : n; a.K = bp; a.x = (const bf16*)u + b * bp; a.ldx = g.ld_u(); a.w = (const bf16*)w.w_gate + b * n * bp; a.ldw = bp;
    if (one) { a.group_n = (int)n; a.group_k = bp; }
    a.e.out_f32 = gates + b * n; a.e.ldo = 2 * g.width;
    SB_TRY(k_gemm_bf16(m->ctx, a));
  }
  return STRICTB200_OK;
}

// The mixer of layer l over the projection's rows p, its output to the first columns of oa. act: what the feed-forward's columns
// of p still need (kind 0: nothing).
int mix_rows(strictb200_model* m, strictb200_kv* kv, int l, const MixRows& r, const ProjRows& p, const ActArgs& act, char* scratch, void* oa) {
  strictb200_ctx* ctx = m->ctx;
  SbStack& st = *m->stack;
  const StackLayer& w = st.L[l];
  MixBufs b;
  size_t total;
  carve_mix(m, w, r.T, r.prompt(), r.nb, r.max_new, scratch, &b, &total);
  float* state = kv->state ? kv->state + kv->state_off[l] + (size_t)r.b0 * w.state : nullptr;
  if (w.kind == STRICTB200_MIXER_GATED) {
    GatedArgs a;
    a.s = w.gs; a.p = p; a.y_bias = w.y_bias; a.x_bias = w.x_bias; a.conv = w.conv; a.conv_bias = w.conv_bias; a.r_bias = w.r_bias; a.i_bias = w.i_bias;
    a.decay = w.decay;
    a.state = kv->state + kv->state_off[l] + (size_t)r.b0 * w.gs.width;
    a.hist = kv->state + kv->state_off[l] + (size_t)kv->B * w.gs.width + (size_t)r.b0 * (w.gs.taps - 1) * w.gs.width;
    a.seq = r.seq; a.qstart = r.qstart; a.lens = r.lens; a.past = r.past; a.nb = r.nb; a.max_new = r.max_new;
    a.u = b.u; a.gates = b.gates; a.out = oa; a.ldo = w.ldo; a.f32 = st.f32; a.act = act;
    PROF(STRICTB200_K_ROPE, k_gated_conv(ctx, a, r.T));
    PROF(STRICTB200_K_GATES, gate_product(m, w, r.T, b.u, b.gates));
    PROF(STRICTB200_K_RECURRENCE, k_gated_scan(ctx, a, r.T));
    return STRICTB200_OK;
  }
  const HeadShape& s = w.hs;
  RetentionArgs t;
  if (w.kind == STRICTB200_MIXER_RETENTION) {
    t.s = s; t.p = p; t.decay = w.decay; t.state = state; t.q = b.q; t.k = b.k; t.v = b.v; t.seg_state = b.seg_state; t.nb = r.nb; t.max_new = r.max_new;
    t.eps = m->c.eps; t.out = oa; t.ldo = w.ldo; t.f32 = st.f32; t.cos_t = w.cos_t; t.sin_t = w.sin_t; t.max_pos = m->c.max_pos;
    if (r.prompt()) { t.qstart = r.qstart; t.lens = r.lens; t.past = r.past; }
    else if (!st.f32 && sb_retention_decode_fits(s) && p.ld % 4 == 0) {
      t.cache_lens = r.lens; t.act = act;
      PROF(STRICTB200_K_RECURRENCE, k_retention_decode(ctx, t, r.T));
      return STRICTB200_OK;
    }
  }
  char *kc = nullptr, *vc = nullptr;
  if (w.kind == STRICTB200_MIXER_ATTENTION) {
    const size_t rows = (size_t)s.G * kv->maxlen * s.row();  // of one sequence
    kc = (char*)kv->k + (kv->layer_off[l] + (size_t)r.b0 * rows) * st.esz();
    vc = kc + (size_t)kv->B * rows * st.esz();
  }
  HeadSplitArgs a;
  a.s = s; a.p = p; a.seq = r.seq; a.pos = r.pos; a.lens = r.prompt() ? nullptr : r.lens; a.cos_t = w.cos_t; a.sin_t = w.sin_t; a.max_pos = m->c.max_pos;
  a.maxlen = kv->maxlen; a.eps = m->c.eps; a.q_out = b.q; a.k_out = kc ? kc : b.k; a.v_out = vc ? vc : b.v; a.dense = !kc; a.gate_out = b.gate; a.f32 = st.f32;
  a.act = act;
  PROF(STRICTB200_K_ROPE, k_head_split(ctx, a, r.T));
  if (w.kind == STRICTB200_MIXER_RETENTION) {
    const bool tc = r.prompt() && !st.f32 && sb_retention_prefill_fits(s);
    PROF(STRICTB200_K_RECURRENCE, tc ? k_retention_prefill(ctx, t, r.T) : k_retention_any(ctx, t));
    return STRICTB200_OK;
  }
  const float* gate = s.gate ? b.gate : nullptr;
  if (r.prompt() && w.fast_prefill) {
    HeadPrefillArgs h;
    h.q = (const bf16*)b.q; h.q_rows = r.T; h.k = (const bf16*)kc; h.v = (const bf16*)vc; h.lens = r.lens; h.past = r.past; h.qstart = r.qstart;
    h.B = r.nb; h.S = r.max_new; h.H = s.H; h.Hkv = s.G; h.maxlen = kv->maxlen; h.row_dims = s.row(); h.vdim = s.vdim; h.scale = s.scale; h.sink = s.sink;
    h.gate = gate; h.out = (bf16*)oa; h.ldo = w.ldo;
    return k_attn_prefill_heads(ctx, h);
  }
  if (!r.prompt() && w.fast_decode) {
    const int chunk = kv->layer_chunk[l] / 32, nsplit = kv->layer_chunk[l] % 32;
    PROF(STRICTB200_K_ATTN, k_attn_decode_chunks(ctx, s.row(), (const bf16*)b.q, (const bf16*)kc, (const bf16*)vc, r.lens, (int)r.T, s.H, s.G, kv->maxlen, s.scale, nsplit,
                                                 chunk, b.o_part, b.ml_part));
    PROF(STRICTB200_K_ATTN_MERGE, k_head_combine(ctx, s, b.o_part, b.ml_part, gate, r.lens, (int)r.T, kv->maxlen, chunk, nsplit, (bf16*)oa, w.ldo));
    return STRICTB200_OK;
  }
  PROF(STRICTB200_K_ATTN, k_head_attn_any(ctx, s, st.f32, b.q, kc, vc, gate, r.seq, r.pos, r.prompt() ? nullptr : r.lens, r.T, kv->maxlen, oa, w.ldo));
  return STRICTB200_OK;
}

// ------------------------------------------------------------------ decode
struct StackDec {
  float* x;        // [B, dp] residual stream
  char* h;         // [2][B, dp] the two norms
  float* part;     // split-K sums of the projection, or its finished rows
  float* part2;    // split-K sums of the output product
  char* q;         // queries, in latent space or not
  char* oa;        // [B, ldo] attention output | activation
  float* attn_ws;
  char* mix;       // the other mixers' rows (carve_mix)
  float* logits;
  void* am_ws;
};
void carve_dec(strictb200_model* m, strictb200_kv* kv, char* base, StackDec* o, size_t* total) {
  SbStack& st = *m->stack;
  const int64_t B = kv->B, d = m->c.d_model;
  size_t part = 1, part2 = 1, q = 1, oa = 1, ws = 4, mix = 1;
  for (const StackLayer& w : st.L) {
    const bool split = !st.f32 && (w.fast_decode || w.kind != STRICTB200_MIXER_LATENT);  // the projection as split-K sums
    const int s1 = split ? sb_gemm_bf16_splits(m->ctx, B, w.n_in, d) : 1;
    part = std::max(part, (size_t)s1 * B * w.n_in);
    if (split) {
      int first, all;
      out_splits(m->ctx, st, w, B, d, &first, &all);
      part2 = std::max(part2, (size_t)all * B * d);
    }
    oa = std::max(oa, (size_t)B * w.ldo);
    if (w.kind != STRICTB200_MIXER_LATENT) {
      MixBufs t;
      size_t n;
      carve_mix(m, w, B, false, (int)B, 1, nullptr, &t, &n);
      mix = std::max(mix, n);
      continue;
    }
    q = std::max(q, (size_t)B * w.s.H * std::max(w.s.row(), w.s.q_head()));
    if (w.fast_decode) ws = std::max(ws, sb_latent_decode_scratch(w.s, kv->B));
  }
  Carver cv{base};
  o->x = cv.take<float>(B * st.dp);
  o->h = cv.take<char>(2 * B * st.dp * st.esz());
  o->part = cv.take<float>(part);
  o->part2 = cv.take<float>(part2);
  o->q = cv.take<char>(q * st.esz());
  o->oa = cv.take<char>(oa * st.esz());
  o->attn_ws = cv.take<float>(ws / sizeof(float));
  o->mix = cv.take<char>(mix);
  o->logits = cv.take<float>(B * m->c.vocab);
  o->am_ws = cv.take<uint8_t>(sb_argmax_scratch(B, m->c.vocab));
  *total = cv.off;
}

// ------------------------------------------------------------------ prefill
struct StackPre {
  float* x;
  char* h;
  float* in;
  char *q, *oa, *mix;
  bf16 *kvx, *lat;
  int32_t* keys;   // [layers][2][nb]: row and position of every sequence's first key
  float *last, *logits;
  char* lasth;
  int32_t* pick;
  void* am_ws;
};
// first key position a layer's prompt rows of a sequence with `past` tokens can see
int first_key(const StackLayer& w, int past) { return w.kind == STRICTB200_MIXER_LATENT && w.s.window > 0 ? std::max(0, past - w.s.window + 1) : 0; }
int64_t key_rows(const StackLayer& w, const PrefillChunk& c) {
  int64_t n = 0;
  for (int j = 0; j < c.nb; j++) n += c.h_after[j] - first_key(w, c.h_past[j]);
  return n;
}
void carve_pre(strictb200_model* m, const PrefillChunk& c, char* base, StackPre* o, size_t* total) {
  SbStack& st = *m->stack;
  const int64_t T = c.T;
  size_t in = 1, q = 1, oa = 1, kvx = 1, lat = 1, mix = 1;
  for (const StackLayer& w : st.L) {
    in = std::max(in, (size_t)T * ld_in_of(st, w));
    oa = std::max(oa, (size_t)T * w.ldo);
    if (w.kind != STRICTB200_MIXER_LATENT) {
      MixBufs t;
      size_t n;
      carve_mix(m, w, T, true, c.nb, c.max_new, nullptr, &t, &n);
      mix = std::max(mix, n);
      continue;
    }
    q = std::max(q, (size_t)T * w.s.H * w.s.q_head());
    if (w.fast_prefill) {
      const size_t n = (size_t)key_rows(w, c);
      kvx = std::max(kvx, n * w.s.n_kv());
      if (c.nb > 1) lat = std::max(lat, n * w.s.row());
    }
  }
  Carver cv{base};
  o->x = cv.take<float>(T * st.dp);
  o->h = cv.take<char>(2 * T * st.dp * st.esz());
  o->in = cv.take<float>(in);
  o->q = cv.take<char>(q * st.esz());
  o->oa = cv.take<char>(oa * st.esz());
  o->kvx = cv.take<bf16>(kvx);
  o->lat = cv.take<bf16>(lat);
  o->mix = cv.take<char>(mix);
  o->keys = cv.take<int32_t>(st.L.size() * 2 * c.nb);
  o->last = cv.take<float>((size_t)c.n_rows * st.dp);
  o->lasth = cv.take<char>((size_t)2 * c.n_rows * st.dp * st.esz());
  o->logits = cv.take<float>((size_t)c.n_rows * m->c.vocab);
  o->pick = cv.take<int32_t>(c.n_rows);
  o->am_ws = cv.take<uint8_t>(sb_argmax_scratch(c.n_rows, m->c.vocab));
  *total = cv.off;
}

}  // namespace

int sb_stack_kv_layout(strictb200_model* m, strictb200_kv* kv, size_t* elements, size_t* state_floats) {
  SbStack& st = *m->stack;
  size_t off = 0, state = 0;
  kv->layer_off.resize(st.L.size());
  kv->state_off.resize(st.L.size());
  for (size_t l = 0; l < st.L.size(); l++) {
    const StackLayer& w = st.L[l];
    kv->layer_off[l] = off;
    kv->state_off[l] = state;
    if (w.kind == STRICTB200_MIXER_LATENT && w.own) off += (size_t)kv->B * kv->maxlen * w.s.row();
    if (w.kind == STRICTB200_MIXER_ATTENTION) off += 2 * (size_t)kv->B * w.hs.G * kv->maxlen * w.hs.row();
    state += (kv->B * w.state + 63) / 64 * 64;
  }
  kv->layer_chunk.assign(st.L.size(), 0);
  *elements = off;
  *state_floats = state;
  return STRICTB200_OK;
}

size_t sb_stack_esz(strictb200_model* m) { return m->stack->esz(); }
size_t sb_stack_decode_bytes(strictb200_model* m, strictb200_kv* kv) {
  StackDec b;
  size_t total;
  carve_dec(m, kv, nullptr, &b, &total);
  return total;
}
float* sb_stack_decode_logits(strictb200_model* m, strictb200_kv* kv) {
  StackDec b;
  size_t total;
  carve_dec(m, kv, (char*)kv->dec, &b, &total);
  return b.logits;
}

// Key chunks of every layer's decode attention, for the lengths the cache holds now (and up to 256 keys more).
bool sb_stack_plan(strictb200_model* m, strictb200_kv* kv, int longest) {
  SbStack& st = *m->stack;
  bool changed = false;
  if (longest > kv->plan_until) {
    const int len = std::min(kv->maxlen, (longest + 255) / 256 * 256);
    for (size_t l = 0; l < st.L.size(); l++) {
      if (!st.L[l].fast_decode) continue;
      const LatentShape& s = st.L[l].s;
      const bool latent = st.L[l].kind == STRICTB200_MIXER_LATENT;
      const int chunk = latent ? sb_latent_decode_chunk(m->ctx, s, kv->B, len) : sb_attn_decode_chunk(m->ctx, kv->B, st.L[l].hs.G, kv->maxlen, len);
      const int n = latent && s.window > 0 ? std::min(s.window, len) : len;
      const int code = chunk * 32 + (n + chunk - 1) / chunk;  // keys per chunk and chunks
      if (code != kv->layer_chunk[l]) { kv->layer_chunk[l] = code; changed = true; }
    }
    kv->plan_until = len;
  }
  if (kv->plan_version != st.version) { kv->plan_version = st.version; changed = true; }
  return changed;
}

int sb_stack_decode_body(strictb200_model* m, strictb200_kv* kv) {
  strictb200_ctx* ctx = m->ctx;
  SbStack& st = *m->stack;
  const int64_t B = kv->B, d = m->c.d_model;
  StackDec b;
  size_t total;
  carve_dec(m, kv, (char*)kv->dec, &b, &total);
  PROF(STRICTB200_K_EMBED, embed_rows(m, kv->d_ids, B, b.x));
  Pending pend;
  MixRows rows;
  rows.T = B; rows.nb = (int)B; rows.max_new = 1; rows.lens = kv->d_lens;
  for (int l = 0; l < (int)st.L.size(); l++) {
    const StackLayer& w = st.L[l];
    PROF(STRICTB200_K_ROWNORM, norm_rows(m, &w, B, b.x, pend, b.h));
    pend = Pending();
    if (w.kind != STRICTB200_MIXER_LATENT) {
      ProjRows p;
      ActArgs act;
      if (st.f32) {
        const int64_t ld_in = ld_in_of(st, w);
        PROF(STRICTB200_K_GEMM_QKV, project_in(m, w, B, b.h, b.part, ld_in, b.oa));
        p = ProjRows{b.part, ld_in, 1};
      } else {
        GemmBf16Args g = gemm_in_args(st, w, d, B, b.h);
        g.part = b.part; g.splits = sb_gemm_bf16_splits(ctx, B, w.n_in, d);
        PROF(STRICTB200_K_GEMM_QKV, k_gemm_bf16(ctx, g));
        p = ProjRows{b.part, w.n_in, g.splits};
        act = act_args(w, b.oa, 2);
      }
      SB_TRY(mix_rows(m, kv, l, rows, p, act, b.mix, b.oa));
      if (st.f32 || B > 256) {
        PROF(STRICTB200_K_GEMM_O, project_out(m, w, B, b.oa, b.x));
      } else {
        PROF(STRICTB200_K_GEMM_O, out_parts(m, w, B, b.oa, b.part2, &pend));
      }
      continue;
    }
    if (!w.fast_decode) {  // fp32, and widths the tensor-core kernels do not take: the prompt's kernels on B rows
      const int64_t ld_in = ld_in_of(st, w);
      PROF(STRICTB200_K_GEMM_QKV, project_in(m, w, B, b.h, b.part, ld_in, b.oa));
      LatentSplitArgs a = split_args(m, kv, l, 0);
      a.in = b.part; a.ld_in = ld_in; a.lens = kv->d_lens; a.q_out = b.q;
      PROF(STRICTB200_K_ROPE, k_latent_split(ctx, a, B));
      PROF(STRICTB200_K_ATTN, k_latent_attn_any(ctx, w.s, st.f32, b.q, latents(m, kv, l, 0), w.w_kv, nullptr, nullptr, kv->d_lens, B, kv->maxlen, b.oa, w.ldo));
      PROF(STRICTB200_K_GEMM_O, project_out(m, w, B, b.oa, b.x));
      continue;
    }
    GemmBf16Args g = gemm_in_args(st, w, d, B, b.h);
    g.part = b.part; g.splits = sb_gemm_bf16_splits(ctx, B, w.n_in, d);
    PROF(STRICTB200_K_GEMM_QKV, k_gemm_bf16(ctx, g));
    LatentDecodeInArgs in;
    in.a = split_args(m, kv, l, 0);
    in.a.in = b.part; in.a.ld_in = w.n_in; in.a.splits = g.splits; in.a.lens = kv->d_lens;
    in.wkv = (const bf16*)w.w_kv; in.q_abs = (bf16*)b.q;
    in.act_col = (int)w.n_switch; in.n_act = w.ff; in.act_pos = w.act_pos; in.act_neg = w.act_neg;
    in.act = (bf16*)b.oa + w.ko_p; in.ld_act = w.ldo;
    PROF(STRICTB200_K_ROPE, k_latent_decode_in(ctx, in, B));
    PROF(STRICTB200_K_ATTN, k_latent_attn_decode(ctx, w.s, (const bf16*)b.q, (const bf16*)latents(m, kv, l, 0), kv->d_lens, (int)B, kv->maxlen,
                                                 kv->layer_chunk[l] / 32, kv->layer_chunk[l] % 32, (bf16*)b.attn_ws, (const bf16*)w.w_kv, (bf16*)b.oa, w.ldo));
    PROF(STRICTB200_K_GEMM_O, out_parts(m, w, B, b.oa, b.part2, &pend));
  }
  PROF(STRICTB200_K_ROWNORM, norm_rows(m, nullptr, B, b.x, pend, b.h));
  PROF(STRICTB200_K_HEAD, head_rows(m, B, b.h, b.logits));
  PROF(STRICTB200_K_HEAD, k_argmax(ctx, b.logits, B, m->c.vocab, m->c.vocab, kv->d_next, nullptr, b.am_ws));
  PROF(STRICTB200_K_EMBED, k_add_i32(ctx, kv->d_lens, nullptr, 1, B));
  return STRICTB200_OK;
}

size_t sb_stack_prefill_bytes(strictb200_model* m, const PrefillChunk& c) {
  StackPre b;
  size_t total;
  carve_pre(m, c, nullptr, &b, &total);
  return total;
}

int sb_stack_prefill_chunk(strictb200_model* m, strictb200_kv* kv, const PrefillChunk& c, char* scratch) {
  strictb200_ctx* ctx = m->ctx;
  SbStack& st = *m->stack;
  const int64_t T = c.T;
  StackPre b;
  size_t total;
  carve_pre(m, c, scratch, &b, &total);
  std::vector<int32_t> keys(st.L.size() * 2 * c.nb);
  for (size_t l = 0; l < st.L.size(); l++) {
    int32_t off = 0;
    for (int j = 0; j < c.nb; j++) {
      const int k0 = first_key(st.L[l], c.h_past[j]);
      keys[(2 * l) * c.nb + j] = off;
      keys[(2 * l + 1) * c.nb + j] = k0;
      off += c.h_after[j] - k0;
    }
  }
  SB_CUDA(cudaMemcpyAsync(b.keys, keys.data(), keys.size() * 4, cudaMemcpyHostToDevice, ctx->stream));
  if (st.pads) {  // padding columns meet zero weights, but they must be finite
    size_t oa = 0;
    for (const StackLayer& w : st.L) oa = std::max(oa, (size_t)T * w.ldo);
    SB_CUDA(cudaMemsetAsync(b.oa, 0, oa * st.esz(), ctx->stream));
    SB_CUDA(cudaMemsetAsync(b.h, 0, 2 * T * st.dp * st.esz(), ctx->stream));
    SB_CUDA(cudaMemsetAsync(b.lasth, 0, (size_t)2 * c.n_rows * st.dp * st.esz(), ctx->stream));
  }
  SB_TRY(embed_rows(m, c.ix.tok, T, b.x));
  MixRows rows;
  rows.T = T; rows.b0 = c.b0; rows.nb = c.nb; rows.max_new = c.max_new; rows.seq = c.ix.seq; rows.pos = c.ix.pos; rows.qstart = c.ix.qs; rows.past = c.ix.past;
  rows.lens = c.ix.la;
  for (int l = 0; l < (int)st.L.size(); l++) {
    const StackLayer& w = st.L[l];
    const LatentShape& s = w.s;
    const int64_t ld_in = ld_in_of(st, w);
    SB_TRY(norm_rows(m, &w, T, b.x, Pending(), b.h));
    SB_TRY(project_in(m, w, T, b.h, b.in, ld_in, b.oa));
    if (w.kind != STRICTB200_MIXER_LATENT) {
      SB_TRY(mix_rows(m, kv, l, rows, ProjRows{b.in, ld_in, 1}, ActArgs(), b.mix, b.oa));
      SB_TRY(project_out(m, w, T, b.oa, b.x));
      continue;
    }
    LatentSplitArgs a = split_args(m, kv, l, c.b0);
    a.in = b.in; a.ld_in = ld_in; a.seq = c.ix.seq; a.pos = c.ix.pos; a.q_out = b.q;
    SB_TRY(k_latent_split(ctx, a, T));
    const char* lat = latents(m, kv, l, c.b0);
    if (!w.fast_prefill) {
      SB_TRY(k_latent_attn_any(ctx, s, st.f32, b.q, lat, w.w_kv, c.ix.seq, c.ix.pos, nullptr, T, kv->maxlen, b.oa, w.ldo));
    } else {
      const int64_t n = key_rows(w, c);
      const int32_t *koff = b.keys + 2 * l * c.nb, *kpos0 = koff + c.nb;
      const bf16* rows;
      if (c.nb == 1) {  // one sequence: its latents lie together in the cache
        rows = (const bf16*)lat + (int64_t)first_key(w, c.h_past[0]) * s.row();
      } else {
        SB_TRY(k_latent_gather(ctx, (const bf16*)lat, kv->maxlen, s.row(), koff, kpos0, c.ix.la, c.nb, (int)std::min<int64_t>(n, INT32_MAX), b.lat));
        rows = b.lat;
      }
      GemmBf16Args g;
      g.M = n; g.N = s.n_kv(); g.K = s.rank; g.x = rows; g.ldx = s.row(); g.w = (const bf16*)w.w_kv; g.ldw = s.rank_p();
      g.e.out_bf16 = b.kvx; g.e.ldo = s.n_kv();
      SB_TRY(k_gemm_bf16(ctx, g));
      LatentPrefillArgs p;
      p.q = (const bf16*)b.q; p.q_rows = T; p.q_head = s.q_head(); p.q_rot = s.dim_p();
      p.k = b.kvx; p.v = b.kvx + (int64_t)s.H * s.kv_head(); p.k_rows = n; p.ldk = s.n_kv(); p.k_head = p.v_head = s.kv_head();
      p.k_rot = rows + s.rank_p(); p.ld_rot = s.row();
      p.lens = c.ix.la; p.past = c.ix.past; p.qstart = c.ix.qs; p.koff = koff; p.kpos0 = kpos0;
      p.B = c.nb; p.S = c.max_new; p.H = s.H; p.dim = s.dim; p.rot = s.rot; p.vdim = s.vdim; p.window = s.window; p.scale = s.scale;
      p.out = (bf16*)b.oa; p.ldo = w.ldo;
      SB_TRY(k_attn_prefill_latent(ctx, p));
    }
    SB_TRY(project_out(m, w, T, b.oa, b.x));
  }
  SB_TRY(k_gather_rows(ctx, b.x, c.ix.last, c.n_rows, st.dp * 4, b.last));
  SB_TRY(norm_rows(m, nullptr, c.n_rows, b.last, Pending(), b.lasth));
  SB_TRY(head_rows(m, c.n_rows, b.lasth, b.logits));
  SB_TRY(k_argmax(ctx, b.logits, c.n_rows, m->c.vocab, m->c.vocab, b.pick, nullptr, b.am_ws));
  SB_CUDA(cudaMemcpyAsync(c.d_next, b.pick + (c.n_rows - c.nb), (size_t)c.nb * 4, cudaMemcpyDeviceToDevice, ctx->stream));
  if (c.h_logits) SB_CUDA(cudaMemcpyAsync(c.h_logits, b.logits, (size_t)c.n_logits * m->c.vocab * 4, cudaMemcpyDeviceToHost, ctx->stream));
  SB_CUDA(cudaStreamSynchronize(ctx->stream));
  return STRICTB200_OK;
}

uint64_t sb_stack_cache_read_bytes(strictb200_model* m, int len) {
  uint64_t n = 0;
  for (const StackLayer& w : m->stack->L) {
    if (w.kind == STRICTB200_MIXER_LATENT) n += (uint64_t)(w.s.window > 0 ? std::min(len, w.s.window) : len) * w.s.row() * m->stack->esz();
    if (w.kind == STRICTB200_MIXER_ATTENTION) n += (uint64_t)len * w.hs.G * (w.hs.dim + w.hs.vdim) * m->stack->esz();
    n += (uint64_t)w.state * 2 * sizeof(float);  // read and written
  }
  return n;
}

void sb_stack_destroy(strictb200_model* m) {
  delete m->stack;
  m->stack = nullptr;
}

int sb_stack_tensor(strictb200_model* m, const char* name, const void* h_in, void* h_out, size_t bytes) {
  strictb200_ctx* ctx = m->ctx;
  Slot s;
  if (!find_slot(m, name, &s)) return sb_fail(STRICTB200_ERR_INVALID_ARG, std::string("unknown tensor ") + name);
  const size_t n = (size_t)s.rows * s.cols;
  if (bytes != n * 2 && bytes != n * 4)
    return sb_fail(STRICTB200_ERR_INVALID_ARG, std::string("tensor ") + name + " has " + std::to_string(n) + " elements: bf16 or fp32 host data");
  const bool f32 = bytes == n * 4;
  if (s.host) {
    for (size_t i = 0; i < n; i++) {
      if (h_in) {
        if (f32) s.host[i] = ((const float*)h_in)[i];
        else { const uint32_t u = (uint32_t)((const uint16_t*)h_in)[i] << 16; std::memcpy(&s.host[i], &u, 4); }
      } else if (f32) {
        ((float*)h_out)[i] = s.host[i];
      } else {
        ((bf16*)h_out)[i] = __float2bfloat16_rn(s.host[i]);
      }
    }
    if (h_in) {
      for (StackLayer& w : m->stack->L) set_act(w);
      m->stack->version++;
    }
    return STRICTB200_OK;
  }
  void* tmp;
  SB_CUDA(cudaMalloc(&tmp, bytes));
  int st = STRICTB200_OK;
  cudaError_t e = cudaSuccess;
  if (h_in) e = cudaMemcpyAsync(tmp, h_in, bytes, cudaMemcpyHostToDevice, ctx->stream);
  if (e == cudaSuccess) st = place(ctx, s, tmp, f32, h_in == nullptr);
  if (e == cudaSuccess && st == STRICTB200_OK && h_out) e = cudaMemcpyAsync(h_out, tmp, bytes, cudaMemcpyDeviceToHost, ctx->stream);
  const cudaError_t e2 = cudaStreamSynchronize(ctx->stream);
  cudaFree(tmp);
  if (h_in && s.lam && st == STRICTB200_OK && e == cudaSuccess) SB_TRY(set_decay(ctx, *s.lam));
  if (e != cudaSuccess || e2 != cudaSuccess) return sb_fail(STRICTB200_ERR_CUDA, std::string("tensor ") + name + ": " + cudaGetErrorString(e != cudaSuccess ? e : e2));
  return st;
}

int sb_stack_init_random(strictb200_model* m, uint64_t seed) {
  strictb200_ctx* ctx = m->ctx;
  SbStack& st = *m->stack;
  const float SD = 0.02f;
  auto fill = [&](const std::string& name, uint64_t id) -> int {
    Slot s;
    if (!find_slot(m, name, &s)) return STRICTB200_OK;  // a part this layer does not have
    const int64_t n = s.rows * s.cols;
    void* tmp;
    SB_CUDA(cudaMalloc(&tmp, (size_t)n * 2));
    int r = k_gen_normal_bf16(ctx, sb_stream_key(seed, id), 0, n, SD, (bf16*)tmp);
    if (r == STRICTB200_OK) r = place(ctx, s, tmp, false, false);
    cudaStreamSynchronize(ctx->stream);
    cudaFree(tmp);
    return r;
  };
  SB_TRY(fill("embed", G_EMBED));
  SB_TRY(fill("head", G_HEAD));
  SB_TRY(fill_f32(ctx, st.normf, m->c.d_model, 1.f));
  for (int l = 0; l < (int)st.L.size(); l++) {
    StackLayer& w = st.L[l];
    const std::string p = "l" + std::to_string(l) + ".";
    SB_TRY(fill_f32(ctx, w.norm1, m->c.d_model, 1.f));
    if (w.norm2) SB_TRY(fill_f32(ctx, w.norm2, m->c.d_model, 1.f));
    if (w.dkv_norm) SB_TRY(fill_f32(ctx, w.dkv_norm, w.s.rank, 1.f));
    for (float* scale : {w.ls1, w.ls2})
      if (scale) SB_TRY(fill_f32(ctx, scale, m->c.d_model, 1.f));
    if (w.kind == STRICTB200_MIXER_LATENT) {
      SB_TRY(fill(p + "mix.q", layer_tensor(l, T_Q)));
      SB_TRY(fill(p + "mix.dkv", layer_tensor(l, T_DKV)));
      SB_TRY(fill(p + "mix.uk", layer_tensor(l, T_UK)));
      SB_TRY(fill(p + "mix.uv", layer_tensor(l, T_UV)));
    } else if (w.kind == STRICTB200_MIXER_GATED) {
      for (float* zero : {w.y_bias, w.x_bias, w.conv_bias, w.r_bias, w.i_bias, w.lam}) SB_TRY(fill_f32(ctx, zero, w.gs.width, 0.f));
      SB_TRY(fill(p + "mix.y", layer_tensor(l, T_Q)));
      SB_TRY(fill(p + "mix.x", layer_tensor(l, T_K)));
      SB_TRY(fill(p + "mix.conv", layer_tensor(l, T_CONV)));
      SB_TRY(fill(p + "mix.ra", layer_tensor(l, T_RA)));
      SB_TRY(fill(p + "mix.ri", layer_tensor(l, T_RI)));
      SB_TRY(set_decay(ctx, w));
    } else {
      SB_TRY(fill(p + "mix.q", layer_tensor(l, T_Q)));
      SB_TRY(fill(p + "mix.k", layer_tensor(l, T_K)));
      SB_TRY(fill(p + "mix.v", layer_tensor(l, T_V)));
      SB_TRY(fill(p + "mix.g", layer_tensor(l, T_G)));
    }
    SB_TRY(fill(p + "mix.o", layer_tensor(l, T_O)));
    if (w.glu()) SB_TRY(fill(p + "mlp.gate", layer_tensor(l, T_GATE)));
    SB_TRY(fill(p + "mlp.up", layer_tensor(l, T_UP)));
    SB_TRY(fill(p + "mlp.down", layer_tensor(l, T_DOWN)));
    w.act[0] = w.act[1] = 0.f;
    set_act(w);
  }
  st.version++;
  return STRICTB200_OK;
}

extern "C" int strictb200_stack_create(strictb200_ctx* ctx, const strictb200_stack_config* cfg, const strictb200_layer_config* layers, strictb200_model** out) {
  SB_ENTER(ctx);
  SB_REQUIRE(cfg && layers && out, "null argument");
  *out = nullptr;
  const strictb200_stack_config& c = *cfg;
  if (ctx->tp_world != 1) return sb_fail(STRICTB200_ERR_UNSUPPORTED, "models described layer by layer are single-GPU");
  SB_REQUIRE(c.n_layers > 0 && c.d_model > 0 && c.vocab > 0 && c.max_pos > 0 && c.eps > 0, "non-positive dimension");
  SB_REQUIRE(c.norm_groups > 0 && c.d_model % c.norm_groups == 0, "the width must be a multiple of the norm groups");
  SB_REQUIRE(c.residual_mult != 0 && c.logit_scale != 0, "the residual and the logits need a factor");
  SB_REQUIRE(c.dtype == STRICTB200_BF16 || c.dtype == STRICTB200_FP32, "unknown dtype");
  for (int l = 0; l < c.n_layers; l++) {
    const strictb200_layer_config& y = layers[l];
    const std::string at = "layer " + std::to_string(l) + ": ";
    if (y.mlp != STRICTB200_MLP_NONE && y.mlp != STRICTB200_MLP_XIELU && y.mlp != STRICTB200_MLP_RELU_GLU) return sb_fail(STRICTB200_ERR_UNSUPPORTED, at + "unknown feed-forward");
    SB_REQUIRE(y.mlp == STRICTB200_MLP_NONE || y.d_ff > 0, "bad feed-forward size");
    if (y.mixer == STRICTB200_MIXER_GATED) {
      SB_REQUIRE(y.width > 0 && y.blocks > 0 && y.width % y.blocks == 0 && y.conv > 0, "bad mixer size");
      continue;
    }
    SB_REQUIRE(y.heads > 0 && y.dim > 0 && y.vdim > 0 && y.rot_dim >= 0 && y.rot_dim % 2 == 0 && y.heads <= 65535, "bad mixer size");
    SB_REQUIRE(y.rot_dim == 0 || y.rot_base > 0, "bad mixer constant");
    SB_REQUIRE(y.rot_factor >= 0 && (y.rot_factor == 0 || (y.rot_dim > 0 && y.rot_base > 1 && y.rot_original > 0 && y.rot_fast > 0 && y.rot_slow > 0)), "bad rotation scaling");
    if (y.mixer == STRICTB200_MIXER_ATTENTION || y.mixer == STRICTB200_MIXER_RETENTION) {
      SB_REQUIRE(y.rot_dim <= y.dim && y.dim <= 1536 && y.vdim <= 1536, "bad mixer size");
      if (y.mixer == STRICTB200_MIXER_ATTENTION) {
        SB_REQUIRE(y.kv_heads > 0 && y.heads % y.kv_heads == 0 && y.scale > 0, "bad mixer size");
      } else {
        SB_REQUIRE(y.decay, "retention needs a decay per head");
        for (int h = 0; h < y.heads; h++) SB_REQUIRE(y.decay[h] >= 0 && y.decay[h] <= 1, "a decay lies between 0 and 1");
      }
      continue;
    }
    if (y.mixer != STRICTB200_MIXER_LATENT) return sb_fail(STRICTB200_ERR_UNSUPPORTED, at + "unknown mixer");
    SB_REQUIRE(y.kv_rank > 0 && y.window >= 0 && y.scale > 0, "bad mixer size");
    if (y.kv_from >= 0) {
      SB_REQUIRE(y.kv_from < l, "a layer can only read the latents of an earlier layer");
      const strictb200_layer_config& z = layers[y.kv_from];
      SB_REQUIRE(z.mixer == STRICTB200_MIXER_LATENT && z.kv_from < 0, "the layer whose latents are read must have its own");
      SB_REQUIRE(z.kv_rank == y.kv_rank && z.rot_dim == y.rot_dim && z.rot_base == y.rot_base, "layers that share latents must agree on their rank and rotation");
    }
  }
  strictb200_model* m = new strictb200_model;
  SbStack* st = new SbStack;
  m->ctx = ctx; m->stack = st;
  m->c = strictb200_model_config{};
  m->c.arch = STRICTB200_STACK; m->c.n_layers = c.n_layers; m->c.d_model = c.d_model; m->c.vocab = c.vocab; m->c.max_pos = c.max_pos; m->c.eps = (float)c.eps;
  m->c.n_q_heads = std::max(layers[0].heads, 1); m->c.n_kv_heads = 1; m->c.head_dim = layers[0].dim; m->c.d_ff = layers[0].d_ff;
  m->V_l = c.vocab;
  st->f32 = c.dtype == STRICTB200_FP32; st->groups = c.norm_groups; st->dp = pad8(c.d_model);
  st->shared_norm = c.shared_norm != 0; st->layer_scale = c.layer_scale != 0; st->mult = (float)c.residual_mult; st->logit_scale = (float)c.logit_scale;
  st->pads = st->dp != c.d_model;
  int r;
  auto fail = [&](int e) { strictb200_model_destroy(m); return e; };
#define S_TRY(e) do { r = (e); if (r != STRICTB200_OK) return fail(r); } while (0)
  const size_t es = st->esz();
  auto gains = [&](float** p, int64_t n) -> int { SB_TRY(dalloc(m, p, (size_t)n)); return fill_f32(ctx, *p, (size_t)n, 1.f); };
  S_TRY(zalloc(m, &st->embed, (size_t)c.vocab * st->dp * es));
  S_TRY(zalloc(m, &st->head, (size_t)c.vocab * st->dp * es));
  S_TRY(gains(&st->normf, c.d_model));
  m->weight_bytes += (uint64_t)c.vocab * c.d_model * es;
  st->L.resize(c.n_layers);
  for (int l = 0; l < c.n_layers; l++) {
    const strictb200_layer_config& y = layers[l];
    StackLayer& w = st->L[l];
    LatentShape& s = w.s;
    w.kind = y.mixer; w.mlp = y.mlp;
    w.ff = y.mlp == STRICTB200_MLP_NONE ? 0 : y.d_ff;
    w.src = l;
    if (w.kind != STRICTB200_MIXER_GATED) {
      w.base = y.rot_base; w.rot = y.rot_dim;
      w.scaling = RopeScaling{y.rot_factor, y.rot_original, y.rot_fast, y.rot_slow};
    }
    if (w.kind == STRICTB200_MIXER_LATENT) {
      s.H = y.heads; s.dim = y.dim; s.rot = y.rot_dim; s.vdim = y.vdim; s.rank = y.kv_rank; s.window = y.window; s.scale = (float)y.scale;
      w.own = y.kv_from < 0;
      w.src = w.own ? l : y.kv_from;
      w.n0 = s.n_q() + (w.own ? s.rank + s.rot : 0);
      w.ko_p = pad8(w.n_out());
      w.fast_prefill = !st->f32 && sb_latent_prefill_fits(s.dim, s.rot, s.vdim) && s.rot > 0;
      w.fast_decode = !st->f32 && sb_latent_decode_fits(s) && !w.glu();
      if (st->layer_scale) w.ko_p = pad64(w.n_out());
    } else if (w.kind == STRICTB200_MIXER_GATED) {
      w.gs.width = y.width; w.gs.taps = y.conv; w.gs.blocks = y.blocks;
      w.n0 = 2 * (int64_t)y.width;
      w.state = (size_t)y.width * y.conv;  // the recurrence's and the convolution's
      w.ko_p = pad64(w.n_out());
    } else {
      HeadShape& q = w.hs;
      const bool ret = w.kind == STRICTB200_MIXER_RETENTION;
      q.H = y.heads; q.G = ret ? y.heads : y.kv_heads; q.dim = y.dim; q.vdim = y.vdim; q.rot = y.rot_dim;
      if (ret) {
        q.k_scale = (float)(1.0 / std::sqrt((double)y.dim));
        w.state = (size_t)y.heads * y.dim * y.vdim;
        w.n0 = (int64_t)y.heads * 2 * (y.dim + y.vdim);
      } else {
        q.scale = (float)y.scale; q.qk_norm = y.qk_norm != 0; q.sink = y.sink != 0; q.gate = y.gate != 0;
        w.n0 = q.n_in();
        w.fast_prefill = !st->f32 && q.row() <= 128;
        w.fast_decode = !st->f32 && q.row() <= 128 && q.H / q.G <= 16;
      }
      w.ko_p = pad64(w.n_out());
    }
    const bool latent = w.kind == STRICTB200_MIXER_LATENT;
    w.n_switch = w.ff ? (w.n0 + 255) / 256 * 256 : 0;
    w.n_in = !w.ff ? (latent ? w.n0 : pad8(w.n0)) : w.n_switch + (w.glu() ? 2 * pad8(w.ff) : w.ff);
    w.ldo = w.ko_p + pad8(w.ff);
    if (w.ldo != w.n_out() + w.ff) st->pads = true;
    if (w.n_in > INT32_MAX || w.ldo > INT32_MAX) return fail(sb_fail(STRICTB200_ERR_INVALID_ARG, "layer too wide"));
    S_TRY(zalloc(m, &w.w_in, (size_t)w.n_in * st->dp * es));
    if (latent) S_TRY(zalloc(m, &w.w_kv, (size_t)s.n_kv() * s.rank_p() * es));
    S_TRY(zalloc(m, &w.w_out, (size_t)c.d_model * w.ldo * es));
    S_TRY(gains(&w.norm1, c.d_model));
    if (w.ff && !st->shared_norm) S_TRY(gains(&w.norm2, c.d_model));
    if (st->layer_scale) S_TRY(gains(&w.ls1, c.d_model));
    if (st->layer_scale && w.ff) S_TRY(gains(&w.ls2, c.d_model));
    if (w.kind == STRICTB200_MIXER_GATED) {
      const size_t n = (size_t)y.width;
      S_TRY(zalloc(m, &w.w_gate, 2 * n * w.gs.bs_p() * es));
      for (float** p : {&w.y_bias, &w.x_bias, &w.conv_bias, &w.r_bias, &w.i_bias, &w.lam, &w.decay}) S_TRY(zalloc(m, (void**)p, n * 4));
      S_TRY(zalloc(m, (void**)&w.conv, n * y.conv * 4));
      S_TRY(set_decay(ctx, w));
    }
    if (w.kind == STRICTB200_MIXER_RETENTION) {
      std::vector<float> decay(y.decay, y.decay + y.heads);
      S_TRY(dalloc(m, &w.decay, decay.size()));
      if (cudaMemcpy(w.decay, decay.data(), decay.size() * 4, cudaMemcpyHostToDevice) != cudaSuccess) return fail(sb_fail(STRICTB200_ERR_CUDA, "model set-up failed"));
    }
    if (latent && w.own) S_TRY(gains(&w.dkv_norm, s.rank));
    set_act(w);
    for (int k = 0; k < l && w.rot > 0; k++)
      if (st->L[k].base == w.base && st->L[k].rot == w.rot && st->L[k].scaling == w.scaling) { w.cos_t = st->L[k].cos_t; w.sin_t = st->L[k].sin_t; break; }
    if (w.rot > 0 && !w.cos_t) {
      S_TRY(sb_rope_table(ctx, c.max_pos, w.rot, y.rot_base, &w.cos_t, &w.sin_t, w.scaling));
      m->allocs.push_back(w.cos_t);
      m->allocs.push_back(w.sin_t);
    }
    m->weight_bytes += ((uint64_t)(w.n0 + (w.glu() ? 2 : 1) * w.ff) * c.d_model + (uint64_t)c.d_model * (w.n_out() + w.ff)) * es;
    if (latent) m->weight_bytes += (uint64_t)s.H * (s.dim + s.vdim) * s.rank * es;
    if (w.kind == STRICTB200_MIXER_GATED) m->weight_bytes += 2ull * w.gs.width * w.gs.bs() * es;
  }
  if (cudaStreamSynchronize(ctx->stream) != cudaSuccess) return fail(sb_fail(STRICTB200_ERR_CUDA, "model set-up failed"));
#undef S_TRY
  *out = m;
  return STRICTB200_OK;
}
