// Model and KV-cache objects shared by the schedules (model.cu: GPT-2 and Qwen3; stack.cu: models described layer by layer).
#pragma once
#include <algorithm>
#include <cmath>
#include <cstring>
#include <string>
#include <vector>

#include "common.cuh"

enum { T_NORM1 = 0, T_Q = 1, T_K = 2, T_V = 3, T_QN = 4, T_KN = 5, T_O = 6, T_NORM2 = 7, T_GATE = 8, T_UP = 9, T_DOWN = 10 };
enum { G_EMBED = 1, G_WPE = 2, G_HEAD = 3, G_NORMF = 4 };
inline uint64_t layer_tensor(int l, int kind) { return 16ull * (uint64_t)(l + 1) + (uint64_t)kind; }

struct QW {
  uint8_t* q = nullptr;
  float* s = nullptr;
  int64_t N = 0, K = 0;
};
struct FW {
  float* w = nullptr;
  float* b = nullptr;
  int64_t N = 0, K = 0;
};
struct LayerW {
  float *norm1_g = nullptr, *norm1_b = nullptr, *norm2_g = nullptr, *norm2_b = nullptr, *qn_g = nullptr, *kn_g = nullptr;
  QW wqkv, wo, wgu, wdown;
  FW fqkv, fo, ffc, fproj;
};

struct SbStack;  // stack.cu: weights and plan of a model described layer by layer

struct strictb200_model {
  strictb200_ctx* ctx = nullptr;
  strictb200_model_config c;
  int world = 1, rank = 0;
  int Hq_l = 0, Hkv_l = 0;
  int64_t I_l = 0, V_l = 0;
  std::vector<LayerW> L;
  bf16* embed = nullptr;   // Qwen3
  float* wte = nullptr;    // GPT-2
  float* wpe = nullptr;
  float *normf_g = nullptr, *normf_b = nullptr;
  QW head;
  float *rope_cos = nullptr, *rope_sin = nullptr;
  std::vector<void*> allocs;
  uint64_t weight_bytes = 0;  // bytes of the tensors a decode step streams (linears + head)
  int use_graph = 1;
  SbStack* stack = nullptr;
};

struct strictb200_kv {
  strictb200_model* m = nullptr;
  int B = 0, maxlen = 0;
  void *k = nullptr, *v = nullptr;
  size_t layer_stride = 0;  // elements per layer
  int32_t* d_lens = nullptr;
  std::vector<int32_t> h_lens;
  // decode state
  int32_t *d_ids = nullptr, *d_next = nullptr, *d_hist = nullptr;
  int hist_cap = 0;
  void* dec = nullptr;  // one allocation carved into the decode buffers
  size_t dec_bytes = 0;
  cudaGraphExec_t graph = nullptr;
  uint64_t graph_kernels = 0;
  bool warmed = false;
  int nsplit = 1;        // key chunks per sequence of the decode attention, and
  int chunk = 0;         // keys per chunk: planned for the lengths the cache holds now (plan_attention), 0 = not planned yet
  int plan_until = 0;    // the plan is kept until a sequence grows beyond this length
  std::vector<void*> allocs;
  std::vector<size_t> layer_off;           // stack models: first element of a layer's rows in k
  float* state = nullptr;                  // stack models: states of the recurrent layers (zero before a sequence's first token)
  size_t state_floats = 0;
  std::vector<size_t> state_off;           // first float of a layer's states
  std::vector<int> layer_chunk;            // stack models: keys per chunk (x 32) + chunks of every layer's decode attention
  uint64_t plan_version = 0;               // stack models: constants the recorded step was made with
};

template <typename T>
inline int dalloc(strictb200_model* m, T** p, size_t count) {
  *p = nullptr;
  if (!count) return STRICTB200_OK;
  void* v;
  SB_CUDA(cudaMalloc(&v, count * sizeof(T)));
  m->allocs.push_back(v);
  *p = (T*)v;
  return STRICTB200_OK;
}
inline int fill_f32(strictb200_ctx* ctx, float* p, size_t n, float v) {
  std::vector<float> h(n, v);
  SB_CUDA(cudaMemcpyAsync(p, h.data(), n * 4, cudaMemcpyHostToDevice, ctx->stream));
  SB_CUDA(cudaStreamSynchronize(ctx->stream));
  return STRICTB200_OK;
}
inline int alloc_qw(strictb200_model* m, QW& w, int64_t N, int64_t K) {
  w.N = N; w.K = K;
  SB_TRY(dalloc(m, &w.q, (size_t)N * K));
  SB_TRY(dalloc(m, &w.s, (size_t)N));
  m->weight_bytes += (uint64_t)N * K + (uint64_t)N * 4;
  return STRICTB200_OK;
}
inline int alloc_fw(strictb200_model* m, FW& w, int64_t N, int64_t K) {
  w.N = N; w.K = K;
  SB_TRY(dalloc(m, &w.w, (size_t)N * K));
  SB_TRY(dalloc(m, &w.b, (size_t)N));
  SB_TRY(fill_f32(m->ctx, w.b, N, 0.f));
  m->weight_bytes += (uint64_t)N * K * 4 + (uint64_t)N * 4;
  return STRICTB200_OK;
}

inline size_t align256(size_t x) { return (x + 255) & ~(size_t)255; }

struct Carver {
  char* base;
  size_t off = 0;
  template <typename T>
  T* take(size_t count) {
    T* p = base ? (T*)(base + off) : nullptr;
    off += align256(count * sizeof(T));
    return p;
  }
};

// ------------------------------------------------------------------ per-class device timing
struct ProfSpan { int cls; cudaEvent_t a, b; };
struct SbProfiler {
  std::vector<ProfSpan> spans;
  std::vector<cudaEvent_t> pool;
  size_t used = 0;
  ProfSpan* open = nullptr;  // the span of the call that is being made
  cudaEvent_t get() {
    if (used == pool.size()) { cudaEvent_t e; cudaEventCreate(&e); pool.push_back(e); }
    return pool[used++];
  }
};
template <typename F>
inline int prof(strictb200_ctx* ctx, int cls, F&& f) {
  SbProfiler* p = ctx->prof;
  if (!p) return f();
  ProfSpan sp{cls, p->get(), p->get()};
  cudaEventRecord(sp.a, ctx->stream);
  p->open = &sp;
  int st = f();
  p->open = nullptr;
  cudaEventRecord(sp.b, ctx->stream);
  p->spans.push_back(sp);
  return st;
}
#define PROF(cls, expr) SB_TRY(prof(ctx, cls, [&]() -> int { return (expr); }))

// ------------------------------------------------------------------ prefill scratch
inline int prefill_scratch(strictb200_ctx* ctx, size_t bytes, char** out) {
  if (bytes > ctx->prefill_ws_bytes) {
    SB_CUDA(cudaStreamSynchronize(ctx->stream));
    if (ctx->prefill_ws) SB_CUDA(cudaFree(ctx->prefill_ws));
    ctx->prefill_ws = nullptr;
    ctx->prefill_ws_bytes = 0;
    SB_CUDA(cudaMalloc(&ctx->prefill_ws, bytes));
    ctx->prefill_ws_bytes = bytes;
  }
  *out = (char*)ctx->prefill_ws;
  return STRICTB200_OK;
}
struct ChunkIdx {
  int32_t *tok, *seq, *pos, *la, *past, *qs, *last;
};
inline void carve_idx(Carver& cv, int64_t T, int nb, int n_rows, ChunkIdx* o) {
  o->tok = cv.take<int32_t>(T); o->seq = cv.take<int32_t>(T); o->pos = cv.take<int32_t>(T);
  o->la = cv.take<int32_t>(nb); o->past = cv.take<int32_t>(nb); o->qs = cv.take<int32_t>(nb); o->last = cv.take<int32_t>(n_rows);
}

// ------------------------------------------------------------------ models described layer by layer (stack.cu)
struct PrefillChunk {  // the rows of one prefill chunk: nb sequences from b0 on, T token rows
  int64_t T = 0;
  int nb = 0, b0 = 0, max_new = 0;
  ChunkIdx ix;
  const int32_t *h_past = nullptr, *h_after = nullptr;  // host copies of the lengths before and after
  int n_rows = 0;                                       // rows of the output gather (ix.last): wanted rows, then the last row of every sequence
  int32_t* d_next = nullptr;
  float* h_logits = nullptr;                            // logits of the first n_logits gathered rows
  int n_logits = 0;
};
int sb_stack_init_random(strictb200_model* m, uint64_t seed);
int sb_stack_tensor(strictb200_model* m, const char* name, const void* h_in, void* h_out, size_t bytes);
void sb_stack_destroy(strictb200_model* m);
int sb_stack_kv_layout(strictb200_model* m, strictb200_kv* kv, size_t* elements, size_t* state_floats);  // layer offsets of the cache and of the states
bool sb_stack_plan(strictb200_model* m, strictb200_kv* kv, int longest);           // true: the decode step changed, record it again
size_t sb_stack_esz(strictb200_model* m);                                          // bytes of a weight or cache element
size_t sb_stack_decode_bytes(strictb200_model* m, strictb200_kv* kv);              // bytes of the decode buffers
int sb_stack_decode_body(strictb200_model* m, strictb200_kv* kv);
float* sb_stack_decode_logits(strictb200_model* m, strictb200_kv* kv);
size_t sb_stack_prefill_bytes(strictb200_model* m, const PrefillChunk& c);
int sb_stack_prefill_chunk(strictb200_model* m, strictb200_kv* kv, const PrefillChunk& c, char* scratch);
uint64_t sb_stack_cache_read_bytes(strictb200_model* m, int len);                  // cache bytes a decode step reads for one sequence of `len` keys
