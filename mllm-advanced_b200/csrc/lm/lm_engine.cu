// Host side of the bf16 language-model engine (include/mllmb200_lm.h): weights in the engine's layout, slots of
// per-sequence state, the step function and the decode graphs.
//
// A step is a ragged batch: rows (tokens) of several sequences, one after the other.  Linears and norms see rows;
// attention, retention and the convolution see sequences through row and entry tables in device memory.  A layer is
//   norm + conv | in-projection | mixer | out-projection | norm | gate-up | down
// where every norm also folds in the residual: x' = x + post_norm(sublayer), h = pre_norm(x'); or, with the norms behind
// the residual sum,
//   in-projection | mixer | out-projection | norm (+ choice of experts) | gate-up | down | norm.
#include <algorithm>
#include <cmath>
#include <cstdarg>
#include <cstdio>
#include <cstring>
#include <tuple>

#include "lm_state.h"

namespace mllmb200 {
__global__ void sample_advance_batched_kernel(const float2*, int, int*, int*, int*, int, const int*, int*);
cudaError_t read_device_status(cudaStream_t, int* status);

namespace lm {
namespace {

constexpr int kArgmaxBlocks = 32;

struct GraphKey {
  int count, chunk, splits;
  bool operator<(const GraphKey& o) const { return std::tie(count, chunk, splits) < std::tie(o.count, o.chunk, o.splits); }
};
// Sequences whose keys and values are made from latents together: their row tiles of the cache (per layer the same) and
// the attention tiles over the result.
struct ExpandPass {
  const int4* rows = nullptr;
  const int4* tiles = nullptr;
  int n_rows = 0, n_tiles = 0, total = 0;
};
// Positions per CTA of the decode attention: small pieces while they are needed to fill the GPU.
int decode_chunk(int sequences, int longest) {
  return (long long)sequences * ((longest + 127) / 128) >= 2 * kSms ? 128 : kMinDecodeChunk;
}
struct Graph {
  cudaGraphExec_t exec;
  long long launches;
};

// Device tables of a step.
struct StepCtx {
  int rows = 0, entries = 0;
  const int *tokens = nullptr, *row_entry = nullptr;
  const int2* row_sp = nullptr;
  const Entry* entry = nullptr;
  bool single = false;  // one token per entry, row r = entry r
  // mixed steps: rows of one-token entries, prompt tiles per head-group size, retention chunks
  const int* single_rows = nullptr;
  int n_single = 0, chunk = kMinDecodeChunk, splits = 1;  // context split of the decode attention
  std::map<int, std::pair<const int4*, int>> tiles;
  const int2 *chunks = nullptr, *entry_chunks = nullptr;
  int n_chunks = 0;
  // latent attention: rows that attend through the latent (nullptr: all), a bound of their contexts, and the others
  const int* latent_rows = nullptr;
  int n_latent = 0, latent_ctx = 1;
  std::vector<ExpandPass> expand;
};

struct Engine {
  mllmb200_lm_config c{};
  bool f32 = false, post = false, latent = false;
  bool absorb_all = false;  // all rows attend through the latent: 32-bit mode, heads too large for the prompt kernel
  int elt = 2, widthp = 0, plane_rows = 0, logit_rows = 0, max_splits_ctx = 1;
  std::vector<LayerState> layers;
  __nv_bfloat16* embed = nullptr;
  Linear head;
  float* final_gain = nullptr;
  unsigned loaded = 0;
  // activations
  float *xa = nullptr, *xb = nullptr, *delta = nullptr, *proj = nullptr, *logits = nullptr, *chunk_state = nullptr, *part_o = nullptr;
  float2 *part_ml = nullptr, *best = nullptr;
  // latent attention: rows before their norm, queries against the latent and outputs in it, keys and values of a step
  float *fresh = nullptr, *lat = nullptr, *lat_part = nullptr;
  float2* lat_ml = nullptr;
  void *qa = nullptr, *ex_k = nullptr, *ex_v = nullptr;
  int latent_cap = 0, expand_cap = 0;
  // experts
  float *route_logits = nullptr, *route_weight = nullptr;
  int *route_sel = nullptr, *route_rank = nullptr, *route_count = nullptr, *pair_row = nullptr, *n_moe_tiles = nullptr;
  int4* moe_tiles = nullptr;
  void* permuted = nullptr;
  ActMap m_permuted;
  int n_route_count = 0, route_planes = 1;
  void *h = nullptr, *mix = nullptr, *act = nullptr, *hf = nullptr;
  ActMap m_h, m_hf;
  // bookkeeping: the host's view of every slot, and the device's for decode graphs
  std::vector<int> pos, tail, ready;
  int *d_pos = nullptr, *d_tail = nullptr, *d_token = nullptr, *d_history = nullptr;
  int *d_slots = nullptr, *d_row_token = nullptr, *d_row_entry = nullptr, *d_identity = nullptr;
  int2* d_row_sp = nullptr;
  Entry* d_entries = nullptr;
  std::vector<int> cur_slots;
  std::vector<int> meta;
  int *meta_h = nullptr, *meta_d = nullptr;
  size_t meta_cap = 0;
  cudaEvent_t meta_free = nullptr;
  cudaStream_t stream = nullptr;
  std::map<GraphKey, Graph> graphs;
  std::vector<void*> owned;
  size_t state_bytes = 0;
  long long launches = 0;
  bool keep = false;
  float* kept = nullptr;
  int kept_rows = 0;
  std::string error;
};

int fail(Engine* e, int status, const char* fmt, ...) {
  char buf[512];
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(buf, sizeof(buf), fmt, ap);
  va_end(ap);
  e->error = buf;
  return status;
}
#define LM_CUDA(expr)                                                                                          \
  do {                                                                                                         \
    const cudaError_t r__ = (expr);                                                                            \
    if (r__ != cudaSuccess) return fail(e, MLLMB200_CUDA_ERROR, "%s: %s", #expr, cudaGetErrorString(r__));     \
  } while (0)
#define LM_OK(expr)                        \
  do {                                     \
    const int s__ = (expr);                \
    if (s__ != MLLMB200_OK) return s__;    \
  } while (0)

// Zeroed device memory owned by the engine.
template <class T>
int dalloc(Engine* e, T** p, size_t count, bool state = false) {
  const size_t bytes = std::max<size_t>(count, 1) * sizeof(T);
  void* q = nullptr;
  LM_CUDA(cudaMalloc(&q, bytes));
  e->owned.push_back(q);
  LM_CUDA(cudaMemsetAsync(q, 0, bytes, e->stream));
  if (state) e->state_bytes += bytes;
  *p = static_cast<T*>(q);
  return MLLMB200_OK;
}
int dalloc_bytes(Engine* e, void** p, size_t bytes, bool state = false) {
  uint8_t* q = nullptr;
  LM_OK(dalloc(e, &q, bytes, state));
  *p = q;
  return MLLMB200_OK;
}
int make_linear(Engine* e, Linear* l, int n, int k, int groups = 1) {
  l->n = n;
  l->k = pad_to(k, 64);
  l->groups = groups;
  LM_OK(dalloc(e, &l->w, (size_t)groups * n * l->k));
  if (make_linear_maps(l) != MLLMB200_OK) return fail(e, MLLMB200_CUDA_ERROR, "tensor map of a [%d, %d] weight", n, l->k);
  return MLLMB200_OK;
}

bool is_attn(const LayerState& L) { return L.d.mixer == MLLMB200_LM_ATTENTION; }
bool is_latent(const LayerState& L) { return L.d.mixer == MLLMB200_LM_LATENT; }
bool owns_latent(const LayerState& L) { return is_latent(L) && L.d.kv_from < 0; }
int qk_cols(const LayerState& L) { return L.d.heads * L.dimp; }
int mix_cols(const LayerState& L) { return L.d.heads * L.vdimp; }

// Exact: the largest m with (n / half)^rest >= (max / half)^m; a quotient of logarithms that lies on an integer up to
// rounding is that integer.
int bucket_of(int n, int rows, int max_distance) {
  const int half = rows / 2, rest = rows - half;
  if (n < half) return n;
  const long double x = logl((long double)n / half) / logl((long double)max_distance / half) * rest;
  const long double r = roundl(x);
  const int m = (int)(fabsl(x - r) < 1e-12L ? r : floorl(x));
  return std::min(rows - 1, half + m);
}

int check_latent(Engine* e, int i, const mllmb200_lm_layer& d) {
  if (d.kv_rank < 1) return fail(e, MLLMB200_INVALID_ARG, "layer %d: size of the latent", i);
  if (d.kv_rank > kMaxRank) return fail(e, MLLMB200_UNSUPPORTED, "layer %d: latents beyond %d", i, kMaxRank);
  if (d.kv_heads != d.heads) return fail(e, MLLMB200_UNSUPPORTED, "layer %d: latent attention has as many key as query heads", i);
  if (d.rot_dims || d.bias_rows || d.sink || d.weights_of >= 0)
    return fail(e, MLLMB200_UNSUPPORTED, "layer %d: rotation, distance bias, sink or shared weights in latent attention", i);
  if (e->c.max_rows > 65535) return fail(e, MLLMB200_UNSUPPORTED, "more than 65535 rows in a step of latent attention");
  if (d.kv_from < 0) return MLLMB200_OK;
  if (d.kv_from >= i || !owns_latent(e->layers[d.kv_from]) || e->layers[d.kv_from].d.kv_rank != d.kv_rank)
    return fail(e, MLLMB200_INVALID_ARG, "layer %d: layer %d has no cache of its own with latents of %d", i, d.kv_from, d.kv_rank);
  return MLLMB200_OK;
}

int check_layer(Engine* e, int i, const mllmb200_lm_layer& d) {
  if (d.mixer != MLLMB200_LM_ATTENTION && d.mixer != MLLMB200_LM_RETENTION && d.mixer != MLLMB200_LM_LATENT)
    return fail(e, MLLMB200_UNSUPPORTED, "layer %d: mixer %d", i, d.mixer);
  if (d.heads < 1 || d.kv_heads < 1 || d.heads % d.kv_heads || d.dim < 1 || d.vdim < 1 || d.ff < 0)
    return fail(e, MLLMB200_INVALID_ARG, "layer %d: sizes", i);
  const int most = d.mixer == MLLMB200_LM_LATENT ? kMaxRank : 256;
  if (d.dim > most || d.vdim > most || d.heads / d.kv_heads > 64) return fail(e, MLLMB200_UNSUPPORTED, "layer %d: head sizes beyond %d or more than 64 heads per key", i, most);
  if (d.act < MLLMB200_LM_ACT_CLAMPED || d.act > MLLMB200_LM_ACT_SILU) return fail(e, MLLMB200_UNSUPPORTED, "layer %d: activation %d", i, d.act);
  if (d.experts) {
    if (d.experts < 1 || d.top < 1 || d.top > d.experts || d.ff < 1) return fail(e, MLLMB200_INVALID_ARG, "layer %d: %d of %d experts", i, d.top, d.experts);
    if (d.experts > kMaxExperts || d.top > kMaxTop) return fail(e, MLLMB200_UNSUPPORTED, "layer %d: more than %d experts or %d at a time", i, kMaxExperts, kMaxTop);
  }
  if (d.mixer == MLLMB200_LM_LATENT) return check_latent(e, i, d);
  if (d.mixer == MLLMB200_LM_RETENTION) {
    if (d.kv_heads != d.heads) return fail(e, MLLMB200_UNSUPPORTED, "layer %d: retention has as many key as query heads", i);
    if (d.rot_dims < 0 || d.rot_dims % 2 || d.rot_dims > d.dim || (d.rot_dims && !(d.rot_base > 0))) return fail(e, MLLMB200_INVALID_ARG, "layer %d: rotation", i);
  } else {
    if (d.bias_rows < 0 || (d.bias_rows && (d.bias_rows < 2 || d.bias_max <= d.bias_rows / 2)))
      return fail(e, MLLMB200_INVALID_ARG, "layer %d: distance bias needs at least two rows and a largest distance beyond half of them", i);
    if (d.rot_dims) return fail(e, MLLMB200_UNSUPPORTED, "layer %d: rotation in attention", i);
  }
  if (d.weights_of >= 0) {
    if (d.weights_of >= i) return fail(e, MLLMB200_INVALID_ARG, "layer %d: weights of a later layer", i);
    const mllmb200_lm_layer &o = e->layers[d.weights_of].d, &m = d;
    if (o.mixer != m.mixer || o.heads != m.heads || o.kv_heads != m.kv_heads || o.dim != m.dim || o.vdim != m.vdim || o.ff != m.ff ||
        o.bias_rows != m.bias_rows || o.bias_max != m.bias_max || o.experts != m.experts)
      return fail(e, MLLMB200_INVALID_ARG, "layer %d differs from layer %d, whose weights it uses", i, d.weights_of);
  }
  return MLLMB200_OK;
}

int create(Engine* e, const mllmb200_lm_layer* descs) {
  const auto& c = e->c;
  if (c.vocab < 1 || c.width < 1 || c.layers < 1 || c.conv_taps < 0 || c.max_seqs < 1 || c.max_ctx < 1 || c.max_rows < 1 ||
      (c.dtype != MLLMB200_LM_BF16 && c.dtype != MLLMB200_LM_F32) ||
      (c.norm_place != MLLMB200_LM_NORM_SANDWICH && c.norm_place != MLLMB200_LM_NORM_POST))
    return fail(e, MLLMB200_INVALID_ARG, "model sizes");
  e->post = c.norm_place == MLLMB200_LM_NORM_POST;
  if (e->post && c.conv_taps) return fail(e, MLLMB200_UNSUPPORTED, "an input convolution with norms behind the residual sum");
  e->f32 = c.dtype == MLLMB200_LM_F32;
  e->elt = e->f32 ? 4 : 2;
  e->widthp = pad_to(c.width, 64);
  if (e->widthp > 8192 || (size_t)c.conv_taps * e->widthp * 4 > 200 * 1024) return fail(e, MLLMB200_UNSUPPORTED, "width %d with %d taps", c.width, c.conv_taps);
  LM_CUDA(cudaStreamCreateWithFlags(&e->stream, cudaStreamNonBlocking));
  LM_CUDA(cudaEventCreateWithFlags(&e->meta_free, cudaEventDisableTiming));
  LM_CUDA(linear_configure());
  LM_CUDA(attention_configure());
  LM_CUDA(retention_configure());
  LM_CUDA(latent_configure());
  const size_t rows = c.max_rows, slots = c.max_seqs;
  e->plane_rows = std::max(c.max_rows, 1024);
  e->logit_rows = std::max(std::min(c.max_rows, 128), c.max_seqs);
  e->max_splits_ctx = (c.max_ctx + kMinDecodeChunk - 1) / kMinDecodeChunk;
  LM_OK(dalloc(e, &e->embed, (size_t)c.vocab * c.width));
  LM_OK(make_linear(e, &e->head, c.vocab, c.width));
  LM_OK(dalloc(e, &e->final_gain, e->post ? e->widthp : 1));
  std::map<std::pair<int, double>, std::pair<float*, float*>> ropes;
  size_t proj_bytes = 0, mix_elems = 0, act_elems = 0, part = 0, heads = 0, chunk_elems = 0;
  size_t rank = 0, head_rank = 0, lat_heads = 0, ex_k = 0, ex_v = 0, experts = 0, top = 0;
  e->layers.resize(c.layers);
  for (int i = 0; i < c.layers; ++i) {
    LayerState& L = e->layers[i];
    LM_OK(check_layer(e, i, descs[i]));
    L.d = descs[i];
    L.src = L.d.weights_of < 0 ? i : e->layers[L.d.weights_of].src;
    L.dimp = pad_to(L.d.dim, 16);
    L.vdimp = pad_to(L.d.vdim, 16);
    L.rankp = is_latent(L) ? pad_to(L.d.kv_rank, 64) : 0;
    const int G = L.d.kv_heads;
    if (L.src == i) {
      const int n_in = is_attn(L)     ? qk_cols(L) + G * (L.dimp + L.vdimp)
                       : is_latent(L) ? qk_cols(L) + (owns_latent(L) ? L.rankp : 0)
                                      : 2 * (qk_cols(L) + mix_cols(L));
      LM_OK(make_linear(e, &L.w.in, n_in, c.width));
      LM_OK(make_linear(e, &L.w.out, c.width, mix_cols(L)));
      if (L.d.ff) {
        LM_OK(make_linear(e, &L.w.gate_up, 2 * L.d.ff, c.width, std::max(1, L.d.experts)));
        LM_OK(make_linear(e, &L.w.down, c.width, L.d.ff, std::max(1, L.d.experts)));
      }
      if (L.d.experts) {
        LM_OK(make_linear(e, &L.w.router, L.d.experts, c.width));
        LM_OK(dalloc(e, &L.w.router_b, L.d.experts));
        L.w.expert_loaded.assign(L.d.experts, 0);
      }
      if (is_latent(L)) {
        LM_OK(make_linear(e, &L.w.uk_uv, qk_cols(L) + mix_cols(L), L.d.kv_rank));
        LM_OK(dalloc(e, &L.w.uk_t, (size_t)L.d.heads * L.rankp * L.dimp));
        if (owns_latent(L)) LM_OK(dalloc(e, &L.w.kv_gain, L.rankp));
      }
      LM_OK(dalloc(e, &L.w.norms, e->post ? 2 * (size_t)e->widthp : 4));
      if (c.conv_taps) LM_OK(dalloc(e, &L.w.conv, (size_t)c.conv_taps * e->widthp));
      if (is_attn(L) && L.d.bias_rows) LM_OK(dalloc(e, &L.w.bias, (size_t)L.d.heads * (L.d.bias_max + 1)));
      if (L.d.mixer == MLLMB200_LM_RETENTION) LM_OK(dalloc(e, &L.w.decay, (size_t)L.d.heads * (kChunk + 1)));
    }
    if (is_attn(L)) {
      LM_OK(dalloc_bytes(e, &L.kc, slots * G * c.max_ctx * L.dimp * e->elt, true));
      LM_OK(dalloc_bytes(e, &L.vc, slots * G * c.max_ctx * L.vdimp * e->elt, true));
      proj_bytes = std::max(proj_bytes, rows * qk_cols(L) * e->elt);
      part = std::max(part, (size_t)mix_cols(L));
      heads = std::max(heads, (size_t)L.d.heads);
    } else if (is_latent(L)) {
      e->latent = true;
      e->absorb_all = e->absorb_all || e->f32 || L.d.dim > 256 || L.d.vdim > 256;
      if (owns_latent(L)) {
        LM_OK(dalloc_bytes(e, &L.kc, slots * c.max_ctx * L.rankp * e->elt, true));
        if (make_act_map(&L.a_kc, L.kc, (int)(slots * c.max_ctx), L.rankp) != MLLMB200_OK) return fail(e, MLLMB200_CUDA_ERROR, "tensor map of a latent cache");
      } else {
        L.kc = e->layers[L.d.kv_from].kc;
        L.a_kc = e->layers[L.d.kv_from].a_kc;
      }
      proj_bytes = std::max(proj_bytes, rows * qk_cols(L) * e->elt);
      rank = std::max(rank, (size_t)L.rankp);
      head_rank = std::max(head_rank, (size_t)L.d.heads * L.rankp);
      lat_heads = std::max(lat_heads, (size_t)L.d.heads);
      ex_k = std::max(ex_k, (size_t)qk_cols(L));
      ex_v = std::max(ex_v, (size_t)mix_cols(L));
    } else {
      LM_OK(dalloc(e, &L.state, slots * L.d.heads * L.dimp * L.vdimp, true));
      proj_bytes = std::max(proj_bytes, rows * 2 * (size_t)(qk_cols(L) + mix_cols(L)) * 4);
      chunk_elems = std::max(chunk_elems, (size_t)L.d.heads * L.dimp * L.vdimp);
      if (L.d.rot_dims) {
        auto& r = ropes[{L.d.rot_dims, L.d.rot_base}];
        if (!r.first) {
          const size_t n = (size_t)c.max_ctx * (L.d.rot_dims / 2);
          LM_OK(dalloc(e, &r.first, n));
          LM_OK(dalloc(e, &r.second, n));
          LM_CUDA(launch_rope_table(e->stream, r.first, r.second, c.max_ctx, L.d.rot_dims, L.d.rot_base));
        }
        L.cos_t = r.first;
        L.sin_t = r.second;
      }
    }
    if (c.conv_taps > 1) LM_OK(dalloc(e, &L.tail, slots * 2 * (c.conv_taps - 1) * e->widthp, true));
    mix_elems = std::max(mix_elems, rows * (size_t)pad_to(mix_cols(L), 64));
    if (L.d.ff) act_elems = std::max(act_elems, rows * (L.d.experts ? L.d.top : 1) * (size_t)pad_to(L.d.ff, 64));
    experts = std::max(experts, (size_t)L.d.experts);
    top = std::max(top, (size_t)L.d.top * (L.d.experts ? 1 : 0));
  }
  e->plane_rows = std::max(e->plane_rows, (int)(rows * top));
  if (e->latent) {
    e->latent_cap = e->absorb_all ? c.max_rows : std::min(c.max_rows, c.max_seqs * kAbsorbMax);
    LM_OK(dalloc(e, &e->fresh, rows * rank));
    LM_OK(dalloc_bytes(e, &e->qa, e->latent_cap * head_rank * e->elt));
    if (e->f32) {
      LM_OK(dalloc(e, &e->lat, rows * head_rank));
    } else {
      LM_OK(dalloc(e, &e->lat_part, latent_parts(e->latent_cap) * head_rank));
      LM_OK(dalloc(e, &e->lat_ml, latent_parts(e->latent_cap) * lat_heads));
      if (!e->absorb_all) {
        e->expand_cap = c.max_ctx + (c.max_seqs > 1 ? c.max_rows : 0);
        LM_OK(dalloc_bytes(e, &e->ex_k, e->expand_cap * ex_k * e->elt));
        LM_OK(dalloc_bytes(e, &e->ex_v, e->expand_cap * ex_v * e->elt));
      }
    }
  }
  if (experts) {
    const size_t pairs = rows * top;
    e->n_route_count = (int)(c.layers * experts);
    e->route_planes = kMaxSplits;
    LM_OK(dalloc(e, &e->route_logits, rows * pad_to((int)experts, 4) * e->route_planes));
    LM_OK(dalloc(e, &e->route_weight, pairs));
    LM_OK(dalloc(e, &e->route_sel, pairs));
    LM_OK(dalloc(e, &e->route_rank, pairs));
    LM_OK(dalloc(e, &e->pair_row, pairs));
    LM_OK(dalloc(e, &e->route_count, e->n_route_count));
    LM_OK(dalloc(e, &e->n_moe_tiles, 1));
    LM_OK(dalloc(e, &e->moe_tiles, experts + pairs / group_tile_rows(e->f32) + 1));
    LM_OK(dalloc_bytes(e, &e->permuted, pairs * e->widthp * e->elt));
    if (make_act_map(&e->m_permuted, e->permuted, (int)pairs, e->widthp) != MLLMB200_OK) return fail(e, MLLMB200_CUDA_ERROR, "tensor map of the activations");
  }
  LM_OK(dalloc(e, &e->xa, rows * e->widthp));
  LM_OK(dalloc(e, &e->xb, rows * e->widthp));
  LM_OK(dalloc(e, &e->delta, (size_t)e->plane_rows * e->widthp));
  LM_OK(dalloc_bytes(e, &e->h, rows * e->widthp * e->elt));
  LM_OK(dalloc_bytes(e, &e->mix, mix_elems * e->elt));
  LM_OK(dalloc_bytes(e, &e->act, act_elems * e->elt));
  LM_OK(dalloc_bytes(e, &e->hf, (size_t)e->logit_rows * e->widthp * e->elt));
  LM_OK(dalloc_bytes(e, reinterpret_cast<void**>(&e->proj), proj_bytes));
  LM_OK(dalloc(e, &e->logits, (size_t)e->logit_rows * c.vocab));
  LM_OK(dalloc(e, &e->best, (size_t)e->logit_rows * kArgmaxBlocks));
  LM_OK(dalloc(e, &e->chunk_state, ((rows + kChunk - 1) / kChunk + slots) * chunk_elems));
  if (e->max_splits_ctx > 1) {
    LM_OK(dalloc(e, &e->part_o, slots * part * e->max_splits_ctx));
    LM_OK(dalloc(e, &e->part_ml, slots * heads * e->max_splits_ctx));
  }
  if (make_act_map(&e->m_h, e->h, c.max_rows, e->widthp) != MLLMB200_OK || make_act_map(&e->m_hf, e->hf, e->logit_rows, e->widthp) != MLLMB200_OK)
    return fail(e, MLLMB200_CUDA_ERROR, "tensor map of the activations");
  for (auto& L : e->layers) {
    bool ok = make_act_map(&L.a_mix, e->mix, c.max_rows, pad_to(mix_cols(L), 64)) == MLLMB200_OK;
    if (L.d.ff) ok = ok && make_act_map(&L.a_act, e->act, c.max_rows * (L.d.experts ? L.d.top : 1), pad_to(L.d.ff, 64)) == MLLMB200_OK;
    if (!ok) return fail(e, MLLMB200_CUDA_ERROR, "tensor map of the activations");
  }
  LM_OK(dalloc(e, &e->d_pos, slots));
  LM_OK(dalloc(e, &e->d_tail, slots));
  LM_OK(dalloc(e, &e->d_token, slots));
  LM_OK(dalloc(e, &e->d_history, slots * c.max_ctx));
  LM_OK(dalloc(e, &e->d_slots, slots));
  LM_OK(dalloc(e, &e->d_row_token, slots));
  LM_OK(dalloc(e, &e->d_row_entry, slots));
  LM_OK(dalloc(e, &e->d_row_sp, slots));
  LM_OK(dalloc(e, &e->d_entries, slots));
  LM_OK(dalloc(e, &e->d_identity, std::max(slots, (size_t)1)));
  std::vector<int> id(slots);
  for (size_t i = 0; i < slots; ++i) id[i] = (int)i;
  LM_CUDA(cudaMemcpyAsync(e->d_identity, id.data(), slots * 4, cudaMemcpyHostToDevice, e->stream));
  LM_CUDA(cudaStreamSynchronize(e->stream));
  e->pos.assign(slots, 0);
  e->tail.assign(slots, 0);
  e->ready.assign(slots, 0);
  return MLLMB200_OK;
}

// ------------------------------------------------------------------------------------------ weights
struct PackSpec {
  Linear* to;
  int rows, cols, row_block, row_pad, row_mul, row_off, col_block, col_pad;
};

int pack(Engine* e, const PackSpec& p, const void* data) {
  __nv_bfloat16* staged = nullptr;
  const size_t bytes = (size_t)p.rows * p.cols * 2;
  LM_CUDA(cudaMalloc(reinterpret_cast<void**>(&staged), bytes));
  cudaError_t r = cudaMemcpyAsync(staged, data, bytes, cudaMemcpyDefault, e->stream);
  if (r == cudaSuccess)
    r = launch_pack_rows(e->stream, staged, p.rows, p.cols, p.to->w, p.to->k, p.row_block, p.row_pad, p.row_mul, p.row_off, p.col_block, p.col_pad);
  if (r == cudaSuccess) r = cudaStreamSynchronize(e->stream);
  cudaFree(staged);
  LM_CUDA(r);
  return MLLMB200_OK;
}
template <class T>
int to_host(Engine* e, std::vector<T>* v, const void* data, size_t n) {
  v->resize(n);
  LM_CUDA(cudaMemcpyAsync(v->data(), data, n * sizeof(T), cudaMemcpyDefault, e->stream));
  LM_CUDA(cudaStreamSynchronize(e->stream));
  return MLLMB200_OK;
}
template <class T>
int to_device(Engine* e, T* dst, const std::vector<T>& v) {
  LM_CUDA(cudaMemcpyAsync(dst, v.data(), v.size() * sizeof(T), cudaMemcpyHostToDevice, e->stream));
  LM_CUDA(cudaStreamSynchronize(e->stream));
  return MLLMB200_OK;
}

// A tensor's rows to one group of a linear, row r to r row_mul + row_off.
int pack_group(Engine* e, const Linear& l, int group, int row_mul, int row_off, const void* data, int rows, int cols) {
  Linear g = l;
  g.w = l.w + (size_t)group * l.n * l.k;
  return pack(e, {&g, rows, cols, rows, rows, row_mul, row_off, cols, cols}, data);
}
int set_vector(Engine* e, float* dst, const void* data, int n) {
  LM_CUDA(cudaMemcpy(dst, data, (size_t)n * 4, cudaMemcpyDefault));
  return MLLMB200_OK;
}

int set_expert(Engine* e, int layer, int expert, int which, const void* data, int rows, int cols) {
  if (layer < 0 || layer >= e->c.layers || e->layers[layer].src != layer || expert < 0 || expert >= e->layers[layer].d.experts)
    return fail(e, MLLMB200_INVALID_ARG, "expert %d of layer %d", expert, layer);
  LayerState& L = e->layers[layer];
  const bool down = which == MLLMB200_LM_T_DOWN;
  const int n = down ? e->c.width : L.d.ff, k = down ? L.d.ff : e->c.width;
  if ((!down && which != MLLMB200_LM_T_GATE && which != MLLMB200_LM_T_UP) || rows != n || cols != k)
    return fail(e, MLLMB200_INVALID_ARG, "tensor %d of expert %d of layer %d is [%d, %d], expected [%d, %d]", which, expert, layer, rows, cols, n, k);
  if (down) LM_OK(pack_group(e, L.w.down, expert, 1, 0, data, rows, cols));
  else LM_OK(pack_group(e, L.w.gate_up, expert, 2, which == MLLMB200_LM_T_UP, data, rows, cols));
  L.w.expert_loaded[expert] |= 1u << which;
  return MLLMB200_OK;
}

int set_tensor(Engine* e, int layer, int which, const void* data, int rows, int cols) {
  const auto& c = e->c;
  auto shape = [&](int r, int k) {
    return rows == r && cols == k ? MLLMB200_OK
                                  : fail(e, MLLMB200_INVALID_ARG, "tensor %d of layer %d is [%d, %d], expected [%d, %d]", which, layer, rows, cols, r, k);
  };
  if (layer == -1) {
    if (which == MLLMB200_LM_T_EMBED) {
      LM_OK(shape(c.vocab, c.width));
      LM_CUDA(cudaMemcpy(e->embed, data, (size_t)rows * cols * 2, cudaMemcpyDefault));
    } else if (which == MLLMB200_LM_T_HEAD) {
      LM_OK(shape(c.vocab, c.width));
      LM_OK(pack(e, {&e->head, rows, cols, rows, rows, 1, 0, cols, cols}, data));
    } else if (which == MLLMB200_LM_T_FINAL_NORM) {
      LM_OK(shape(1, e->post ? c.width : 1));
      LM_OK(set_vector(e, e->final_gain, data, cols));
    } else {
      return fail(e, MLLMB200_INVALID_ARG, "tensor %d", which);
    }
    e->loaded |= 1u << (which - MLLMB200_LM_T_EMBED);
    return MLLMB200_OK;
  }
  if (layer < 0 || layer >= c.layers || e->layers[layer].src != layer || which < 0 || which >= MLLMB200_LM_T_COUNT)
    return fail(e, MLLMB200_INVALID_ARG, "tensor %d of layer %d", which, layer);
  LayerState& L = e->layers[layer];
  const auto& d = L.d;
  const int H = d.heads, G = d.kv_heads, k_off = qk_cols(L), v_off = k_off + G * L.dimp, g_off = v_off + G * L.vdimp;
  switch (which) {
    case MLLMB200_LM_T_Q:
      LM_OK(shape(H * d.dim, c.width));
      LM_OK(pack(e, {&L.w.in, rows, cols, d.dim, L.dimp, 1, 0, cols, cols}, data));
      break;
    case MLLMB200_LM_T_DKV:
      if (!owns_latent(L)) return fail(e, MLLMB200_INVALID_ARG, "layer %d makes no latents", layer);
      LM_OK(shape(d.kv_rank, c.width));
      LM_OK(pack(e, {&L.w.in, rows, cols, rows, rows, 1, qk_cols(L), cols, cols}, data));
      break;
    case MLLMB200_LM_T_DKV_NORM:
      if (!owns_latent(L)) return fail(e, MLLMB200_INVALID_ARG, "layer %d makes no latents", layer);
      LM_OK(shape(1, d.kv_rank));
      LM_OK(set_vector(e, L.w.kv_gain, data, cols));
      break;
    case MLLMB200_LM_T_UK: {
      if (!is_latent(L)) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no latent attention", layer);
      LM_OK(shape(H * d.dim, d.kv_rank));
      LM_OK(pack(e, {&L.w.uk_uv, rows, cols, d.dim, L.dimp, 1, 0, cols, cols}, data));
      std::vector<uint16_t> src;
      LM_OK(to_host(e, &src, data, (size_t)rows * cols));
      __nv_bfloat16* staged = nullptr;
      LM_CUDA(cudaMalloc(reinterpret_cast<void**>(&staged), src.size() * 2));
      cudaError_t r = cudaMemcpyAsync(staged, src.data(), src.size() * 2, cudaMemcpyHostToDevice, e->stream);
      if (r == cudaSuccess) r = launch_pack_heads_transposed(e->stream, staged, H, d.dim, d.kv_rank, L.w.uk_t, L.rankp, L.dimp);
      if (r == cudaSuccess) r = cudaStreamSynchronize(e->stream);
      cudaFree(staged);
      LM_CUDA(r);
      break;
    }
    case MLLMB200_LM_T_UV:
      if (!is_latent(L)) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no latent attention", layer);
      LM_OK(shape(H * d.vdim, d.kv_rank));
      LM_OK(pack(e, {&L.w.uk_uv, rows, cols, d.vdim, L.vdimp, 1, qk_cols(L), cols, cols}, data));
      break;
    case MLLMB200_LM_T_ROUTER:
      if (!d.experts) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no experts", layer);
      LM_OK(shape(d.experts, c.width));
      LM_OK(pack(e, {&L.w.router, rows, cols, rows, rows, 1, 0, cols, cols}, data));
      break;
    case MLLMB200_LM_T_ROUTER_B:
      if (!d.experts) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no experts", layer);
      LM_OK(shape(1, d.experts));
      LM_OK(set_vector(e, L.w.router_b, data, cols));
      break;
    case MLLMB200_LM_T_K:
      if (is_latent(L)) return fail(e, MLLMB200_INVALID_ARG, "layer %d makes its keys from latents", layer);
      LM_OK(shape(G * d.dim, c.width));
      LM_OK(pack(e, {&L.w.in, rows, cols, d.dim, L.dimp, 1, k_off, cols, cols}, data));
      break;
    case MLLMB200_LM_T_V:
      if (is_latent(L)) return fail(e, MLLMB200_INVALID_ARG, "layer %d makes its values from latents", layer);
      LM_OK(shape(G * d.vdim, c.width));
      LM_OK(pack(e, {&L.w.in, rows, cols, d.vdim, L.vdimp, 1, v_off, cols, cols}, data));
      break;
    case MLLMB200_LM_T_G:
      if (!L.w.decay) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no output gate", layer);
      LM_OK(shape(H * d.vdim, c.width));
      LM_OK(pack(e, {&L.w.in, rows, cols, d.vdim, L.vdimp, 1, g_off, cols, cols}, data));
      break;
    case MLLMB200_LM_T_O:
      LM_OK(shape(c.width, H * d.vdim));
      LM_OK(pack(e, {&L.w.out, rows, cols, rows, rows, 1, 0, d.vdim, L.vdimp}, data));
      break;
    case MLLMB200_LM_T_GATE:
    case MLLMB200_LM_T_UP:
      if (!d.ff || d.experts) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no dense feed-forward", layer);
      LM_OK(shape(d.ff, c.width));
      LM_OK(pack(e, {&L.w.gate_up, rows, cols, rows, rows, 2, which == MLLMB200_LM_T_UP, cols, cols}, data));
      break;
    case MLLMB200_LM_T_DOWN:
      if (!d.ff || d.experts) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no dense feed-forward", layer);
      LM_OK(shape(c.width, d.ff));
      LM_OK(pack(e, {&L.w.down, rows, cols, rows, rows, 1, 0, cols, cols}, data));
      break;
    case MLLMB200_LM_T_NORM1:
    case MLLMB200_LM_T_NORM1B:
    case MLLMB200_LM_T_NORM2:
    case MLLMB200_LM_T_NORM2B:
      if (e->post) {
        if (which != MLLMB200_LM_T_NORM1 && which != MLLMB200_LM_T_NORM2) return fail(e, MLLMB200_INVALID_ARG, "tensor %d: one norm per sublayer", which);
        LM_OK(shape(1, c.width));
        LM_OK(set_vector(e, L.w.norms + (which == MLLMB200_LM_T_NORM2 ? e->widthp : 0), data, cols));
      } else {
        LM_OK(shape(1, 1));
        LM_OK(set_vector(e, L.w.norms + (which - MLLMB200_LM_T_NORM1), data, 1));
      }
      break;
    case MLLMB200_LM_T_CONV: {
      LM_OK(shape(c.width, c.conv_taps));
      std::vector<float> src, t((size_t)c.conv_taps * e->widthp, 0.0f);
      LM_OK(to_host(e, &src, data, (size_t)rows * cols));
      for (int w = 0; w < rows; ++w)
        for (int j = 0; j < cols; ++j) t[(size_t)j * e->widthp + w] = src[(size_t)w * cols + j];
      LM_OK(to_device(e, L.w.conv, t));
      break;
    }
    case MLLMB200_LM_T_REL: {
      if (!L.w.bias) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no distance bias", layer);
      LM_OK(shape(d.bias_rows, H));
      std::vector<float> src, t((size_t)H * (d.bias_max + 1));
      LM_OK(to_host(e, &src, data, (size_t)rows * cols));
      for (int n = 0; n <= d.bias_max; ++n) {
        const int b = bucket_of(n, d.bias_rows, d.bias_max);
        for (int h = 0; h < H; ++h) t[(size_t)h * (d.bias_max + 1) + n] = src[(size_t)b * H + h];
      }
      LM_OK(to_device(e, L.w.bias, t));
      break;
    }
    case MLLMB200_LM_T_DECAY: {
      if (!L.w.decay) return fail(e, MLLMB200_INVALID_ARG, "layer %d has no decays", layer);
      LM_OK(shape(1, H));
      std::vector<double> src;
      LM_OK(to_host(e, &src, data, H));
      std::vector<float> t((size_t)H * (kChunk + 1));
      for (int h = 0; h < H; ++h)
        for (int n = 0; n <= kChunk; ++n) t[(size_t)h * (kChunk + 1) + n] = (float)std::pow(src[h], (double)n);
      LM_OK(to_device(e, L.w.decay, t));
      break;
    }
  }
  L.w.loaded |= 1u << which;
  return MLLMB200_OK;
}

int check_loaded(Engine* e) {
  if (e->loaded != 7u) return fail(e, MLLMB200_INVALID_ARG, "embedding, head or final norm not loaded");
  for (int i = 0; i < e->c.layers; ++i) {
    const LayerState& L = e->layers[i];
    if (L.src != i) continue;
    auto bit = [](int w) { return 1u << w; };
    const unsigned mlp = bit(MLLMB200_LM_T_GATE) | bit(MLLMB200_LM_T_UP) | bit(MLLMB200_LM_T_DOWN);
    unsigned need = bit(MLLMB200_LM_T_Q) | bit(MLLMB200_LM_T_O) | bit(MLLMB200_LM_T_NORM1);
    need |= is_latent(L) ? bit(MLLMB200_LM_T_UK) | bit(MLLMB200_LM_T_UV) : bit(MLLMB200_LM_T_K) | bit(MLLMB200_LM_T_V);
    if (owns_latent(L)) need |= bit(MLLMB200_LM_T_DKV) | bit(MLLMB200_LM_T_DKV_NORM);
    if (!e->post) need |= bit(MLLMB200_LM_T_NORM1B);
    if (L.d.ff) need |= bit(MLLMB200_LM_T_NORM2) | (e->post ? 0 : bit(MLLMB200_LM_T_NORM2B));
    if (L.d.experts) {
      need |= bit(MLLMB200_LM_T_ROUTER) | bit(MLLMB200_LM_T_ROUTER_B);
      for (int x = 0; x < L.d.experts; ++x)
        if (L.w.expert_loaded[x] != mlp) return fail(e, MLLMB200_INVALID_ARG, "layer %d: tensors of expert %d missing", i, x);
    } else if (L.d.ff) {
      need |= mlp;
    }
    if (e->c.conv_taps) need |= bit(MLLMB200_LM_T_CONV);
    if (L.w.bias) need |= bit(MLLMB200_LM_T_REL);
    if (L.w.decay) need |= bit(MLLMB200_LM_T_G) | bit(MLLMB200_LM_T_DECAY);
    if ((L.w.loaded & need) != need) return fail(e, MLLMB200_INVALID_ARG, "layer %d: tensors missing (have %x, need %x)", i, L.w.loaded, need);
  }
  return MLLMB200_OK;
}

// ------------------------------------------------------------------------------------------ forward
// The residual stream between sublayers: x, and the sublayer output that the next norm folds in.
struct Stream {
  float *x, *other;
  Delta delta{};              // p = nullptr: nothing to fold in
  const float* gain = nullptr;
};

NormArgs norm_args(Engine* e, const StepCtx& t, const Stream& r, const float* g_pre, void* out) {
  NormArgs a{};
  a.x_in = r.x;
  a.delta = r.delta;
  a.g_post = r.gain;
  a.g_pre = g_pre;
  a.eps = e->c.eps;
  a.width = e->c.width;
  a.ldx = e->widthp;
  a.out = out;
  a.rows = t.rows;
  a.entries = t.entry;
  a.row_entry = t.row_entry;
  a.rows_per_cta = 1;
  return a;
}

int fold_norm(Engine* e, const StepCtx& t, Stream* r, const float* g_pre, LayerState* conv_layer) {
  NormArgs a = norm_args(e, t, *r, g_pre, e->h);
  if (r->delta.p) a.x_out = r->other;
  if (conv_layer && e->c.conv_taps) {
    a.taps = e->c.conv_taps;
    a.conv_w = e->layers[conv_layer->src].w.conv;
    a.tail = conv_layer->tail;
    // the rows in front of a CTA's first one are recomputed: longer runs once there are enough of them
    if (!t.single) a.rows_per_cta = std::max(1, std::min(16, t.rows / (2 * kSms)));
  }
  LM_CUDA(launch_norm(e->stream, e->f32, a));
  if (r->delta.p) std::swap(r->x, r->other);
  r->delta = Delta{};
  return MLLMB200_OK;
}

int linear_failed(Engine* e) { return fail(e, MLLMB200_CUDA_ERROR, "linear launch: %s", cudaGetErrorString(cudaGetLastError())); }

RouterArgs router_args(Engine* e, int layer, bool gemv) {
  const LayerState& L = e->layers[layer];
  const Weights& w = e->layers[L.src].w;
  RouterArgs a{};
  a.w = w.router.w;
  a.b = w.router_b;
  a.experts = L.d.experts;
  a.top = L.d.top;
  a.ldw = w.router.k;
  a.sel = e->route_sel;
  a.weight = e->route_weight;
  a.count = e->route_count + (size_t)layer * (e->n_route_count / e->c.layers);
  a.rank = gemv ? nullptr : e->route_rank;
  return a;
}

// x = norm(residual_scale x + sublayer), in place, and h; router: the experts of a mixture behind this norm, if it takes them.
int post_norm(Engine* e, const StepCtx& t, Stream* r, const float* gain, const RouterArgs* router) {
  PostNormArgs a{};
  a.x_in = a.x_out = r->x;
  a.delta = r->delta;
  a.alpha = e->c.residual_scale;
  a.gain = gain;
  a.eps = e->c.eps;
  a.width = e->c.width;
  a.ldx = e->widthp;
  a.rows = t.rows;
  a.out = e->h;
  if (router) a.router = *router;
  LM_CUDA(launch_post_norm(e->stream, e->f32, a));
  r->delta = Delta{};
  return MLLMB200_OK;
}

// A linear whose result the next norm folds in.
int delta_linear(Engine* e, const StepCtx& t, const Linear& w, const ActMap& m, const void* x, const float* gain, Stream* r) {
  Epi p{};
  p.kind = kEpiPlanes;
  p.y = e->delta;
  p.plane = (size_t)t.rows * e->widthp;
  p.ldy = e->widthp;
  p.scale = 1.0f;
  const int planes = launch_linear(e->stream, e->f32, w, m, x, t.rows, p, std::max(1, std::min(kMaxSplits, e->plane_rows / t.rows)));
  if (planes < 1) return linear_failed(e);
  r->delta = Delta{e->delta, planes, e->widthp, p.plane, nullptr, nullptr, 1};
  r->gain = gain;
  return MLLMB200_OK;
}

Epi gate_epi(Engine* e, const LayerState& L, const Weights& w) {
  Epi p{};
  p.kind = kEpiGate;
  p.act = e->act;
  p.ld_act = w.down.k;
  p.act_kind = L.d.act;
  p.limit = L.d.ff_limit;
  return p;
}

// A mixture of experts on e->h; `routed`: the norm before has chosen the experts.
int moe(Engine* e, const StepCtx& t, int layer, bool routed, const float* gain, Stream* r) {
  const LayerState& L = e->layers[layer];
  const Weights& w = e->layers[L.src].w;
  const int pairs = t.rows * L.d.top;
  const bool gemv = t.rows <= kGemvRows;
  const RouterArgs ra = router_args(e, layer, gemv);
  if (!routed) {
    Epi p{};
    p.kind = kEpiPlanes;
    p.y = e->route_logits;
    p.ldy = pad_to(L.d.experts, 4);
    p.plane = (size_t)t.rows * p.ldy;
    p.scale = 1.0f;
    const int planes = launch_linear(e->stream, e->f32, w.router, e->m_h, e->h, t.rows, p, e->route_planes);
    if (planes < 1) return linear_failed(e);
    LM_CUDA(launch_topk(e->stream, ra, e->route_logits, p.ldy, planes, p.plane, t.rows));
  }
  Groups g;
  g.rows = pairs;
  const void* x = e->h;
  if (gemv) {
    g.group_of = e->route_sel;
    g.div = L.d.top;
  } else {
    LM_CUDA(launch_moe_permute(e->stream, e->f32, ra, e->h, e->widthp, t.rows, e->permuted, e->pair_row, e->moe_tiles, e->n_moe_tiles));
    const int tile = group_tile_rows(e->f32), active = std::min(L.d.experts, pairs);
    g.tiles = e->moe_tiles;
    g.n_tiles = e->n_moe_tiles;
    g.max_tiles = active + pairs / tile;
    g.likely_tiles = active * ((pairs / active + tile - 1) / tile);
    x = e->permuted;
  }
  if (launch_linear_groups(e->stream, e->f32, w.gate_up, e->m_permuted, x, g, gate_epi(e, L, w), 1) < 1) return linear_failed(e);
  g.div = 1;
  Epi p{};
  p.kind = kEpiPlanes;
  p.y = e->delta;
  p.plane = (size_t)pairs * e->widthp;
  p.ldy = e->widthp;
  p.scale = 1.0f;
  const int planes = launch_linear_groups(e->stream, e->f32, w.down, L.a_act, e->act, g, p, std::max(1, std::min(kMaxSplits, e->plane_rows / pairs)));
  if (planes < 1) return linear_failed(e);
  r->delta = Delta{e->delta, planes, e->widthp, p.plane, e->route_weight, gemv ? nullptr : e->pair_row, L.d.top};
  r->gain = gain;
  return MLLMB200_OK;
}

int keep_residual(Engine* e, const StepCtx& t, int layer, const float* x) {
  if (!e->keep) return MLLMB200_OK;
  LM_CUDA(cudaMemcpyAsync(e->kept + (size_t)layer * e->c.max_rows * e->widthp, x, (size_t)t.rows * e->widthp * 4, cudaMemcpyDeviceToDevice, e->stream));
  e->kept_rows = t.rows;
  return MLLMB200_OK;
}

int latent_mixer(Engine* e, const StepCtx& t, LayerState& L) {
  const Weights& w = L.w;
  const auto& d = L.d;
  Epi p{};
  p.kind = kEpiQLatent;
  p.q = e->proj;
  p.ldq = p.q_end = qk_cols(L);
  p.y = e->fresh;
  p.ldy = L.rankp;
  if (launch_linear(e->stream, e->f32, w.in, e->m_h, e->h, t.rows, p, 1) < 1) return linear_failed(e);
  LatentArgs a{};
  a.heads = d.heads;
  a.dimp = L.dimp;
  a.vdimp = L.vdimp;
  a.rank = d.kv_rank;
  a.rankp = L.rankp;
  a.max_ctx = e->c.max_ctx;
  a.scale = d.score_scale;
  a.eps = e->c.eps;
  a.q = e->proj;
  a.ldq = p.ldq;
  a.cache = L.kc;
  a.fresh = e->fresh;
  a.gain = w.kv_gain;
  a.uk_t = w.uk_t;
  a.uv = w.uk_uv.w + (size_t)qk_cols(L) * L.rankp;
  a.row_sp = t.row_sp;
  a.rows = t.latent_rows;
  a.n_rows = t.n_latent;
  a.ctx = t.latent_ctx;
  a.qa = e->qa;
  a.part_o = e->lat_part;
  a.part_ml = e->lat_ml;
  a.lat = e->lat;
  a.out = e->mix;
  a.ldo = w.out.k;
  const bool with_cache = owns_latent(L) && !t.latent_rows;  // every row attends through the latent
  if (owns_latent(L) && !with_cache) LM_CUDA(launch_latent_cache(e->stream, e->f32, a, t.rows));
  if (a.n_rows) LM_CUDA(launch_latent_absorbed(e->stream, e->f32, a, with_cache));
  for (const ExpandPass& x : t.expand) {
    Groups g;
    g.tiles = x.rows;
    g.max_tiles = g.likely_tiles = x.n_rows;
    g.rows = x.total;
    Epi kv{};
    kv.kind = kEpiQkv;
    kv.kc = e->ex_k;
    kv.vc = e->ex_v;
    kv.k_end = qk_cols(L);
    kv.dimp = L.dimp;
    kv.vdimp = L.vdimp;
    kv.kv_heads = d.heads;
    kv.max_ctx = x.total;
    if (launch_linear_groups(e->stream, e->f32, w.uk_uv, L.a_kc, L.kc, g, kv, 1) < 1) return linear_failed(e);
    AttnShape s{};
    s.heads = s.kv_heads = d.heads;
    s.dimp = L.dimp;
    s.vdimp = L.vdimp;
    s.slot_rows = 1;  // a tile names its sequence's first row
    s.head_rows = x.total;
    s.scale = d.score_scale;
    LM_CUDA(launch_attention(e->stream, e->f32, s, e->proj, p.ldq, t.row_sp, t.rows, e->ex_k, e->ex_v, nullptr, e->mix, a.ldo, x.tiles, x.n_tiles,
                             nullptr, 0, 0, 0, nullptr, nullptr));
  }
  return MLLMB200_OK;
}

int mixer(Engine* e, const StepCtx& t, LayerState& L) {
  if (is_latent(L)) return latent_mixer(e, t, L);
  const Weights& w = e->layers[L.src].w;
  const auto& d = L.d;
  const int ldo = w.out.k;
  Epi p{};
  p.scale = 1.0f;
  if (is_attn(L)) {
    p.kind = kEpiQkv;
    p.q = e->proj;
    p.kc = L.kc;
    p.vc = L.vc;
    p.ldq = qk_cols(L);
    p.q_end = qk_cols(L);
    p.k_end = p.q_end + d.kv_heads * L.dimp;
    p.dimp = L.dimp;
    p.vdimp = L.vdimp;
    p.kv_heads = d.kv_heads;
    p.max_ctx = e->c.max_ctx;
    p.row_sp = t.row_sp;
    if (launch_linear(e->stream, e->f32, w.in, e->m_h, e->h, t.rows, p, 1) < 1) return linear_failed(e);
    AttnShape s{};
    s.heads = d.heads;
    s.kv_heads = d.kv_heads;
    s.dimp = L.dimp;
    s.vdimp = L.vdimp;
    s.slot_rows = (size_t)d.kv_heads * e->c.max_ctx;
    s.head_rows = e->c.max_ctx;
    s.sink = d.sink;
    s.has_bias = d.bias_rows > 0;
    s.bias_max = d.bias_max;
    s.scale = d.score_scale;
    const auto it = t.tiles.find(d.heads / d.kv_heads);
    const int4* tiles = it == t.tiles.end() ? nullptr : it->second.first;
    const int n_tiles = it == t.tiles.end() ? 0 : it->second.second;
    LM_CUDA(launch_attention(e->stream, e->f32, s, e->proj, p.ldq, t.row_sp, t.rows, L.kc, L.vc, w.bias, e->mix, ldo, tiles, n_tiles,
                             t.single ? nullptr : t.single_rows, t.single ? t.rows : t.n_single, t.chunk, t.splits, e->part_o, e->part_ml));
    return MLLMB200_OK;
  }
  p.kind = kEpiPlanes;
  p.y = e->proj;
  p.ldy = 2 * (qk_cols(L) + mix_cols(L));
  if (launch_linear(e->stream, e->f32, w.in, e->m_h, e->h, t.rows, p, 1) < 1) return linear_failed(e);
  RetentionArgs a{};
  a.qkvg = e->proj;
  a.ld = p.ldy;
  a.heads = d.heads;
  a.dim = d.dim;
  a.dimp = L.dimp;
  a.vdim = d.vdim;
  a.vdimp = L.vdimp;
  a.rot_dims = d.rot_dims;
  a.cos_t = L.cos_t;
  a.sin_t = L.sin_t;
  a.decay = w.decay;
  a.state = L.state;
  a.chunk_state = e->chunk_state;
  a.row_sp = t.row_sp;
  a.entries = t.entry;
  a.chunks = t.chunks;
  a.entry_chunks = t.entry_chunks;
  a.n_entries = t.entries;
  a.n_chunks = t.n_chunks;
  a.rows = t.rows;
  a.eps = e->c.eps;
  a.out = e->mix;
  a.ldo = ldo;
  LM_CUDA(t.single ? launch_retention_decode(e->stream, e->f32, a) : launch_retention_prefill(e->stream, e->f32, a));
  return MLLMB200_OK;
}

// Layers with the norms behind the residual sum; the sublayers read x itself.
int forward_post(Engine* e, const StepCtx& t, Stream* r) {
  for (int l = 0; l < e->c.layers; ++l) {
    LayerState& L = e->layers[l];
    const Weights& w = e->layers[L.src].w;
    const bool routed = L.d.experts && fused_router(t.rows);
    LM_OK(mixer(e, t, L));
    LM_OK(delta_linear(e, t, w.out, L.a_mix, e->mix, nullptr, r));
    const RouterArgs ra = router_args(e, l, t.rows <= kGemvRows);
    LM_OK(post_norm(e, t, r, w.norms, routed ? &ra : nullptr));
    if (L.d.ff) {
      if (L.d.experts) {
        LM_OK(moe(e, t, l, routed, nullptr, r));
      } else {
        if (launch_linear(e->stream, e->f32, w.gate_up, e->m_h, e->h, t.rows, gate_epi(e, L, w), 1) < 1) return linear_failed(e);
        LM_OK(delta_linear(e, t, w.down, L.a_act, e->act, nullptr, r));
      }
      LM_OK(post_norm(e, t, r, w.norms + e->widthp, nullptr));
    }
    LM_OK(keep_residual(e, t, l, r->x));
  }
  return MLLMB200_OK;
}

int forward(Engine* e, const StepCtx& t, Stream* r) {
  r->x = e->xa;
  r->other = e->xb;
  LM_CUDA(launch_embed(e->stream, e->f32, t.tokens, e->embed, e->c.width, e->widthp, t.rows, r->x, e->post ? e->h : nullptr, e->route_count,
                       e->n_route_count));
  if (e->post) return forward_post(e, t, r);
  for (int l = 0; l < e->c.layers; ++l) {
    LayerState& L = e->layers[l];
    const Weights& w = e->layers[L.src].w;
    LM_OK(fold_norm(e, t, r, w.norms + 0, &L));
    if (l > 0) LM_OK(keep_residual(e, t, l - 1, r->x));
    LM_OK(mixer(e, t, L));
    LM_OK(delta_linear(e, t, w.out, L.a_mix, e->mix, w.norms + 1, r));
    if (!L.d.ff) continue;
    LM_OK(fold_norm(e, t, r, w.norms + 2, nullptr));
    if (L.d.experts) {
      LM_OK(moe(e, t, l, false, w.norms + 3, r));
      continue;
    }
    if (launch_linear(e->stream, e->f32, w.gate_up, e->m_h, e->h, t.rows, gate_epi(e, L, w), 1) < 1) return linear_failed(e);
    LM_OK(delta_linear(e, t, w.down, L.a_act, e->act, w.norms + 3, r));
  }
  if (e->keep) {
    NormArgs a = norm_args(e, t, *r, e->final_gain, e->h);
    a.x_out = r->other;
    LM_CUDA(launch_norm(e->stream, e->f32, a));
    LM_OK(keep_residual(e, t, e->c.layers - 1, r->other));
  }
  return MLLMB200_OK;
}

// Logits of n <= logit_rows rows named by `gather` (device) into e->logits.
int logits_of(Engine* e, const StepCtx& t, const Stream& r, const int* gather, int n) {
  if (e->post) {
    PostNormArgs a{};
    a.x_in = r.x;
    a.alpha = 1.0f;
    a.gain = e->final_gain;
    a.eps = e->c.eps;
    a.width = e->c.width;
    a.ldx = e->widthp;
    a.rows = n;
    a.out = e->hf;
    a.gather = gather;
    LM_CUDA(launch_post_norm(e->stream, e->f32, a));
  } else {
    NormArgs a = norm_args(e, t, r, e->final_gain, e->hf);
    a.gather = gather;
    a.rows = n;
    LM_CUDA(launch_norm(e->stream, e->f32, a));
  }
  Epi p{};
  p.kind = kEpiPlanes;
  p.y = e->logits;
  p.ldy = e->c.vocab;
  p.scale = e->c.logit_scale;
  if (launch_linear(e->stream, e->f32, e->head, e->m_hf, e->hf, n, p, 1) < 1) return linear_failed(e);
  return MLLMB200_OK;
}

// Greedy tokens of the n rows in e->logits for slots[0, n) (device).
int sample(Engine* e, int n, const int* slots, int* flip) {
  LM_CUDA(launch_argmax(e->stream, e->logits, n, e->c.vocab, kArgmaxBlocks, e->best));
  LM_CUDA(launch_pdl(sample_advance_batched_kernel, dim3(n), dim3(32), 0, e->stream, e->best, kArgmaxBlocks, e->d_pos, e->d_token,
                     e->d_history, e->c.max_ctx, slots, flip));
  return MLLMB200_OK;
}

__global__ void lm_commit_kernel(int n, const int* slots, const int* last_pos, const int* tail, int* d_pos, int* d_tail) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) d_pos[slots[i]] = last_pos[i], d_tail[slots[i]] = tail[i];
}

// ------------------------------------------------------------------------------------------ steps
// Tables of a step, gathered into one host buffer and copied in one piece; offsets are in ints, 16-byte aligned.
struct MetaBuilder {
  std::vector<int>& v;
  explicit MetaBuilder(std::vector<int>& buf) : v(buf) { v.clear(); }
  size_t add(const void* p, size_t ints) {
    const size_t at = (v.size() + 3) / 4 * 4;
    v.resize(at + ints);
    if (ints) memcpy(v.data() + at, p, ints * 4);
    return at;
  }
};

int upload_meta(Engine* e) {
  const size_t n = e->meta.size();
  if (n > e->meta_cap) {
    LM_CUDA(cudaStreamSynchronize(e->stream));
    if (e->meta_h) cudaFreeHost(e->meta_h);
    if (e->meta_d) cudaFree(e->meta_d);
    e->meta_h = e->meta_d = nullptr;
    e->meta_cap = 0;
    LM_CUDA(cudaMallocHost(reinterpret_cast<void**>(&e->meta_h), n * 2 * 4));
    LM_CUDA(cudaMalloc(reinterpret_cast<void**>(&e->meta_d), n * 2 * 4));
    e->meta_cap = n * 2;
  } else {
    LM_CUDA(cudaEventSynchronize(e->meta_free));  // the copy of the step before has left the host buffer
  }
  memcpy(e->meta_h, e->meta.data(), n * 4);
  LM_CUDA(cudaMemcpyAsync(e->meta_d, e->meta_h, n * 4, cudaMemcpyHostToDevice, e->stream));
  LM_CUDA(cudaEventRecord(e->meta_free, e->stream));
  return MLLMB200_OK;
}

int step(Engine* e, int n_entries, const int* slots, const int* counts, const int* tokens, int n_want, const int* want,
         float* logits_out, int do_sample) {
  const auto& c = e->c;
  LM_OK(check_loaded(e));
  if (n_entries < 1 || !slots || !counts || !tokens || n_want < 0 || (n_want && (!want || !logits_out))) return fail(e, MLLMB200_INVALID_ARG, "step arguments");
  std::vector<Entry> entries(n_entries);
  std::vector<char> seen(c.max_seqs, 0);
  long long total = 0;
  bool all_single = true;
  for (int i = 0; i < n_entries; ++i) {
    const int s = slots[i];
    if (s < 0 || s >= c.max_seqs || seen[s] || counts[i] < 1) return fail(e, MLLMB200_INVALID_ARG, "entry %d: slot %d, %d tokens", i, s, counts[i]);
    if ((long long)e->pos[s] + counts[i] > c.max_ctx) return fail(e, MLLMB200_TOO_LARGE, "slot %d: %d + %d tokens, room for %d", s, e->pos[s], counts[i], c.max_ctx);
    seen[s] = 1;
    entries[i] = Entry{s, e->pos[s], (int)total, counts[i], e->tail[s]};
    total += counts[i];
    all_single = all_single && counts[i] == 1;
  }
  if (total > c.max_rows) return fail(e, MLLMB200_TOO_LARGE, "%lld rows in a step, room for %d", total, c.max_rows);
  const int rows = (int)total;
  for (int i = 0; i < rows; ++i)
    if (tokens[i] < 0 || tokens[i] >= c.vocab) return fail(e, MLLMB200_INVALID_ARG, "token %d", tokens[i]);
  for (int i = 0; i < n_want; ++i)
    if (want[i] < 0 || want[i] >= rows) return fail(e, MLLMB200_INVALID_ARG, "wanted place %d of %d rows", want[i], rows);

  std::vector<int2> row_sp(rows), chunks, entry_chunks(n_entries);
  std::vector<int> row_entry(rows), single_rows, last_rows(n_entries), last_pos(n_entries), new_tail(n_entries);
  std::map<int, std::vector<int4>> tiles;
  if (!e->f32 && !all_single)
    for (const auto& L : e->layers)
      if (is_attn(L)) tiles[L.d.heads / L.d.kv_heads];
  int max_single = 0;
  for (int i = 0; i < n_entries; ++i) {
    const Entry& en = entries[i];
    for (int j = 0; j < en.count; ++j) {
      row_sp[en.row0 + j] = make_int2(en.slot, en.pos0 + j);
      row_entry[en.row0 + j] = i;
    }
    last_rows[i] = en.row0 + en.count - 1;
    last_pos[i] = en.pos0 + en.count - 1;
    new_tail[i] = en.tail ^ 1;
    entry_chunks[i] = make_int2((int)chunks.size(), (en.count + kChunk - 1) / kChunk);
    for (int j = 0; j < en.count; j += kChunk) chunks.push_back(make_int2(i, j));
    if (en.count == 1) {
      single_rows.push_back(en.row0);
      max_single = std::max(max_single, en.pos0);
    } else {
      for (auto& g : tiles) {
        const int toks = attention_tile_rows() / g.first;
        for (int j = 0; j < en.count; j += toks)
          g.second.push_back(make_int4(en.row0 + j, std::min(toks, en.count - j), en.slot, en.pos0 + j));
      }
    }
  }
  auto longest_first = [](std::vector<int4>* v) {  // by causal range
    std::stable_sort(v->begin(), v->end(), [](const int4& a, const int4& b) { return a.w + a.y > b.w + b.y; });
  };
  for (auto& g : tiles) longest_first(&g.second);

  struct Pass {
    std::vector<int4> rows, tiles;
    int total = 0;
  };
  std::vector<Pass> passes;
  std::vector<int> latent_rows;
  int latent_ctx = 1;
  bool all_latent = true;
  if (e->latent)
    for (const Entry& en : entries) {
      const int ctx = en.pos0 + en.count;
      if (e->absorb_all || en.count <= kAbsorbMax) {
        for (int j = 0; j < en.count; ++j) latent_rows.push_back(en.row0 + j);
        latent_ctx = std::max(latent_ctx, ctx);
        continue;
      }
      all_latent = false;
      if (passes.empty() || passes.back().total + ctx > e->expand_cap) passes.emplace_back();
      Pass& ps = passes.back();
      const int first = ps.total, cache0 = en.slot * c.max_ctx, tile = group_tile_rows(false), toks = attention_tile_rows();
      for (int j = 0; j < ctx; j += tile) ps.rows.push_back(make_int4(0, cache0 + j, std::min(tile, ctx - j), first + j));
      for (int j = 0; j < en.count; j += toks) ps.tiles.push_back(make_int4(en.row0 + j, std::min(toks, en.count - j), first, en.pos0 + j));
      ps.total += ctx;
    }
  for (auto& ps : passes) longest_first(&ps.tiles);

  MetaBuilder m(e->meta);
  const size_t o_tok = m.add(tokens, rows), o_sp = m.add(row_sp.data(), 2 * (size_t)rows), o_re = m.add(row_entry.data(), rows);
  const size_t o_en = m.add(entries.data(), 5 * (size_t)n_entries), o_ch = m.add(chunks.data(), 2 * chunks.size());
  const size_t o_ec = m.add(entry_chunks.data(), 2 * (size_t)n_entries), o_sr = m.add(single_rows.data(), single_rows.size());
  const size_t o_lr = m.add(last_rows.data(), n_entries), o_lp = m.add(last_pos.data(), n_entries), o_nt = m.add(new_tail.data(), n_entries);
  const size_t o_sl = m.add(slots, n_entries), o_want = m.add(want, n_want);
  std::map<int, size_t> o_tiles;
  for (auto& g : tiles) o_tiles[g.first] = m.add(g.second.data(), 4 * g.second.size());
  const size_t o_lat = m.add(latent_rows.data(), latent_rows.size());
  std::vector<std::pair<size_t, size_t>> o_pass;
  for (auto& ps : passes) {
    const size_t o_rows = m.add(ps.rows.data(), 4 * ps.rows.size());
    o_pass.push_back({o_rows, m.add(ps.tiles.data(), 4 * ps.tiles.size())});
  }
  LM_OK(upload_meta(e));

  const int* d = e->meta_d;
  StepCtx t;
  t.rows = rows;
  t.entries = n_entries;
  t.tokens = d + o_tok;
  t.row_sp = reinterpret_cast<const int2*>(d + o_sp);
  t.row_entry = d + o_re;
  t.entry = reinterpret_cast<const Entry*>(d + o_en);
  t.chunks = reinterpret_cast<const int2*>(d + o_ch);
  t.entry_chunks = reinterpret_cast<const int2*>(d + o_ec);
  t.n_chunks = (int)chunks.size();
  t.single = all_single;
  t.single_rows = d + o_sr;
  t.n_single = (int)single_rows.size();
  t.chunk = decode_chunk(t.n_single, max_single + 1);
  t.splits = max_single / t.chunk + 1;
  for (auto& g : tiles) t.tiles[g.first] = {reinterpret_cast<const int4*>(d + o_tiles[g.first]), (int)g.second.size()};

  t.latent_rows = all_latent ? nullptr : d + o_lat;
  t.n_latent = (int)latent_rows.size();
  t.latent_ctx = latent_ctx;
  for (size_t i = 0; i < passes.size(); ++i)
    t.expand.push_back({reinterpret_cast<const int4*>(d + o_pass[i].first), reinterpret_cast<const int4*>(d + o_pass[i].second),
                        (int)passes[i].rows.size(), (int)passes[i].tiles.size(), passes[i].total});

  const long long before = g_launches;
  Stream r{};
  LM_OK(forward(e, t, &r));
  for (int w0 = 0; w0 < n_want; w0 += e->logit_rows) {
    const int n = std::min(e->logit_rows, n_want - w0);
    LM_OK(logits_of(e, t, r, d + o_want + w0, n));
    LM_CUDA(cudaMemcpyAsync(logits_out + (size_t)w0 * c.vocab, e->logits, (size_t)n * c.vocab * 4, cudaMemcpyDeviceToHost, e->stream));
  }
  if (do_sample) {
    lm_commit_kernel<<<(n_entries + 127) / 128, 128, 0, e->stream>>>(n_entries, d + o_sl, d + o_lp, d + o_nt, e->d_pos, e->d_tail);
    ++g_launches;
    LM_OK(logits_of(e, t, r, d + o_lr, n_entries));
    LM_OK(sample(e, n_entries, d + o_sl, nullptr));
  }
  LM_CUDA(cudaGetLastError());
  if (n_want) LM_CUDA(cudaStreamSynchronize(e->stream));
  e->launches += g_launches - before;
  for (const Entry& en : entries) {
    e->pos[en.slot] = en.pos0 + en.count;
    e->tail[en.slot] ^= 1;
    e->ready[en.slot] = do_sample != 0;
  }
  return MLLMB200_OK;
}

int enqueue_decode(Engine* e, int count, int chunk, int splits) {
  StepCtx t;
  t.rows = t.entries = count;
  t.tokens = e->d_row_token;
  t.row_sp = e->d_row_sp;
  t.row_entry = e->d_row_entry;
  t.entry = e->d_entries;
  t.single = true;
  t.chunk = chunk;
  t.splits = splits;
  t.n_latent = count;
  t.latent_ctx = std::min(chunk * splits, e->c.max_ctx);
  LM_CUDA(launch_decode_prep(e->stream, count, e->d_slots, e->d_pos, e->d_token, e->d_tail, e->d_row_sp, e->d_row_token, e->d_entries, e->d_row_entry));
  Stream r{};
  LM_OK(forward(e, t, &r));
  LM_OK(logits_of(e, t, r, e->d_identity, count));
  return sample(e, count, e->d_slots, e->d_tail);
}

int decode(Engine* e, int count, const int* slots, int steps) {
  const auto& c = e->c;
  LM_OK(check_loaded(e));
  if (count < 1 || count > c.max_seqs || count > c.max_rows || !slots || steps < 0) return fail(e, MLLMB200_INVALID_ARG, "decode arguments");
  std::vector<char> seen(c.max_seqs, 0);
  int longest = 0;
  for (int i = 0; i < count; ++i) {
    const int s = slots[i];
    if (s < 0 || s >= c.max_seqs || seen[s] || !e->ready[s]) return fail(e, MLLMB200_INVALID_ARG, "slot %d has no current token", s);
    if (e->pos[s] + steps > c.max_ctx) return fail(e, MLLMB200_TOO_LARGE, "slot %d: %d + %d tokens, room for %d", s, e->pos[s], steps, c.max_ctx);
    seen[s] = 1;
    longest = std::max(longest, e->pos[s]);
  }
  std::vector<int> now(slots, slots + count);
  if (now != e->cur_slots) {
    LM_CUDA(cudaMemcpyAsync(e->d_slots, now.data(), (size_t)count * 4, cudaMemcpyHostToDevice, e->stream));
    e->cur_slots = now;
  }
  for (int i = 0; i < steps; ++i, ++longest) {
    const int chunk = decode_chunk(count, longest + 1);
    int splits = 1;  // one graph per power of two of context chunks
    while (splits * chunk < longest + 1) splits *= 2;
    splits = std::min(splits, (c.max_ctx + chunk - 1) / chunk);
    auto it = e->graphs.find({count, chunk, splits});
    if (it == e->graphs.end()) {
      const long long before = g_launches;
      cudaGraph_t g = nullptr;
      LM_CUDA(cudaStreamBeginCapture(e->stream, cudaStreamCaptureModeThreadLocal));
      const int st = enqueue_decode(e, count, chunk, splits);
      const cudaError_t r = cudaStreamEndCapture(e->stream, &g);
      Graph gr{nullptr, g_launches - before};
      if (st == MLLMB200_OK && r == cudaSuccess) {
        const cudaError_t q = cudaGraphInstantiate(&gr.exec, g, 0);
        cudaGraphDestroy(g);
        LM_CUDA(q);
      } else {
        if (g) cudaGraphDestroy(g);
        LM_OK(st);
        LM_CUDA(r);
      }
      it = e->graphs.emplace(GraphKey{count, chunk, splits}, gr).first;
    }
    LM_CUDA(cudaGraphLaunch(it->second.exec, e->stream));
    e->launches += it->second.launches;
    for (int s : now) {
      ++e->pos[s];
      e->tail[s] ^= 1;
    }
  }
  return MLLMB200_OK;
}

Engine* from(void* h) { return static_cast<Engine*>(h); }

void destroy(Engine* e) {
  if (e->stream) cudaStreamSynchronize(e->stream);
  for (auto& g : e->graphs) cudaGraphExecDestroy(g.second.exec);
  for (void* p : e->owned) cudaFree(p);
  if (e->kept) cudaFree(e->kept);
  if (e->meta_h) cudaFreeHost(e->meta_h);
  if (e->meta_d) cudaFree(e->meta_d);
  if (e->meta_free) cudaEventDestroy(e->meta_free);
  if (e->stream) cudaStreamDestroy(e->stream);
  delete e;
}

thread_local std::string t_create_error;

}  // namespace
}  // namespace lm
}  // namespace mllmb200

using namespace mllmb200;
using namespace mllmb200::lm;

extern "C" {

int mllmb200_lm_create(const mllmb200_lm_config* cfg, const mllmb200_lm_layer* layers, void** handle) {
  if (!cfg || !layers || !handle) return MLLMB200_INVALID_ARG;
  auto* e = new Engine();
  e->c = *cfg;
  const int st = create(e, layers);
  if (st != MLLMB200_OK) {
    t_create_error = e->error;
    destroy(e);
    return st;
  }
  *handle = e;
  return MLLMB200_OK;
}
void mllmb200_lm_destroy(void* handle) {
  if (handle) destroy(from(handle));
}
int mllmb200_lm_set_tensor(void* handle, int layer, int which, const void* data, int rows, int cols) {
  if (!handle || !data) return MLLMB200_INVALID_ARG;
  return set_tensor(from(handle), layer, which, data, rows, cols);
}
int mllmb200_lm_set_expert(void* handle, int layer, int expert, int which, const void* data, int rows, int cols) {
  if (!handle || !data) return MLLMB200_INVALID_ARG;
  return set_expert(from(handle), layer, expert, which, data, rows, cols);
}
int mllmb200_lm_step(void* handle, int entries, const int* slots, const int* counts, const int* tokens, int n_want, const int* want,
                     float* logits_out, int sample) {
  return handle ? step(from(handle), entries, slots, counts, tokens, n_want, want, logits_out, sample) : MLLMB200_INVALID_ARG;
}
int mllmb200_lm_decode(void* handle, int count, const int* slots, int steps) {
  return handle ? decode(from(handle), count, slots, steps) : MLLMB200_INVALID_ARG;
}
int mllmb200_lm_free_slot(void* handle, int slot) {
  auto* e = from(handle);
  if (!e || slot < 0 || slot >= e->c.max_seqs) return MLLMB200_INVALID_ARG;
  e->pos[slot] = e->tail[slot] = e->ready[slot] = 0;
  return MLLMB200_OK;
}
int mllmb200_lm_read(void* handle, int slot, int first, int count, int* tokens_out, int* length_out) {
  auto* e = from(handle);
  if (!e || slot < 0 || slot >= e->c.max_seqs || first < 0 || count < 0 || first + count > e->c.max_ctx) return MLLMB200_INVALID_ARG;
  LM_CUDA(cudaStreamSynchronize(e->stream));
  if (tokens_out && count) LM_CUDA(cudaMemcpy(tokens_out, e->d_history + (size_t)slot * e->c.max_ctx + first, (size_t)count * 4, cudaMemcpyDeviceToHost));
  if (length_out) *length_out = e->pos[slot];
  return MLLMB200_OK;
}
int mllmb200_lm_keep_residual(void* handle, int on) {
  auto* e = from(handle);
  if (!e) return MLLMB200_INVALID_ARG;
  if (on && !e->kept) LM_CUDA(cudaMalloc(reinterpret_cast<void**>(&e->kept), (size_t)e->c.layers * e->c.max_rows * e->widthp * 4));
  e->keep = on != 0;
  return MLLMB200_OK;
}
int mllmb200_lm_read_residual(void* handle, int layer, int rows, float* out) {
  auto* e = from(handle);
  if (!e || !out || !e->kept || layer < 0 || layer >= e->c.layers || rows < 0 || rows > e->kept_rows) return MLLMB200_INVALID_ARG;
  LM_CUDA(cudaStreamSynchronize(e->stream));
  LM_CUDA(cudaMemcpy2D(out, (size_t)e->c.width * 4, e->kept + (size_t)layer * e->c.max_rows * e->widthp, (size_t)e->widthp * 4,
                       (size_t)e->c.width * 4, rows, cudaMemcpyDeviceToHost));
  return MLLMB200_OK;
}
int mllmb200_lm_stats(void* handle, size_t* state_bytes, long long* launches) {
  auto* e = from(handle);
  if (!e) return MLLMB200_INVALID_ARG;
  if (state_bytes) *state_bytes = e->state_bytes;
  if (launches) *launches = e->launches;
  return MLLMB200_OK;
}
int mllmb200_lm_synchronize(void* handle) {
  auto* e = from(handle);
  if (!e) return MLLMB200_INVALID_ARG;
  LM_CUDA(cudaStreamSynchronize(e->stream));
  return MLLMB200_OK;
}
void* mllmb200_lm_stream(void* handle) { return handle ? from(handle)->stream : nullptr; }
const char* mllmb200_lm_last_error(void* handle) { return handle ? from(handle)->error.c_str() : t_create_error.c_str(); }
int mllmb200_lm_check_device_status(void* handle) {
  auto* e = from(handle);
  if (!e) return MLLMB200_INVALID_ARG;
  int status = MLLMB200_OK;
  LM_CUDA(read_device_status(e->stream, &status));
  return status;
}
int mllmb200_lm_distance_buckets(int bias_rows, int bias_max, int count, int* out) {
  if (bias_rows < 2 || bias_max <= bias_rows / 2 || count < 0 || !out) return MLLMB200_INVALID_ARG;
  for (int n = 0; n < count; ++n) out[n] = bucket_of(n, bias_rows, bias_max);
  return MLLMB200_OK;
}

}  // extern "C"
