// Types shared by the translation units of the bf16 language-model engine.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <map>
#include <string>
#include <vector>

#include "../../../include/mllmb200_lm.h"

namespace mllmb200 {
namespace lm {

constexpr int kSms = 148;
constexpr int kChunk = 64;      // tokens per retention chunk
constexpr int kMaxSplits = 8;   // K splits of a linear whose consumer adds the partial sums

inline int pad_to(int v, int a) { return (v + a - 1) / a * a; }

// One sequence's share of a step.
struct Entry {
  int slot, pos0, row0, count;
  int tail;  // which of the two convolution tails holds the state before this step
};

// Where a linear's result goes.
enum EpiKind { kEpiPlanes = 0, kEpiQkv = 1, kEpiGate = 2, kEpiQLatent = 3 };
struct Epi {
  int kind;
  // kEpiPlanes: fp32 [split][M][ldy] partial sums times scale (one plane when K is not split)
  float* y;
  size_t plane;
  int ldy;
  float scale;
  // kEpiQkv: columns [0, q_end) to q [M][ldq], then the keys and values of every kv head straight into the caches
  // [slot][kv_heads][max_ctx][dimp | vdimp] at the row's slot and position (slot 0, position = row without row_sp)
  // kEpiQLatent: columns [0, q_end) to q [M][ldq], the rest in fp32 to y [M][ldy]
  void *q, *kc, *vc;
  int ldq, q_end, k_end, dimp, vdimp, kv_heads, max_ctx;
  const int2* row_sp;  // {slot, position} of every row
  // kEpiGate: columns (2 i, 2 i + 1) = (gate_i, up_i); writes act(gate_i, up_i), an MLLMB200_LM_ACT_* form
  void* act;
  int ld_act, act_kind;
  float limit;
};

// A linear map in the engine's layout: bf16 [groups][n][k] with k a multiple of 64 (zero padded).
struct Linear {
  __nv_bfloat16* w = nullptr;
  int n = 0, k = 0, groups = 1;
  CUtensorMap map32, map128;  // boxes of 32 / 128 rows x 64 columns, 128-byte swizzle
};

// Rows that choose among the groups of a Linear (experts), or scattered runs of rows.
struct Groups {
  // tiles of up to group_tile_rows() rows that share a group: {group, first row of x, rows, first row of the result}
  const int4* tiles = nullptr;
  const int* n_tiles = nullptr;  // device count; nullptr: max_tiles are there
  int max_tiles = 0;
  int rows = 0;                  // rows of all tiles
  int likely_tiles = 0;          // for the choice of the tile shape
  // few rows: result row i takes x row i / div and group group_of[i]
  const int* group_of = nullptr;
  int div = 1;
};

// Activations of a linear: [max_rows][k] in a fixed buffer.
struct ActMap {
  CUtensorMap map16, map128;
};

// Keys and values of head g of slot s lie at rows s * slot_rows + g * head_rows + position.
struct AttnShape {
  int heads, kv_heads, dimp, vdimp, sink, bias_max, has_bias;
  size_t slot_rows, head_rows;
  float scale;
};

struct Weights {  // tensors of a layer that owns some
  // in = q|k|v (attention), q|k|v|g (retention), q|down-projection (latent attention that makes its own rows)
  // gate_up, down: one group, or one per expert
  Linear in, out, gate_up, down;
  float* norms = nullptr;         // sandwich: norm1, norm1b, norm2, norm2b; post: norm1 and norm2, [2][widthp]
  Linear uk_uv;                   // latent attention: k rows of all heads | v rows of all heads, [..][rankp]
  __nv_bfloat16* uk_t = nullptr;  // the k rows transposed per head, [heads][rankp][dimp]
  float* kv_gain = nullptr;       // [rankp]
  Linear router;                  // [experts][widthp]
  float* router_b = nullptr;
  std::vector<unsigned> expert_loaded;
  float* conv = nullptr;          // [taps][widthp]
  float* bias = nullptr;          // attention: [heads][bias_max + 1]
  float* decay = nullptr;         // retention: [heads][kChunk + 1] powers
  unsigned loaded = 0;            // bit per tensor
};

struct LayerState {
  mllmb200_lm_layer d;
  int src = 0;            // layer whose weights it uses
  int dimp = 0, vdimp = 0, rankp = 0;
  Weights w;
  ActMap a_mix, a_act, a_kc;
  void *kc = nullptr, *vc = nullptr;  // attention caches; latent attention: kc [slot][max_ctx][rankp], maybe an earlier layer's
  float* state = nullptr;             // retention [slot][heads][dimp][vdimp]
  float* tail = nullptr;              // convolution [slot][2][taps - 1][widthp]
  float *cos_t = nullptr, *sin_t = nullptr;  // rotation tables [max_ctx][rot_dims / 2], shared between equal layers
};

// The sublayer output a norm folds in: `planes` partial sums of fp32 [rows][ldx], or with `mix_w` the weighted sum of the
// rows mix_row[row * top + k] (row * top + k without mix_row).
struct Delta {
  const float* p;
  int planes, ldx;
  size_t plane;
  const float* mix_w;
  const int* mix_row;
  int top;
};

// Choice of experts for every row: logits of x and the router, the `top` largest, softmax over those.
struct RouterArgs {
  const __nv_bfloat16* w;  // [experts][ldw]; nullptr: no router
  const float* b;
  int experts, top, ldw;
  int* sel;                // [rows][top]
  float* weight;           // [rows][top]
  int *count, *rank;       // rows per expert so far, and a pair's place among them (nullptr: not wanted)
};

// x' = rms_unit(alpha x + delta) * gain (one number per column), to x_out (fp32) and out; x_out may be x_in.
struct PostNormArgs {
  const float* x_in;
  float* x_out;            // nullptr: not kept
  Delta delta;             // p = nullptr: none
  float alpha;
  const float* gain;
  float eps;
  int width, ldx, rows;
  void* out;
  const int* gather;       // out row r reads row gather[r]
  RouterArgs router;       // with few rows only (see fused_router)
};

struct NormArgs {
  const float* x_in;
  float* x_out;               // nullptr: not kept
  Delta delta;                // p = nullptr: none
  const float *g_post, *g_pre;
  float eps;
  int width, ldx;             // ldx = width rounded up to 64, zero padded
  void* out;                  // [rows][ldx]
  const int* gather;          // out row r reads row gather[r] (no convolution then)
  int rows;
  // convolution (taps = 0: none)
  int taps;
  const float* conv_w;
  float* tail;
  const Entry* entries;
  const int* row_entry;
  int rows_per_cta;
};

// launchers -----------------------------------------------------------------------------------
int make_act_map(ActMap* m, const void* buf, int rows, int k);
int make_linear_maps(Linear* l);
// x: [>= M][k] activations; returns the number of K splits used (planes written), negative on error
int launch_linear(cudaStream_t s, bool f32, const Linear& w, const ActMap& am, const void* x, int M, const Epi& e, int max_splits);
// the same over groups of rows
int launch_linear_groups(cudaStream_t s, bool f32, const Linear& w, const ActMap& am, const void* x, const Groups& g, const Epi& e, int max_splits);
int group_tile_rows(bool f32);
constexpr int kGemvRows = 4;  // up to that many rows a linear takes the GEMV kernel
cudaError_t linear_configure();
// src [heads * dim][rank] to dst [heads][rankp][dimp]
cudaError_t launch_pack_heads_transposed(cudaStream_t s, const __nv_bfloat16* src, int heads, int dim, int rank, __nv_bfloat16* dst,
                                         int rankp, int dimp);
cudaError_t launch_pack_rows(cudaStream_t s, const __nv_bfloat16* src, int n, int k, __nv_bfloat16* dst, int ldk, int row_block,
                             int row_block_pad, int row_mul, int row_off, int col_block, int col_block_pad);
cudaError_t launch_norm(cudaStream_t s, bool f32, const NormArgs& a);
cudaError_t launch_post_norm(cudaStream_t s, bool f32, const PostNormArgs& a);
bool fused_router(int rows);  // whether launch_post_norm takes a router with that many rows
// h (may be nullptr): the same rows in the number format of the activations; zeroes n_zero ints at zero
cudaError_t launch_embed(cudaStream_t s, bool f32, const int* tokens, const __nv_bfloat16* table, int width, int ldx, int rows, float* x,
                         void* h, int* zero, int n_zero);
// experts chosen from router logits [planes][rows][ldl]
cudaError_t launch_topk(cudaStream_t s, const RouterArgs& a, const float* logits, int ldl, int planes, size_t plane, int rows);
// rows of x to their places in expert order, and the tiles of the experts' rows
cudaError_t launch_moe_permute(cudaStream_t s, bool f32, const RouterArgs& a, const void* x, int ldx, int rows, void* out, int* pair_row,
                               int4* tiles, int* n_tiles);
constexpr int kMaxExperts = 1024, kMaxTop = 32;
cudaError_t launch_decode_prep(cudaStream_t s, int n, const int* slots, const int* pos, const int* token, const int* flip,
                               int2* row_sp, int* row_token, Entry* entries, int* row_entry);
cudaError_t launch_argmax(cudaStream_t s, const float* logits, int rows, int vocab, int blocks, float2* best);
cudaError_t launch_attention(cudaStream_t s, bool f32, const AttnShape& a, const void* q, int ldq, const int2* row_sp, int rows,
                             const void* kc, const void* vc, const float* bias, void* out, int ldo, const int4* tiles, int n_tiles,
                             const int* single_rows, int n_single, int chunk, int splits, float* part_o, float2* part_ml);
int attention_tile_rows();
constexpr int kMinDecodeChunk = 64;  // cache positions per CTA of the decode attention: 64, or 128 in large batches
cudaError_t attention_configure();
cudaError_t launch_rope_table(cudaStream_t s, float* cos_t, float* sin_t, int max_pos, int dims, double base);
// Latent attention: one cached row of rankp numbers per position, shared by all heads.
struct LatentArgs {
  int heads, dimp, vdimp, rank, rankp, max_ctx;
  float scale, eps;
  const void* q;               // [rows][ldq]
  int ldq;
  void* cache;                 // [slot][max_ctx][rankp]
  const float *fresh, *gain;   // rows of the step before their norm, fp32 [rows][rankp]; nullptr: another layer makes them
  const __nv_bfloat16 *uk_t, *uv;
  const int2* row_sp;
  const int* rows;             // rows that attend through the latent itself; nullptr = 0 .. n_rows - 1
  int n_rows, ctx;             // ctx: at least the longest context among them
  void* qa;                    // [n_rows][heads][rankp] queries against the latent
  float *part_o, *lat;         // bf16: partial outputs per context split; fp32 mode: [n_rows][heads][rankp]
  float2* part_ml;
  void* out;                   // [rows][ldo]
  int ldo;
};
cudaError_t latent_configure();
cudaError_t launch_latent_cache(cudaStream_t s, bool f32, const LatentArgs& a, int rows);
// cache_rows: the rows of the step are the rows of `a`, and the first kernel writes their latents to the cache as well
cudaError_t launch_latent_absorbed(cudaStream_t s, bool f32, const LatentArgs& a, bool cache_rows);
size_t latent_parts(int rows);  // (row, split) pairs that launch_latent_absorbed needs room for, at most
constexpr int kAbsorbMax = 16;  // a sequence's share of a step up to which its rows attend through the latent
constexpr int kMaxRank = 1024;
struct RetentionArgs {
  const float* qkvg;  // [rows][ld]: q | k | v | g, heads x dimp, heads x dimp, heads x vdimp, heads x vdimp
  int ld, heads, dim, dimp, vdim, vdimp, rot_dims;
  const float *cos_t, *sin_t, *decay;
  float* state;        // [slot][heads][dimp][vdimp]
  float* chunk_state;  // [chunks][heads][dimp][vdimp]
  const int2* row_sp;
  const Entry* entries;
  const int2* chunks;       // {entry, first row offset inside the entry}
  const int2* entry_chunks; // per entry: {first chunk, count}
  int n_entries, n_chunks, rows;
  float eps;
  void* out;
  int ldo;
};
cudaError_t launch_retention_decode(cudaStream_t s, bool f32, const RetentionArgs& a);
cudaError_t launch_retention_prefill(cudaStream_t s, bool f32, const RetentionArgs& a);
cudaError_t retention_configure();

// launch with the programmatic-dependent-launch attribute (the kernels call griddepcontrol themselves)
extern thread_local long long g_launches;
template <class... KArgs, class... Args>
cudaError_t launch_pdl_cluster(void (*kernel)(KArgs...), dim3 grid, dim3 block, dim3 cluster, size_t smem, cudaStream_t s, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = cluster.x;
  attr[1].val.clusterDim.y = cluster.y;
  attr[1].val.clusterDim.z = cluster.z;
  cfg.attrs = attr;
  cfg.numAttrs = cluster.x * cluster.y * cluster.z > 1 ? 2 : 1;
  ++g_launches;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}
template <class... KArgs, class... Args>
cudaError_t launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args... args) {
  return launch_pdl_cluster(kernel, grid, block, dim3(1, 1, 1), smem, s, args...);
}

}  // namespace lm
}  // namespace mllmb200
