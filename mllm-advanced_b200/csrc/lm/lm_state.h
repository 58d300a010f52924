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
enum EpiKind { kEpiPlanes = 0, kEpiQkv = 1, kEpiGate = 2 };
struct Epi {
  int kind;
  // kEpiPlanes: fp32 [split][M][ldy] partial sums times scale (one plane when K is not split)
  float* y;
  size_t plane;
  int ldy;
  float scale;
  // kEpiQkv: columns [0, q_end) to q [M][ldq], then the keys and values of every kv head straight into the caches
  // [slot][kv_heads][max_ctx][dimp | vdimp] at the row's slot and position
  void *q, *kc, *vc;
  int ldq, q_end, k_end, dimp, vdimp, kv_heads, max_ctx;
  const int2* row_sp;  // {slot, position} of every row
  // kEpiGate: columns (2 i, 2 i + 1) = (gate_i, up_i); writes min(g,l) sigmoid(1.702 min(g,l)) (clamp(u,-l,l) + 1)
  void* act;
  int ld_act;
  float limit;
};

// A linear map in the engine's layout: bf16 [n][k] with k a multiple of 64 (zero padded).
struct Linear {
  __nv_bfloat16* w = nullptr;
  int n = 0, k = 0;
  CUtensorMap map32, map128;  // boxes of 32 / 128 rows x 64 columns, 128-byte swizzle
};

// Activations of a linear: [max_rows][k] in a fixed buffer.
struct ActMap {
  CUtensorMap map16, map128;
};

struct AttnShape {
  int heads, kv_heads, dimp, vdimp, max_ctx, sink, bias_max, has_bias;
  float scale;
};

struct Weights {  // tensors of a layer that owns some
  Linear in, out, gate_up, down;  // in = q|k|v (attention), q|k|v|g (retention)
  float* norms = nullptr;         // norm1, norm1b, norm2, norm2b
  float* conv = nullptr;          // [taps][widthp]
  float* bias = nullptr;          // attention: [heads][bias_max + 1]
  float* decay = nullptr;         // retention: [heads][kChunk + 1] powers
  unsigned loaded = 0;            // bit per tensor
};

struct LayerState {
  mllmb200_lm_layer d;
  int src = 0;            // layer whose weights it uses
  int dimp = 0, vdimp = 0;
  Weights w;
  ActMap a_mix, a_act;
  void *kc = nullptr, *vc = nullptr;  // attention caches
  float* state = nullptr;             // retention [slot][heads][dimp][vdimp]
  float* tail = nullptr;              // convolution [slot][2][taps - 1][widthp]
  float *cos_t = nullptr, *sin_t = nullptr;  // rotation tables [max_ctx][rot_dims / 2], shared between equal layers
};

struct NormArgs {
  const float* x_in;
  float* x_out;               // nullptr: not kept
  const float* delta;         // [planes][rows][ldx] sublayer output, or nullptr
  int planes;
  size_t plane;
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
cudaError_t linear_configure();
cudaError_t launch_pack_rows(cudaStream_t s, const __nv_bfloat16* src, int n, int k, __nv_bfloat16* dst, int ldk, int row_block,
                             int row_block_pad, int row_mul, int row_off, int col_block, int col_block_pad);
cudaError_t launch_norm(cudaStream_t s, bool f32, const NormArgs& a);
cudaError_t launch_embed(cudaStream_t s, const int* tokens, const __nv_bfloat16* table, int width, int ldx, int rows, float* x);
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
cudaError_t launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr;
  attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr.val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = &attr;
  cfg.numAttrs = 1;
  ++g_launches;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

}  // namespace lm
}  // namespace mllmb200
