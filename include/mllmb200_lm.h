/*
 * mllmb200_lm.h - C ABI of the bf16 language-model engine (library lib/libmllm_b200_lm.so).
 *
 * The engine runs decoder-only models that are described layer by layer: a sequence mixer (softmax attention, latent
 * attention or retention), an optional gated feed-forward (dense or a mixture of experts), norms around or behind the
 * sublayers and an optional causal input convolution, every size and constant a parameter.  It owns the weights, the
 * per-sequence state (key/value caches, latent caches, retention states, convolution tails) in `max_seqs` slots, and a step function that advances any mix of sequences - whole prompts, portions of
 * prompts and single tokens - in one ragged batch.  Pure decoding replays one CUDA graph per token.
 * The reference project drives its models the same way from above (config, load by name, prompt then greedy loop:
 * mllm/Models/AutoLLM.hpp:39-105) but holds one sequence only.
 *
 * Status codes are those of mllmb200.h.  All calls are made from one thread at a time per handle.
 */
#ifndef MLLMB200_LM_H_
#define MLLMB200_LM_H_

#include "mllmb200.h"

#ifdef __cplusplus
extern "C" {
#endif

enum { MLLMB200_LM_BF16 = 0, MLLMB200_LM_F32 = 1 };           /* activations, caches and matrix products */
enum { MLLMB200_LM_ATTENTION = 0, MLLMB200_LM_RETENTION = 1, MLLMB200_LM_LATENT = 2 }; /* mixers */
/* Gated feed-forwards, act(g) times a form of u:
 * CLAMPED: min(g, l) sigmoid(1.702 min(g, l)) (clamp(u, -l, l) + 1), l = ff_limit
 * GELU:    gelu(g) u, gelu in its tanh form;   SILU: g sigmoid(g) u */
enum { MLLMB200_LM_ACT_CLAMPED = 0, MLLMB200_LM_ACT_GELU = 1, MLLMB200_LM_ACT_SILU = 2 };
/* Norms around the sublayers:
 * SANDWICH: x + norm_b(sublayer(norm(x))), one gain per norm
 * POST:     norm(residual_scale x + sublayer(x)), one gain per column */
enum { MLLMB200_LM_NORM_SANDWICH = 0, MLLMB200_LM_NORM_POST = 1 };

typedef struct mllmb200_lm_config {
  int vocab, width, layers;
  int dtype;        /* MLLMB200_LM_BF16: bf16 matrix products with fp32 accumulation; MLLMB200_LM_F32: fp32 throughout */
  int conv_taps;    /* causal input convolution of every layer, h + conv(h); 0 = none */
  int max_seqs;     /* slots */
  int max_ctx;      /* tokens per slot */
  int max_rows;     /* tokens per step over all sequences */
  float eps;        /* of every RMS norm */
  float logit_scale;
  int norm_place;   /* MLLMB200_LM_NORM_* */
  float residual_scale; /* POST only */
} mllmb200_lm_config;

typedef struct mllmb200_lm_layer {
  int mixer;                 /* MLLMB200_LM_ATTENTION / MLLMB200_LM_RETENTION / MLLMB200_LM_LATENT */
  int heads, kv_heads;       /* retention and latent attention: kv_heads = heads */
  int dim, vdim;             /* per head: query/key and value size */
  float score_scale;         /* attention, latent attention: multiplies q.k (the distance bias is added after it) */
  int sink;                  /* attention: 1 = a key of score 0 without a value joins the softmax */
  int bias_rows, bias_max;   /* attention: rows of the learned distance-bias table and its largest distance; rows 0 = no bias */
  int rot_dims;              /* retention: rotated coordinates of every head, 0 = none */
  double rot_base;
  int ff;                    /* feed-forward width (of one expert), 0 = the layer has none */
  float ff_limit;            /* clamp of the gated feed-forward: min(g, limit), clamp(u, -limit, limit) */
  int weights_of;            /* -1, or the layer whose tensors this one uses (cache and state stay its own) */
  int kv_rank;               /* latent attention: cached numbers per position, from which every head's key and value are made */
  int kv_from;               /* latent attention: -1, or the earlier layer whose cached rows this one uses */
  int act;                   /* MLLMB200_LM_ACT_* */
  int experts, top;          /* mixture of experts: their number and how many a token uses; experts 0 = a dense feed-forward */
} mllmb200_lm_layer;

/* Tensors of a layer; linear maps are bf16 [out, in] row-major. */
enum {
  MLLMB200_LM_T_Q = 0, MLLMB200_LM_T_K, MLLMB200_LM_T_V, MLLMB200_LM_T_G, MLLMB200_LM_T_O,
  MLLMB200_LM_T_GATE, MLLMB200_LM_T_UP, MLLMB200_LM_T_DOWN,
  MLLMB200_LM_T_NORM1, MLLMB200_LM_T_NORM1B, MLLMB200_LM_T_NORM2, MLLMB200_LM_T_NORM2B, /* fp32: one number each (SANDWICH);
                                                                                        NORM1 and NORM2, [width] (POST) */
  MLLMB200_LM_T_CONV,        /* fp32 [width, taps] */
  MLLMB200_LM_T_REL,         /* fp32 [bias_rows, heads] */
  MLLMB200_LM_T_DECAY,       /* fp64 [heads] */
  MLLMB200_LM_T_DKV,         /* latent attention: bf16 [kv_rank, width], fp32 [kv_rank], bf16 [heads dim, kv_rank], [heads vdim, kv_rank] */
  MLLMB200_LM_T_DKV_NORM, MLLMB200_LM_T_UK, MLLMB200_LM_T_UV,
  MLLMB200_LM_T_ROUTER,      /* bf16 [experts, width] */
  MLLMB200_LM_T_ROUTER_B,    /* fp32 [experts] */
  MLLMB200_LM_T_COUNT,
  /* tensors of the model (layer = -1) */
  MLLMB200_LM_T_EMBED = 100, MLLMB200_LM_T_HEAD, /* bf16 [vocab, width] */
  MLLMB200_LM_T_FINAL_NORM                       /* fp32: one number (SANDWICH) or [width] (POST) */
};

MLLMB200_API int mllmb200_lm_create(const mllmb200_lm_config* cfg, const mllmb200_lm_layer* layers, void** handle);
MLLMB200_API void mllmb200_lm_destroy(void* handle);

/* Loads one tensor (layer -1: a tensor of the model).  `data` may be host or device memory; rows x cols must be the
 * tensor's shape ([1, n] for a vector).  The engine keeps its own packed copy. */
MLLMB200_API int mllmb200_lm_set_tensor(void* handle, int layer, int which, const void* data, int rows, int cols);
/* The same for GATE, UP and DOWN of one expert of a mixture. */
MLLMB200_API int mllmb200_lm_set_expert(void* handle, int layer, int expert, int which, const void* data, int rows, int cols);

/* One step over `entries` sequences: entry e appends counts[e] >= 1 tokens to slot slots[e] (each slot at most once per
 * step).  tokens: all entries' tokens one after the other (host).  want: places among these sum(counts) rows whose
 * logits are copied to logits_out (host, fp32 [n_want, vocab], in the order of want).  sample != 0: the greedy next
 * token of every entry's last row is kept on the device as the slot's current token (see decode and read).
 * Synchronizes when logits are wanted.  MLLMB200_TOO_LARGE: more than max_rows rows, or a slot beyond max_ctx. */
MLLMB200_API int mllmb200_lm_step(void* handle, int entries, const int* slots, const int* counts, const int* tokens,
                                  int n_want, const int* want, float* logits_out, int sample);

/* `steps` greedy steps for `count` slots together, each feeding the slot's current token; the last call on every slot
 * must have been a sampling step or a decode.  One CUDA graph replay per step. */
MLLMB200_API int mllmb200_lm_decode(void* handle, int count, const int* slots, int steps);

/* Gives a slot back: its next token is position 0 of a new sequence. */
MLLMB200_API int mllmb200_lm_free_slot(void* handle, int slot);

/* Synchronizes; history[first, first + count) of a slot (entry p = the token sampled after position p) and the number
 * of tokens it holds, to host memory; NULLs are skipped. */
MLLMB200_API int mllmb200_lm_read(void* handle, int slot, int first, int count, int* tokens_out, int* length_out);

/* Inspection: keep the residual stream after every layer of the following steps (on != 0), and read the rows of the
 * last step after `layer` (fp32 [rows, width], host). */
MLLMB200_API int mllmb200_lm_keep_residual(void* handle, int on);
MLLMB200_API int mllmb200_lm_read_residual(void* handle, int layer, int rows, float* out);

/* Bytes of per-sequence state in all slots, and kernels launched so far by steps (graph replays counted). */
MLLMB200_API int mllmb200_lm_stats(void* handle, size_t* state_bytes, long long* launches);

MLLMB200_API int mllmb200_lm_synchronize(void* handle);
MLLMB200_API void* mllmb200_lm_stream(void* handle);
MLLMB200_API const char* mllmb200_lm_last_error(void* handle);
MLLMB200_API int mllmb200_lm_check_device_status(void* handle);

/* Host only: the distance buckets of a bias table, out[n] for n in [0, count). */
MLLMB200_API int mllmb200_lm_distance_buckets(int bias_rows, int bias_max, int count, int* out);

#ifdef __cplusplus
}
#endif
#endif /* MLLMB200_LM_H_ */
