/*
 * skainet_cuda_fomalix.h — the Fomalix design of the decoder runtime (skainet_cuda_llama.h): BF16 weights, a configurable order
 * of three mixers (chunked attention with a sink, the gated delta rule, Mamba-2), norms before and after every sublayer, a gated
 * feed-forward where a layer has one, and a span of layers that runs several times with the same weights. Created and loaded
 * here, run through the skainet_cuda_llama_* entries that take any model handle. The reference has no counterpart.
 */
#ifndef SKAINET_CUDA_FOMALIX_H
#define SKAINET_CUDA_FOMALIX_H

#include "skainet_cuda_llama.h"

#ifdef __cplusplus
extern "C" {
#endif

#define SKAINET_FX_ATTENTION 0
#define SKAINET_FX_DELTA     1
#define SKAINET_FX_MAMBA2    2

typedef struct {
    int32_t type;             /* SKAINET_FX_* */
    int32_t heads;            /* query heads of attention, value heads of the recurrences */
    int32_t kv_heads;         /* key/value heads of attention; query/key heads of the delta rule; groups of Mamba-2 */
    int32_t dim;              /* query/key size; state size of Mamba-2 */
    int32_t vdim;
    int32_t conv;             /* taps of the short convolution (recurrences) */
    int32_t norm_groups;      /* Mamba-2 */
    int32_t chunk;            /* attention: a position sees the keys of its own chunk of this many positions; 0: every earlier key */
    float scale;              /* attention: factor of the scores */
    int32_t ff;               /* inner size of the feed-forward, 0: none */
} skainet_fomalix_layer;

typedef struct {
    int32_t n_layers, width, vocab;
    float eps, embed_scale;
    int32_t loop_start, loop_stop, loop_times;   /* the span [start, stop) of layers is gone through `times` times; 1: once, as the others */
    int32_t max_seq, max_batch;
    int32_t prefill_rows;     /* rows of one prompt pass; 0: the library's choice */
    int32_t act_f32;          /* 0: bf16 activations and cache, 32-bit accumulation and state; 1: everything in 32-bit */
} skainet_fomalix_config;

/* Matrices, BF16 [out, in] */
#define SKAINET_FX_EMBED   0
#define SKAINET_FX_HEAD    1
#define SKAINET_FX_Q       2   /* attention [heads * dim, width]; delta rule [kv_heads * dim, width]     */
#define SKAINET_FX_K       3   /* [kv_heads * dim, width]                                                 */
#define SKAINET_FX_V       4   /* attention [kv_heads * vdim, width]; delta rule [heads * vdim, width]   */
#define SKAINET_FX_B       5   /* delta rule [heads, width]                                               */
#define SKAINET_FX_A       6   /* delta rule [heads, width]                                               */
#define SKAINET_FX_G       7   /* delta rule [heads * vdim, width]                                        */
#define SKAINET_FX_IN      8   /* Mamba-2 [2 heads * vdim + 2 kv_heads * dim + heads, width]             */
#define SKAINET_FX_O       9   /* [width, heads * vdim]                                                   */
#define SKAINET_FX_GATE    10  /* [ff, width] */
#define SKAINET_FX_UP      11
#define SKAINET_FX_DOWN    12  /* [width, ff] */
/* Vectors, host floats */
#define SKAINET_FX_NORM1      0    /* width: before the mixer          */
#define SKAINET_FX_NORM1B     1    /* width: after it                  */
#define SKAINET_FX_NORM2      2    /* width: around the feed-forward   */
#define SKAINET_FX_NORM2B     3
#define SKAINET_FX_Q_BIAS     4    /* attention */
#define SKAINET_FX_K_BIAS     5
#define SKAINET_FX_V_BIAS     6
#define SKAINET_FX_SINK       7    /* heads */
#define SKAINET_FX_Q_CONV     8    /* delta rule, [channels][taps] */
#define SKAINET_FX_K_CONV     9
#define SKAINET_FX_V_CONV     10
#define SKAINET_FX_CONV       11   /* Mamba-2, [heads * vdim + 2 kv_heads * dim][taps] */
#define SKAINET_FX_CONV_BIAS  12
#define SKAINET_FX_A_LOG      13   /* recurrences, heads */
#define SKAINET_FX_DT_BIAS    14   /* heads */
#define SKAINET_FX_D          15   /* Mamba-2, heads */
#define SKAINET_FX_MIX_NORM   16   /* delta rule vdim; Mamba-2 heads * vdim */
#define SKAINET_FX_FINAL_NORM 17   /* width (layer ignored) */

SKAINET_CUDA_API int32_t skainet_cuda_fomalix_create(const skainet_fomalix_config* cfg, const skainet_fomalix_layer* layers, skainet_model_t* out);
/* Copies a resident BF16 weight into the model (the weight stays the caller's). layer is ignored for EMBED and HEAD. */
SKAINET_CUDA_API int32_t skainet_cuda_fomalix_set_weight(skainet_model_t m, int32_t layer, int32_t which, skainet_weight_t w);
SKAINET_CUDA_API int32_t skainet_cuda_fomalix_set_vector(skainet_model_t m, int32_t layer, int32_t which, const float* values_host, int32_t n);
/* Random weights of the configured shape: matrices std * N(0,1), gains 1, biases, sinks and skips 0, convolutions that pass the
 * current token, slow decays. */
SKAINET_CUDA_API int32_t skainet_cuda_fomalix_synth(skainet_model_t m, uint64_t seed, float std);

#ifdef __cplusplus
}
#endif
#endif /* SKAINET_CUDA_FOMALIX_H */
