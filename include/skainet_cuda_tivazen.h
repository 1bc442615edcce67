/*
 * skainet_cuda_tivazen.h — the Tivazen design of the decoder runtime (skainet_cuda_llama.h): BF16 weights, windowed latent
 * attention whose cache several layers may share, gated or routed feed-forward, one-number RMS norms on the sublayer
 * outputs, and a weighted sum over all earlier layers' results after every layer. Created and loaded here, run through the
 * skainet_cuda_llama_* entries that take any model handle. The reference has no counterpart.
 */
#ifndef SKAINET_CUDA_TIVAZEN_H
#define SKAINET_CUDA_TIVAZEN_H

#include "skainet_cuda_llama.h"

#ifdef __cplusplus
extern "C" {
#endif

#define SKAINET_TV_MLP_NONE  0
#define SKAINET_TV_MLP_DENSE 1
#define SKAINET_TV_MLP_MOE   2

typedef struct {
    /* latent attention */
    int32_t heads, dim, rot_dim, vdim, kv_rank;
    int32_t kv_from;          /* -1: own latent and cache; j: those of layer j, an earlier layer that has its own */
    int32_t window;           /* keys a position sees, itself included */
    float scale;              /* factor of the scores */
    double rope_base;
    /* feed-forward */
    int32_t mlp, ff;          /* SKAINET_TV_MLP_*; inner size (of one expert when routed) */
    int32_t experts, top;     /* routed only */
} skainet_tivazen_layer;

typedef struct {
    int32_t n_layers, width, vocab;
    float eps;
    int32_t max_seq, max_batch;
    int32_t prefill_rows;     /* rows of one prompt pass; 0: the library's choice */
    int32_t act_f32;          /* 0: bf16 activations and cache, 32-bit accumulation; 1: everything in 32-bit */
} skainet_tivazen_config;

/* Matrices, BF16 [out, in] */
#define SKAINET_TV_EMBED   0
#define SKAINET_TV_HEAD    1
#define SKAINET_TV_Q       2   /* [heads * (dim + rot_dim), width], per head [dim | rot_dim]        */
#define SKAINET_TV_DKV     3   /* [kv_rank + rot_dim, width]; layers with their own cache           */
#define SKAINET_TV_UK      4   /* [heads * dim, kv_rank]                                            */
#define SKAINET_TV_UV      5   /* [heads * vdim, kv_rank]                                           */
#define SKAINET_TV_G       6   /* [heads, width]                                                    */
#define SKAINET_TV_O       7   /* [width, heads * vdim]                                             */
#define SKAINET_TV_ROUTER  8   /* [experts, width]                                                  */
#define SKAINET_TV_GATE    9   /* [ff, width], one per expert when routed                           */
#define SKAINET_TV_UP      10
#define SKAINET_TV_DOWN    11  /* [width, ff]                                                       */
/* Vectors, host floats */
#define SKAINET_TV_NORM1       0   /* 1 */
#define SKAINET_TV_NORM2       1   /* 1; layers with a feed-forward */
#define SKAINET_TV_DKV_NORM    2   /* kv_rank; layers with their own cache */
#define SKAINET_TV_DEPTH       3   /* layer + 2 */
#define SKAINET_TV_FINAL_NORM  4   /* 1 (layer ignored) */

SKAINET_CUDA_API int32_t skainet_cuda_tivazen_create(const skainet_tivazen_config* cfg, const skainet_tivazen_layer* layers, skainet_model_t* out);
/* Copies a resident BF16 weight into the model (the weight stays the caller's). layer is ignored for EMBED and HEAD, expert
 * for everything but GATE, UP and DOWN of a routed layer. */
SKAINET_CUDA_API int32_t skainet_cuda_tivazen_set_weight(skainet_model_t m, int32_t layer, int32_t which, int32_t expert, skainet_weight_t w);
SKAINET_CUDA_API int32_t skainet_cuda_tivazen_set_vector(skainet_model_t m, int32_t layer, int32_t which, const float* values_host, int32_t n);
/* Random weights of the configured shape: matrices std * N(0,1), gains 1, depth weights 1 for the layer's own result and 1/8
 * for the others. */
SKAINET_CUDA_API int32_t skainet_cuda_tivazen_synth(skainet_model_t m, uint64_t seed, float std);

#ifdef __cplusplus
}
#endif
#endif /* SKAINET_CUDA_TIVAZEN_H */
