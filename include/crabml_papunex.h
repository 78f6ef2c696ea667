/*
 * crabml_papunex.h -- creation of the host driver of the Papunex decoder family (crabml_b200/csrc/host/papunex_runner.cpp); the runner it
 * returns is served through crabml_seqrunner.h (slots, step, greedy generation) like every multi-sequence runner.
 *
 * The stack: x = embed[token] (the table arrives already multiplied by the embedding scale).  The sublayers read the residual stream itself
 * and only their OUTPUT is normed: x += norm1(mixer(x)) ; x += norm2(ff(x))  (RMS norms with a weight per column).
 * Mixers: latent attention -- causal, softmax with a per-head sink, the heads' outputs gated by sigmoid(W_g x) element by element; a layer
 * may read another layer's cache of latent rows (kv_from) with up-projections of its own -- and the state-space mixer (Mamba-2).
 * Feed-forward: plain units with the squared relu, dense, routed (softmax scores over all experts, renormalised and scaled weights) with an
 * optional shared expert weighted by one sigmoid gate per token, or none.
 * Output: RMS norm, head, logits capped by softcap * tanh(logits / softcap).
 */
#ifndef CRABML_PAPUNEX_H
#define CRABML_PAPUNEX_H

#include "crabml_seqops.h"
#include "crabml_seqrunner.h"

#ifdef __cplusplus
extern "C" {
#endif

#define CPR_MIXER_LATENT 0
#define CPR_MIXER_STATE_SPACE 1

#define CPR_FF_NONE 0
#define CPR_FF_DENSE 1
#define CPR_FF_ROUTED 2

typedef struct cpr_layer_config {
    int32_t mixer;                  /* CPR_MIXER_* */
    /* latent attention */
    int32_t heads, dim, rot_dim, vdim, kv_rank;
    int32_t kv_from;                /* index of the EARLIER layer whose cache this layer reads; -1: its own */
    float scale, rot_mag;           /* score scale; factor on cos and sin */
    /* state space */
    int32_t s_heads, s_vdim, s_state, s_groups, s_conv, s_norm_groups;
    /* feed-forward */
    int32_t ff_kind;                /* CPR_FF_* */
    int32_t ff;                     /* dense: hidden width; routed: an expert's hidden width */
    int32_t experts, top;
    int32_t shared;                 /* routed: pieces of width ff that the shared expert is cut into (the last one zero-padded); 0: none */
    float route_scale;              /* routed: factor on the renormalised weights */
} cpr_layer_config;

typedef struct cpr_config {
    int32_t n_layers, width, vocab;
    float norm_eps;
    float softcap;                  /* cap of the logits; <= 0: none */
    int32_t chunk;                  /* longest run of tokens one pass takes.  <= 0: 256 */
    int32_t max_seq;                /* rows of an attention layer's cache.  <= 0: 4096 */
} cpr_config;

/* every pointer is a tensor uploaded by the caller; unused ones are NULL.  Matrices of dense products: F32 or BF16; uk_t, uv_f32, conv,
 * router, shared_gate and everything else: F32. */
typedef struct cpr_layer_weights {
    cc_buf *norm1, *norm2;                          /* [width] each; norm2: layers with a feed-forward */
    /* latent attention.  h_stack: everything that multiplies the layer's input, stacked one under the other so that it is ONE product:
     * mix.q [heads * (dim + rot_dim), width], mix.g [heads * vdim, width], then, in a layer with a cache of its own, mix.dkv [kv_rank +
     * rot_dim, width] */
    cc_buf *h_stack, *dkv_norm;                     /* dkv_norm: [kv_rank], layers with a cache of their own */
    cc_buf *uk, *uv, *uk_t, *uv_f32;                /* as in crabml_meresun.h */
    cc_buf *sink, *rot_freq, *o;                    /* [heads] or NULL; [P], 2 P <= rot_dim, or NULL; [width, heads * vdim] */
    /* state space */
    cc_buf *in, *conv, *conv_bias, *dt_bias, *a_log, *d_skip, *s_norm, *s_o;
    /* dense: [ff, width], [width, ff].  routed: expert-major stacks [(experts + shared) * ff, width], [(experts + shared) * width, ff], the
     * shared expert's pieces last */
    cc_buf *up, *down;
    cc_buf *router, *shared_gate;                   /* routed: [experts, width]; [width] or NULL */
} cpr_layer_weights;

CC_API int cpr_runner_create(cc_device* dev, const cpr_config* conf, const cpr_layer_config* layers, const cpr_layer_weights* weights, cc_buf* embed,
                             cc_buf* final_norm, cc_buf* head, csr_runner** out);

#ifdef __cplusplus
}
#endif
#endif
