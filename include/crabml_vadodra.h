/*
 * crabml_vadodra.h -- creation of the host driver of the Vadodra decoder family (crabml_b200/csrc/host/vadodra_runner.cpp); the runner it
 * returns is served through crabml_seqrunner.h (slots, step, greedy generation) like every multi-sequence runner.
 *
 * The stack: x = embed[token] (the table arrives already multiplied by the embedding scale).  Every layer takes ONE layer norm (weight, no
 * bias) of the 32-bit residual stream and hands it to its mixer and its feed-forward side by side: x += mixer(LN(x)) + ff(LN(x)).
 * Mixers:
 *   CVD_MIXER_WINDOW  grouped key / value heads, a sliding window, softmax.  Queries and keys are RMS-normalised per head (a weight vector all
 *                     heads share), then their leading column pairs (2i, 2i + 1) turn with the position; the values are the keys as
 *                     projected, before norm and rotation.
 *   CVD_MIXER_LATENT  causal latent attention (one cached row [c | r] per position) whose rotated part pairs the columns (i, i + rot_dim / 2),
 *                     every head's output times a sigmoid of one number per head.  A layer may read an earlier layer's cache (kv_from) through
 *                     up-projections of its own.
 * Feed-forward: W_down of gated units act(min(g, limit)) * (clamp(u, -limit, limit) + shift), or none.
 * Output: the final layer norm, the head (tied: the embedding table without its scale).
 */
#ifndef CRABML_VADODRA_H
#define CRABML_VADODRA_H

#include "crabml_seqops.h"
#include "crabml_seqrunner.h"

#ifdef __cplusplus
extern "C" {
#endif

#define CVD_MIXER_WINDOW 0
#define CVD_MIXER_LATENT 1

typedef struct cvd_layer_config {
    int32_t mixer;                  /* CVD_MIXER_* */
    int32_t heads, kv_heads, dim, vdim;   /* window: vdim = dim, the values are keys; latent: dim = the unrotated part, kv_heads is not used */
    int32_t window;                 /* window: position i sees j with 0 <= i - j < window; <= 0: every j <= i */
    int32_t rot_dim, kv_rank;       /* latent */
    int32_t kv_from;                /* latent: index of the EARLIER layer whose cache this layer reads; -1: its own */
    float scale, rot_mag;           /* score scale; factor on cos and sin */
    int32_t ff;                     /* hidden width of the feed-forward; 0: the layer is its mixer only */
    cc_glu_params glu;              /* its gated unit */
} cvd_layer_config;

typedef struct cvd_config {
    int32_t n_layers, width, vocab;
    float norm_eps;
    int32_t chunk;                  /* longest run of tokens one pass takes.  <= 0: 256 */
    int32_t max_seq;                /* rows of a cache that must hold the whole sequence.  <= 0: 4096 */
} cvd_config;

/* every pointer is a tensor uploaded by the caller; unused ones are NULL.  Matrices of dense products: F32 or BF16; uk_t, uv_f32 and everything
 * else: F32. */
typedef struct cvd_layer_weights {
    cc_buf* norm;                                   /* [width] */
    /* everything that multiplies the normed input, stacked one under the other so that it is ONE product.
     * window: mix.q [heads * dim, width], mix.k [kv_heads * dim, width]; latent: mix.q [heads * (dim + rot_dim), width], mix.g [heads, width]
     * and, in a layer with a cache of its own, mix.dkv [kv_rank + rot_dim, width]; then, with a feed-forward, mlp.gate and mlp.up [ff, width] */
    cc_buf* h_stack;
    cc_buf* o_stack;                                /* mix.o [width, heads * vdim] and mlp.down [width, ff] side by side: ONE product again */
    cc_buf *q_norm, *k_norm;                        /* window: [dim] each */
    cc_buf* rot_freq;                               /* [P], 2 P <= dim (window) or rot_dim (latent), or NULL */
    cc_buf *dkv_norm, *uk, *uv, *uk_t, *uv_f32;     /* latent, as in crabml_meresun.h; dkv_norm: layers with a cache of their own */
} cvd_layer_weights;

CC_API int cvd_runner_create(cc_device* dev, const cvd_config* conf, const cvd_layer_config* layers, const cvd_layer_weights* weights, cc_buf* embed,
                             cc_buf* final_norm, cc_buf* head, csr_runner** out);

#ifdef __cplusplus
}
#endif
#endif
