/*
 * tllm_b200_mixed.h -- decoders whose layers are a list of different token mixers (latent
 * attention, selective scan, real-gated linear recurrence, grouped-query attention, linear
 * attention, gated delta rule, or two of the last three side by side) with dense or routed
 * feed-forwards and BF16 weights.
 *
 * No counterpart in the reference engine, whose Transformer (src/transformer.cpp) has one kind
 * of layer.  A decoder made here is driven by the same entry points as every other model of
 * the library (tllm_b200_layer.h: tllm_b200_decoder_forward, _forward_seq, _forward_batch,
 * _generate, _reset, _destroy); logits are FP32.
 *
 * A sequence's state is a cache of one row per position for attention (with a chunk mask: a ring
 * of as many rows as a chunk and a pass need) and a fixed-size recurrent state otherwise.  A call with start_pos 0 starts a new sequence in its
 * slot; with recurrent layers, every other call must continue where the slot's sequence ended
 * (TLLM_ERR_SHAPE otherwise), and so it must with a ring of cache rows.
 */
#ifndef TLLM_B200_MIXED_H
#define TLLM_B200_MIXED_H

#include "tllm_b200_layer.h"

#ifdef __cplusplus
extern "C" {
#endif

enum {
    TLLM_MIXER_LATENT_ATTENTION = 1,
    TLLM_MIXER_SELECTIVE_SCAN = 2,   /* Mamba */
    TLLM_MIXER_GATED_RECURRENCE = 3, /* Griffin's RG-LRU block */
    TLLM_MIXER_ATTENTION = 4,        /* grouped-query softmax attention */
    TLLM_MIXER_LINEAR_ATTENTION = 5, /* a decaying sum of (key, value) pairs per head, read by the query */
    TLLM_MIXER_DELTA_RULE = 6        /* a decaying memory per head in which a key's value is replaced, not added */
};
enum { TLLM_ACT_NONE = 0, TLLM_ACT_GELU_TANH = 1, TLLM_ACT_SILU = 2, TLLM_ACT_SIGMOID = 4 };

/* Tensors of a layer: device pointers to BF16 data, row-major [out, in]; copied (and padded)
 * at creation.  Unused entries are NULL. */
enum {
    TLLM_T_NORM1 = 0,   /* [width], before the mixer (norm_after_sum: of the sum behind it) */
    TLLM_T_NORM1B,      /* [width], after the mixer; NULL: plain residual add */
    TLLM_T_NORM2,       /* [width], before the feed-forward (norm_after_sum: of the sum behind it) */
    TLLM_T_NORM2B,      /* [width], after it; NULL: plain residual add */
    TLLM_T_GATE,        /* [ff, width], or [experts, ff, width] */
    TLLM_T_UP,          /* [ff, width], or [experts, ff, width] */
    TLLM_T_DOWN,        /* [width, ff], or [experts, width, ff] */
    TLLM_T_OUT,         /* [width, mixer output] */
    /* latent attention */
    TLLM_T_Q,           /* [heads * (dim + rot_dim), width], per head unrotated then rotated; attention and
                           linear attention: [heads * dim, width]; delta rule: [kv_heads * dim, width] */
    TLLM_T_KV_DOWN,     /* [kv_rank + rot_dim, width]: latent, then the shared rotated key part */
    TLLM_T_KV_NORM,     /* [kv_rank] */
    TLLM_T_K_UP,        /* [heads * dim, kv_rank] */
    TLLM_T_V_UP,        /* [heads * vdim, kv_rank] */
    TLLM_T_SINK,        /* [heads], NULL: no sink */
    TLLM_T_HEAD_GATE,   /* [heads, width], NULL: no output gate */
    /* selective scan and gated recurrence */
    TLLM_T_IN,          /* scan: [2 * inner, width] (x, then z); recurrence: [channels, width] of the recurrent branch */
    TLLM_T_IN_BIAS,     /* recurrence: [channels] */
    TLLM_T_CONV,        /* [channels, taps] */
    TLLM_T_CONV_BIAS,   /* [channels] */
    TLLM_T_X,           /* scan: [dt_rank + 2 * state, inner] (dt, B, C) */
    TLLM_T_DT,          /* scan: [inner, dt_rank] */
    TLLM_T_DT_BIAS,     /* scan: [inner] */
    TLLM_T_A_LOG,       /* scan: [inner, state] */
    TLLM_T_D,           /* scan: [inner] */
    TLLM_T_Y,           /* recurrence: [channels, width] of the gating branch */
    TLLM_T_Y_BIAS,      /* recurrence: [channels] */
    TLLM_T_RA,          /* recurrence: [blocks, channels / blocks, channels / blocks] */
    TLLM_T_RA_BIAS,     /* recurrence: [channels] */
    TLLM_T_RI,
    TLLM_T_RI_BIAS,
    TLLM_T_LAM,         /* recurrence: [channels] */
    /* attention, linear attention, delta rule */
    TLLM_T_K,           /* [kv_heads * dim, width] */
    TLLM_T_V,           /* attention: [kv_heads * vdim, width], else [heads * vdim, width] */
    TLLM_T_Q_NORM,      /* attention: [dim], NULL: no norm */
    TLLM_T_K_NORM,
    TLLM_T_Q_CONV,      /* delta rule: [kv_heads * dim, taps] */
    TLLM_T_K_CONV,
    TLLM_T_V_CONV,      /* delta rule: [heads * vdim, taps] */
    TLLM_T_STEP,        /* delta rule: [heads, width], before the sigmoid */
    TLLM_T_DECAY,       /* delta rule: [heads, width]; with TLLM_T_DT_BIAS and TLLM_T_A_LOG [heads] */
    TLLM_T_MIX_NORM,    /* of the output -- linear attention: [heads * vdim]; delta rule: [vdim], every head alone */
    TLLM_T_MIX_GATE,    /* linear attention, delta rule: [heads * vdim, width], multiplies the normed output */
    /* feed-forward */
    TLLM_T_ROUTER,      /* [experts, width] */
    TLLM_T_COUNT
};

typedef struct tllm_b200_mixed_layer {
    int type;                                        /* TLLM_MIXER_... */
    int heads, dim, rot_dim, rot_dims, vdim, kv_rank; /* latent attention; rot_dims of the rot_dim entries turn */
    float scale;
    double rot_base;
    int channels, taps;                              /* scan and recurrence */
    int state, dt_rank;                              /* scan */
    int blocks;                                      /* recurrence */
    float decay;                                     /* recurrence: c in log a = -c r softplus(lam) */
    int gate_act;                                    /* activation of the gating branch or the output gate */
    int ff, ff_act;                                  /* ff = 0: no feed-forward */
    int experts, top;                                /* experts > 0: mixture, `top` per token; ff is an expert's */
    int kv_heads;                                    /* attention, delta rule */
    int chunk;                                       /* attention: only positions of the same chunk; 0: all */
    int in_act;                                      /* linear attention: of q, k, v; delta rule: of the convolutions */
    float out_scale;                                 /* of the mixer's output (attention, linear attention, delta rule) */
    const float* head_decay;                         /* linear attention: host array [heads] */
    /* a second mixer of the three that reads the same input and is added (its own `beside`, feed-forward
     * and layer norms are ignored), or NULL */
    const struct tllm_b200_mixed_layer* beside;
    const void* t[TLLM_T_COUNT];
} tllm_b200_mixed_layer;

typedef struct tllm_b200_mixed_desc {
    int vocab_size, width, n_layers, max_seq_len;
    float norm_eps;
    /* layers loop_start .. loop_stop-1 run loop_times times in a row with the same weights, each
     * pass with its own cache or state; loop_inject: the embedding output is added to the
     * residual before the first layer of every pass but the first */
    int loop_start, loop_stop, loop_times, loop_inject;
    int norm_after_sum;      /* x = norm(residual_scale * x + sublayer(x)) instead of x + sublayer(norm(x)) */
    float residual_scale;
    float logit_softcap;     /* logits = cap * tanh(logits / cap); 0: none */
    const void* embedding;   /* BF16 [vocab, width] */
    const void* head;        /* BF16 [vocab, width], NULL: the embedding */
    const void* final_norm;  /* BF16 [width] */
    const tllm_b200_mixed_layer* layers; /* host array of n_layers */
} tllm_b200_mixed_desc;

#define TLLM_DECODER_FLOAT32 2 /* weights, activations and products in true 32-bit instead of BF16 */

/* max_batch (1..TLLM_DECODER_MAX_BATCH) sequences with their own state. */
int tllm_b200_mixed_decoder_create(const tllm_b200_mixed_desc* desc, int flags, int max_batch, void** out);

/* Layer runs of one pass (a looped layer counts once per pass). */
int tllm_b200_mixed_decoder_runs(void* decoder);

/* tllm_b200_decoder_forward_seq with the logits of chosen tokens: want_host (host array) lists
 * n_want places among the n_tokens, logits (device, float [n_want, vocab]) receives theirs in
 * that order.  taps: NULL, or device float [runs, n_tokens, width] for the residual stream
 * after every layer run.  n_want may be 0. */
int tllm_b200_decoder_forward_logits(void* decoder, int seq, const int* token_ids, int n_tokens, int start_pos,
                                     const int* want_host, int n_want, float* logits, float* taps, void* stream);

/* ---- stand-alone operators; `bf16` selects BF16 activations and weights, else FP32 ---------
 * Rows are n_seq sequences of seq_len tokens; sequence b uses slot b of the state.  Channel
 * counts, ranks and dimensions must be multiples of 8 (states of a scan: any). */

/* y = x . W^T (+ bias), x [rows, cols], w [n, cols], y float [rows, n]; glu: w holds n gate rows
 * then n up rows and y = act(gate) * up; y in the activation type then. */
int tllm_b200_dense_linear(int bf16, const void* x, const void* w, const float* bias, void* y, int rows, int n, int cols, int act,
                           int glu, void* stream);
/* state: activation type [n_seq][taps - 1][channels]; w float [channels, taps]; act: TLLM_ACT_... */
int tllm_b200_causal_conv(int bf16, const void* x, const float* w, const float* bias, void* state, void* y, int channels, int taps,
                          int act, int n_seq, int seq_len, int start_pos, void* stream);
/* x, z, y [rows, channels]; dt float [rows, channels]; bc [rows, 2 * ld]: B then C, ld = states
 * padded to a multiple of 8 with zeros; a2 float [channels, states] = A / ln 2; z may be NULL;
 * state float [n_seq][channels][states]. */
int tllm_b200_selective_scan(int bf16, const void* x, const float* dt, const void* bc, const void* z, const float* a2,
                             const float* d, float* state, void* y, int channels, int states, int n_seq, int seq_len,
                             int start_pos, void* stream);
/* gates float [rows, blocks, 2, channels / blocks]: r then i; soft_lam float [channels];
 * state float [n_seq][channels]; out = S * act(y). */
int tllm_b200_gated_scan(int bf16, const void* u, const float* gates, const float* soft_lam, const void* y, float* state, void* out,
                         int channels, int blocks, float decay, int act, int n_seq, int seq_len, int start_pos, void* stream);
/* q [rows, heads, rank + rot] (absorbed, rotated), cache [n_seq][max_seq][rank + rot], sink float
 * [heads] or NULL, o [rows, heads, rank]. */
int tllm_b200_latent_attention(int bf16, const void* q, const void* cache, const float* sink, void* o, int heads, int rank, int rot,
                               float scale, int max_seq, int n_seq, int seq_len, int start_pos, void* stream);
/* One sequence with expanded keys and values, BF16: q [seq_len, heads, dim + rot], kx [context,
 * heads, dim], vx [context, heads, vdim], cache rows hold the shared key part behind `rank`
 * entries; gate BF16 [seq_len, heads] (before the sigmoid) or NULL; o [seq_len, heads, vdim]. */
int tllm_b200_latent_attention_expanded(const void* q, const void* kx, const void* vx, const void* cache, const float* sink,
                                        const void* gate, void* o, int heads, int dim, int rot, int vdim, int rank, float scale,
                                        int max_seq, int seq_len, int start_pos, void* stream);

/* Norms, rotation, cache append and attention of a step (TLLM_MIXER_ATTENTION): proj [rows,
 * heads * dim + kv_heads * (dim + vdim)] = q, k, v (q is overwritten); norms float [dim] or NULL;
 * rope float [positions][rot_dims / 2][2] = cos, sin; kc [n_seq][cache_rows][kv_heads * dim], vc
 * alike; position p is cache row p % cache_rows, so cache_rows is at least chunk + seq_len, or all
 * positions; o [rows, heads * vdim]. */
int tllm_b200_grouped_attention(int bf16, void* proj, const float* q_norm, const float* k_norm, float eps, const float* rope, int rot_dims,
                                void* kc, void* vc, void* o, int heads, int kv_heads, int dim, int vdim, int chunk, int cache_rows, int max_seq,
                                float scale, float out_scale, int n_seq, int seq_len, int start_pos, void* stream);
/* Linear attention (delta = 0: decay float [heads], kv_heads = heads) or the gated delta rule
 * (delta = 1: a, b float [rows, heads], neg_a = -exp(A_log) and dt_bias float [heads]): q, k [rows,
 * kv_heads * dim], v [rows, heads * vdim] as one row q, k, v each; state float
 * [n_seq][heads][vdim][dim]; o float [rows, heads * vdim]. */
int tllm_b200_matrix_scan(int bf16, int delta, const void* qkv, const float* decay, const float* a, const float* b, const float* neg_a,
                          const float* dt_bias, float q_scale, float* state, float* o, int heads, int kv_heads, int dim, int vdim, int n_seq,
                          int seq_len, int start_pos, void* stream);
/* out = out_scale * o / rms(o) * w * act(gate): o float, gate and out [rows, groups * n], the norm
 * over each group of n; w float [n]. */
int tllm_b200_gated_norm(int bf16, const float* o, const float* w, const void* gate, void* out, int rows, int groups, int n, float eps,
                         float out_scale, int act, void* stream);
/* y float [rows, width] = sum over the `top` experts with the largest z (softmax over them) of
 * down (act(gate h) * up h); z float [rows, experts]; gate_up [experts][2 * ff, width], down
 * [experts][width, ff]. */
int tllm_b200_experts(int bf16, const void* h, const float* z, const void* gate_up, const void* down, float* y, int rows, int width, int ff,
                      int experts, int top, int act, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* TLLM_B200_MIXED_H */
