/*
 * C ABI of libb200hybrid.so: forward passes of decoder designs given as a list of layers (each with its own token
 * mixer and feed-forward), bf16 weights, bf16 or fp32 activations.  Conventions of b200_eagle.h: plain pointers and
 * sizes, device pointers unless stated otherwise, asynchronous on `stream`, no allocation, no printing; 0 on
 * success, a negative B200_E* code otherwise.
 *
 * A pass is a sequence of kernel launches issued by b200_hybrid_forward from host-side tables (structs below live in
 * HOST memory; the pointers inside them are device pointers).  Every data-dependent quantity (tokens, positions,
 * masks, committed length) is read from device memory, so a pass can be captured into a CUDA graph.
 */
#ifndef B200_HYBRID_H
#define B200_HYBRID_H

#include <stddef.h>
#include <stdint.h>

#include "b200_eagle.h"

#ifdef __cplusplus
extern "C" {
#endif

#define B200_ACT_BF16 0 /* activations and cache bf16, tensor-core products with fp32 accumulation */
#define B200_ACT_F32 1  /* everything fp32, plain fp32 multiply-adds                               */

#define B200_MIXER_ATTENTION 0  /* softmax attention, 1 or 2 maps per head (2: differential), window + kept first keys */
#define B200_MIXER_RECURRENCE 1 /* gated linear recurrence, S += (1-f) (v - S) per channel row, o = S^T q              */
#define B200_MIXER_DELTA 2      /* gated delta rule with a decay per key channel, convolutions on q, k, v              */
#define B200_MIXER_LATENT 3     /* softmax attention over a shared low-rank latent and one rotated key part            */

#define B200_FF_POLYNORM 0 /* W_down polynorm(W_up h)                                                                  */
#define B200_FF_GATED 1    /* W_down (gelu_tanh(W_gate h + b) * (W_up h + b)) + b                                      */
#define B200_FF_EXPERTS 2  /* sum over the chosen experts of W_down (swish_alpha(min(g, l)) * (clamp(u, l) + shift))   */

#define B200_HYBRID_PENDING 64 /* rows of a request whose inputs are kept until they are committed */
#define B200_HYBRID_MAX_TAPS 8
#define B200_HYBRID_MAX_EXPERTS 512
#define B200_HYBRID_MAX_TOP 16

/* y = x W^T; W bf16 [n rounded up to 128][pitch], pitch = k rounded up to 64, rows past n and columns past k zero.
 * groups > 1: a stack of such matrices, each over pitch columns of x of its own (group g reads x columns g*pitch.. and gives
 * output columns g*n ..). */
typedef struct b200_linear {
    const void* w;
    int n, k, pitch, groups;
} b200_linear;

typedef struct b200_hybrid_layer {
    int mixer, taps;                    /* taps of the input convolution (>= 1)                                      */
    int heads, kv_heads, dim, vdim;     /* recurrence: kv_heads = heads                                              */
    int maps;                           /* attention maps per head                                                   */
    int window, keep_first;             /* position i sees j <= i with i - j < window or j < keep_first              */
    int ff;                             /* feed-forward width, 0: the layer has none                                 */
    float scale, lambda, out_scale;     /* score scale; maps = 2: weight of map 2, factor after the head's norm      */
    float act[4];                       /* polynorm: a N(z) + b N(z^2) + c N(z^3) + e; experts: limit, alpha, shift  */
    int ff_kind;
    const float* norm1;                 /* [width] multiplicative weights (1 + w already added where w is zero-centred) */
    const float* norm2;
    const float* conv;                  /* [taps][width]                                                             */
    const float* gate_bias;             /* recurrence: bias and lower bound of the forget gate [heads * dim]         */
    const float* gate_lower;
    const float* head_norm;             /* recurrence: [vdim]                                                        */
    b200_linear in;                     /* rows q | k | v | gate (attention), q | f | v (recurrence),
                                           q | k | v | beta | low-rank inputs (delta), unrotated queries | rotated query
                                           parts | latent | rotated key part (latent)                                */
    b200_linear out, up, down;          /* gated kinds: rows of `up` alternate gate, up; experts: groups = experts   */
    /* delta */
    int conv_taps;                      /* taps of the convolutions on q, k, v                                       */
    int low_rank;                       /* columns of the low-rank inputs of decay and output gate together          */
    const float* mix_conv;              /* [conv_taps][2*kv_heads*dim + heads*vdim], last tap: the current token     */
    const float* decay_bias;            /* [heads*dim]                                                               */
    const float* decay_rate;            /* [heads*dim]: g = exp(-rate * softplus(z + bias)); kept as g - 1            */
    b200_linear low;                    /* rows decay | output gate over the low-rank inputs                         */
    /* latent */
    int kv_rank, rot_dim;
    float rot_mag;                      /* factor on cos and sin                                                     */
    int reserved;
    const float* rot_freq;              /* [rot_dim / 2] angle per position                                          */
    const float* latent_norm;           /* [kv_rank]                                                                 */
    b200_linear absorb;                 /* groups = heads: unrotated query -> its form over the latent               */
    b200_linear value;                  /* groups = heads: latent -> value                                           */
    b200_linear expand;                 /* rows unrotated keys | values of all heads over the latent                 */
    /* gated feed-forwards and experts */
    int experts, top;
    const float* up_bias;               /* [2*ff], alternating like the rows of `up`                                 */
    const float* down_bias;             /* [width]                                                                   */
    b200_linear router;
} b200_hybrid_layer;

/* One execution of a layer in a pass (a repeated layer has one per repetition), with the place of its cache / state
 * inside a request's cache (byte offsets) and of its pending rows inside the model's pending buffer. */
typedef struct b200_hybrid_run {
    int layer;
    int inject;                         /* the embedding output is added to the residual stream after this run       */
    long long conv_off;                 /* fp32 [taps - 1][width], oldest first                                      */
    long long k_off, v_off;             /* attention: [kv_heads][rows][maps * dim16], [kv_heads][rows][vdim16];
                                           latent: k_off [rows][kv_rank16 + rot_dim16]                               */
    long long state_off;                /* recurrence: fp32 [heads][dim][vdim], delta: fp32 [heads][vdim][dim]       */
    long long pend_h, pend_g, pend_v;   /* fp32 [64][width], fp32 [64][heads*dim], activations [64][heads*vdim]      */
    long long mix_off;                  /* delta: activations [conv_taps - 1][channels], oldest first                */
    long long pend_c, pend_k, pend_b;   /* delta: activations [64][channels], fp32 [64][kv_heads*dim], fp32 [64][heads] */
} b200_hybrid_run;

typedef struct b200_hybrid_model {
    int act_type, width, vocab, n_layers, n_runs, max_rows;
    int injects;                        /* some run injects: the embedding output is kept during the pass            */
    int conv_max_taps;
    float eps, residual_mult, softcap;  /* softcap <= 0: none                                                        */
    int norm_out;                       /* 0: sublayers read the normed stream; 1: they read the stream, their outputs are
                                           normed before they are added (residual_mult unused)                       */
    const void* embed;                  /* bf16 [vocab][width]                                                       */
    const float* final_norm;
    const b200_hybrid_layer* layers;    /* HOST                                                                      */
    const b200_hybrid_run* runs;        /* HOST                                                                      */
    const b200_hybrid_layer* dev_layers;/* device copies of the same tables (commit kernel)                          */
    const b200_hybrid_run* dev_runs;
    b200_linear head;
    /* activation buffers for max_rows rows; pitches are the widths rounded up to 64 where a product reads them     */
    float* x;                           /* residual stream [max_rows][width]                                         */
    float* emb;                         /* embedding output, same shape                                              */
    void* hb;                           /* product input [max_rows][width64]                                         */
    void* qb;                           /* [max_rows][heads * maps * dim16], recurrence: heads * dim                 */
    void* gb;                           /* output gate [max_rows][heads * vdim]                                      */
    void* vb;                           /* recurrence values [max_rows][heads * vdim]                                */
    float* gf;                          /* 1 - forget gate [max_rows][heads * dim]                                   */
    float* o32;                         /* recurrence output [max_rows][heads * vdim]                                */
    void* ab;                           /* mixer output [max_rows][heads * vdim rounded up to 64]                    */
    void* zb;                           /* feed-forward [max_rows][ff64], before and after the activation            */
    void* zab;                          /* (experts: max_rows * top rows)                                            */
    float* y;                           /* sublayer output before its norm / expert outputs [max_rows * top][width]  */
    void* cb;                           /* delta: convolution inputs [max_rows][channels]                            */
    void* lowb;                         /* delta: low-rank inputs [max_rows][low_rank64]                             */
    float* q32;                         /* delta: unit queries and keys [max_rows][kv_heads*dim]                     */
    float* k32;
    float* beta;                        /* delta: [max_rows][heads]                                                  */
    float* chunk;                       /* delta: floats of b200_hybrid_chunk_floats                                 */
    float* lat32;                       /* latent: rotated query parts | latent | rotated key part, before norm and rotation */
    void* qn;                           /* latent: unrotated queries [max_rows][heads][dim64]                        */
    void* ob;                           /* latent: attention output over the latent [max_rows][heads][kv_rank64]     */
    void* kx;                           /* latent: keys and values of all heads for `x_rows` cache rows, prompts     */
    void* vx;
    float* zr;                          /* experts: router logits [max_rows][experts]                                */
    int* route;                         /* experts: see b200_hybrid_route_ints                                       */
    void* xg;                           /* experts: gathered inputs [max_rows * top][width64]                        */
    int x_rows, route_top, route_experts, reserved;
    void* pending;
    float* attn_part;                   /* attention partials                                                        */
    size_t attn_part_bytes;
    int* error;                         /* error word (0: none)                                                      */
} b200_hybrid_model;

typedef struct b200_hybrid_pass {
    int M;                              /* token rows of the pass                                                    */
    int tree;                           /* 0: the rows continue the sequence and are committed by the pass; 1: rows
                                           are tail rows write_off .. write_off+M-1 after `prefix` committed ones,
                                           row m sees tail row j iff bit j of mask[m] is set, nothing is committed    */
    int write_off, tail, rows_out, cache_rows;
    int max_keys;                       /* upper bound of prefix + tail (or prefix + M) this launch must serve        */
    int reserved;
    const int* tokens;                  /* [M]                                                                       */
    const int* pos;                     /* [M] positions                                                             */
    const unsigned long long* mask;     /* [M], tree only                                                            */
    const int* prefix;                  /* [1] committed length before the pass                                      */
    const int* out_rows;                /* rows whose logits are wanted [rows_out]; null: row_index[0] + i           */
    const int* row_index;               /* null: 0                                                                   */
    int* tail_pos;                      /* [64] positions of the tail rows, tree only                                */
    void* cache;
    float* logits;                      /* [rows_out][vocab]                                                         */
    void* logits16;                     /* fp16 copy or null                                                         */
    float* dump;                        /* null, or [n_runs][M][width]: residual stream after every run              */
} b200_hybrid_pass;

/* Bytes of attention partials a pass of `rows` tree rows (or fp32 / short chain rows) needs at most. */
size_t b200_hybrid_attention_workspace_bytes(const b200_hybrid_model* model, int rows);

/* Floats of `chunk`: vectors and coefficients of a delta layer's prompt rows, 8 tokens at a time. */
size_t b200_hybrid_chunk_floats(int max_rows, int heads, int dim);

/* Ints of `route`: expert and position of every (row, choice), the choices' scores, first place of every expert. */
size_t b200_hybrid_route_ints(int max_rows, int top, int experts);

int b200_hybrid_forward(const b200_hybrid_model* model, const b200_hybrid_pass* pass, void* stream);

/* Commits tail rows of the last tree pass to `cache`: n = count[0] + 1 rows, tail row 0 and rows[1 .. count]
 * (rows null: 0 .. count; a negative entry counts from `tree_rows`): convolution and recurrent states advance over
 * them; with compact != 0 their K/V rows move to prefix[0] .. prefix[0] + n - 1. */
int b200_hybrid_commit(const b200_hybrid_model* model, void* cache, int cache_rows, const int* count, const int* rows,
                       int tree_rows, const int* prefix, int compact, void* stream);

/* Single operators, as the passes use them (tests, tools). act_type selects the type of x / y. */
int b200_hybrid_linear(const b200_hybrid_model* model, const b200_linear* lin, const void* x, int x_pitch, int x_rows,
                       float* y, int y_pitch, int M, void* stream);

int b200_hybrid_version(void);
int b200_hybrid_last_cuda_error(void);
void b200_hybrid_set_pdl(int enabled);

#ifdef __cplusplus
}
#endif
#endif
