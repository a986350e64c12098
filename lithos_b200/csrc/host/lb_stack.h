/* Models described by a list of layers (bf16 weights, fp32 residual stream): what a design hands to the stack (lb_stack.c).
 * A design (lb_nufalorn.c) turns its config.json into this description and says which tensor feeds which part; every
 * mechanism takes its constants from here. */
#ifndef LB_STACK_H
#define LB_STACK_H
#include "lb_internal.h"
#include "lb_json.h"

enum { LB_MIX_ATTENTION = 0, LB_MIX_DECAY = 1, LB_MIX_LATENT = 2, LB_MIX_SSM = 3 };
enum { LB_FF_RELU_GLU = 0, LB_FF_RELU2 = 1, LB_FF_EXPERTS = 2 };

/* weight roles of a layer; a role without a name is absent */
enum {
    LB_T_NORM1, LB_T_NORM2,                                    /* norms in front of mixer and feed-forward ... */
    LB_T_NORM1_B, LB_T_NORM2_B,                                /* ... and their biases (layer norm) */
    LB_T_Q, LB_T_K, LB_T_V, LB_T_G, LB_T_F, LB_T_A1, LB_T_O,   /* projections */
    LB_T_A2, LB_T_GATE_BIAS, LB_T_LOWER, LB_T_HEAD_NORM,       /* small tensors of a decaying mixer */
    LB_T_DQ, LB_T_DQ_NORM, LB_T_UQ, LB_T_DKV, LB_T_DKV_NORM, LB_T_UK, LB_T_UV, LB_T_SINK, /* latent attention */
    LB_T_IN, LB_T_CONV, LB_T_CONV_B, LB_T_DT_BIAS, LB_T_A_LOG, LB_T_D,                   /* state-space mixer (its norm is LB_T_HEAD_NORM) */
    LB_T_FF_GATE, LB_T_FF_UP, LB_T_FF_DOWN,                    /* experts: with a %d for the expert's number */
    LB_T_TABLE,                                                /* experts of every token id, int32 [vocab, top] */
    LB_T_COUNT
};

typedef struct {
    int mixer;                       /* LB_MIX_* */
    int heads, kv_heads, dim, vdim;
    /* attention */
    int kv_from;                     /* layer whose cache is read; -1: its own */
    int block;                       /* positions seen in blocks of this size; 0: all earlier ones */
    int rot_dims; double rot_base;   /* rotation of queries and keys, neighbouring pairs */
    int v_norm, v_rot, sink;
    double scale;
    /* decaying linear attention */
    int decay;                       /* LB_DA_* */
    int rank;                        /* GLA: rows of the first gate projection */
    double tau;
    /* latent attention (also dim, vdim, rot_base, scale, sink): rot_dim more key dimensions, rotated and shared by all heads */
    int q_rank, kv_rank, rot_dim;
    struct { double factor, original, fast, slow; } yarn; /* factor 0: none */
    /* state-space mixer (heads of vdim channels) */
    int state, groups, taps, norm_groups;
    /* feed-forward */
    int ff_kind;                     /* LB_FF_* */
    int ff;                          /* width (of an expert), 0: none */
    int experts, top;
    double limit, alpha;             /* experts: clamped gating */
    char tensor[LB_T_COUNT][48];     /* tensor names */
} lb_stack_layer;

typedef struct {
    const char* design;
    int n_layers, width, vocab, max_ctx, dtype;
    int norm;                        /* LB_NORM_* of norm1, norm2 and the final norm */
    int serial;                      /* x += m mixer(norm1 x), then x += m ff(norm2 x); 0: both read the same x */
    double eps, residual_mult, logit_softcap;
    struct { int buckets, mul_prev, mul_cur; char name[48]; } bigram; /* pair embedding [buckets + 1, width]; 0 buckets: none */
    lb_stack_layer* layer;
    char embed[48], head[48], final_norm[48], final_norm_b[48];
} lb_stack_desc;

/* where weights come from: the safetensors files of a directory, or a seeded generator (dir == NULL) */
typedef struct { const void* files; uint64_t seed; uint64_t stream; } lb_weight_source;

/* config.json members every design reads: present, of the right kind and in range */
int lb_cfg_int(lb_ctx* c, const lb_json* j, const char* key, int lo, int hi, int layer, int* out);
int lb_cfg_num(lb_ctx* c, const lb_json* j, const char* key, int layer, double* out);

/* builds the model; takes its own copy of the description */
int lb_stack_create(lb_ctx* c, const lb_stack_desc* d, const lb_weight_source* src, lb_model** out);

/* designs: config.json -> description (layer array malloc'ed) */
int lb_vobunex_describe(lb_ctx* c, const lb_json* cfg, const lb_weight_source* src, lb_stack_desc* d);
int lb_nufalorn_describe(lb_ctx* c, const lb_json* cfg, const lb_weight_source* src, lb_stack_desc* d);
#endif
