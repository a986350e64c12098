/* Models described by a list of layers (bf16 weights, fp32 residual stream): what a design hands to the stack (lb_stack.c).
 * A design (lb_nufalorn.c) turns its config.json into this description and says which tensor feeds which part; every
 * mechanism takes its constants from here. */
#ifndef LB_STACK_H
#define LB_STACK_H
#include "lb_internal.h"
#include "lb_json.h"

enum { LB_MIX_ATTENTION = 0, LB_MIX_DECAY = 1 };

/* weight roles of a layer; a role without a name is absent */
enum {
    LB_T_NORM1, LB_T_NORM2,                                    /* zero-centred RMS norms in front of mixer and feed-forward */
    LB_T_Q, LB_T_K, LB_T_V, LB_T_G, LB_T_F, LB_T_A1, LB_T_O,   /* projections */
    LB_T_A2, LB_T_GATE_BIAS, LB_T_LOWER, LB_T_HEAD_NORM,       /* small tensors of a decaying mixer */
    LB_T_FF_GATE, LB_T_FF_UP, LB_T_FF_DOWN,
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
    int ff;                          /* feed-forward width, 0: none (ReLU-gated) */
    char tensor[LB_T_COUNT][48];     /* tensor names */
} lb_stack_layer;

typedef struct {
    const char* design;
    int n_layers, width, vocab, max_ctx, dtype;
    double eps, residual_mult, logit_softcap;
    lb_stack_layer* layer;
    char embed[48], head[48], final_norm[48];
} lb_stack_desc;

/* where weights come from: the safetensors files of a directory, or a seeded generator (dir == NULL) */
typedef struct { const void* files; uint64_t seed; uint64_t stream; } lb_weight_source;

/* builds the model; takes its own copy of the description */
int lb_stack_create(lb_ctx* c, const lb_stack_desc* d, const lb_weight_source* src, lb_model** out);

/* designs: config.json -> description (layer array malloc'ed) */
int lb_nufalorn_describe(lb_ctx* c, const lb_json* cfg, const lb_weight_source* src, lb_stack_desc* d);
#endif
