/* Private view of a model: what the shared runtime (lb_model.c: decode step, graph, sampling, generation; lb_prefill.c: prompt
 * pass) keeps for every architecture, and the table of calls an architecture fills in (lb_hybrid.c: the int4 DeltaNet /
 * attention hybrid; lb_stack.c: bf16 models described by a list of layers). */
#ifndef LB_MODEL_PRIV_H
#define LB_MODEL_PRIV_H
#include "lb_internal.h"
#include "../kernels/params.h"

enum { /* src/launcher.s:92-141 */
    WS_DN_QKV = 0, WS_DN_Z = 3, WS_DN_OUT = 6, WS_DN_PROJ_A = 9, WS_DN_PROJ_B = 10, WS_DN_A_LOG = 11, WS_DN_DT_BIAS = 12,
    WS_DN_CONV1D = 13, WS_DN_NORM = 14,
    WS_FA_Q = 0, WS_FA_K = 3, WS_FA_V = 6, WS_FA_O = 9, WS_FA_Q_NORM = 12, WS_FA_K_NORM = 13,
    WS_GATE = 15, WS_UP = 18, WS_DOWN = 21, WS_INPUT_NORM = 24, WS_POST_NORM = 25,
    WG_EMBED = 0, WG_LM_HEAD = 1, WG_FINAL_NORM = 2
};

typedef struct {
    CUdeviceptr qweight, scales, qzeros; /* the reference format */
    CUdeviceptr packed;                  /* strip-packed copy for the persistent GEMV chain (0 = none) */
    int K, N;
} q4_mat;

typedef struct {
    int is_fa;
    q4_mat w_in, w_out, w_gateup, w_down;
    CUdeviceptr input_norm, post_norm;
    /* DeltaNet */
    CUdeviceptr proj_a, proj_b, a_log, dt_bias, conv_w, dn_norm, dn_state, conv_ring;
    CUdeviceptr snap_state, snap_conv; /* lb_model_checkpoint copies of dn_state and conv_ring (allocated on first use) */
    CUdeviceptr dn_params; /* lb_dn_layer_params of this layer in device memory, for the persistent chain */
    /* attention */
    CUdeviceptr q_norm, k_norm, k_cache, v_cache;
    int loaded;
} layer_t;

/* the activations of one prompt chunk: an architecture names the buffers it uses; the residual stream comes first */
#define LB_PF_MAX_BUFS 24
typedef union {
    CUdeviceptr b[LB_PF_MAX_BUFS];
    struct { CUdeviceptr X, xn16, proj, q, k, v, g, beta, mix, mix16, y, gu, act16; } hy; /* lb_hybrid.c */
    struct { CUdeviceptr X, h1, h2, proj, cat, q, k, a, o, seg_state, seg_decay, lq, kx, vx, lat_q, lat_part, xbc, dt, act, xg, ye, plan; } st; /* lb_stack.c */
} pf_set;

/* What an architecture supplies.  The runtime owns embedding, order of calls, positions, graph capture, chunking and
 * streams of the prompt pass, sampling and the generation loop. */
typedef struct lb_arch {
    const char* name;
    int pf_streams;                                     /* prompt pass: chunks in flight (<= LB_PF_MAX_STREAMS) */
    int (*reset_state)(lb_model* m);                    /* caches and recurrent states of the sequence back to empty (stream-ordered) */
    int (*snapshot)(lb_model* m, int restore);          /* checkpoint / rollback of the recurrent states */
    int (*state_ptr)(lb_model* m, int layer, int which, uint64_t* dptr, size_t* bytes);
    int (*step_layers)(lb_model* m);                    /* one token: m->X (its embedding) through every layer; position in m->d_pos */
    int (*head)(lb_model* m, CUdeviceptr x_row);        /* final norm + LM head of one row -> m->logits, arg-max candidates */
    int (*head_ctas)(lb_model* m);                      /* how many candidates head leaves */
    int (*head_rows)(lb_model* m, CUdeviceptr rows, int n, CUdeviceptr logits); /* the same for n <= lb_model.pf_chunk rows, no candidates */
    void (*pf_sizes)(const lb_model* m, size_t bytes[LB_PF_MAX_BUFS]);          /* bytes of each buffer of a chunk (0 = unused) */
    int (*pf_layer)(lb_model* m, pf_set* w, int l, int pos0, int T);           /* one layer over a chunk; on c->stream */
    void (*destroy)(lb_model* m);
} lb_arch;
#define LB_PF_MAX_STREAMS 4

struct lb_model {
    lb_ctx* c;
    const lb_arch* arch;
    void* impl;       /* lb_stack.c: its own description and weights */
    lb_model_cfg cfg; /* n_layers, hidden, vocab, max_ctx and eps hold for every architecture, the rest for the hybrid */
    int pf_chunk;     /* prompt pass: tokens per chunk, set by the architecture */
    int tp_rank, tp_size;
    /* per-shard sizes */
    int HV, HK, HQ, HKV, inter_s; /* heads / intermediate columns on this shard */
    int C_s;                      /* conv channels on this shard: 2*HK*128 + HV*128 */
    layer_t* L;
    CUdeviceptr embed, lm_head, final_norm;
    CUdeviceptr bigram; /* embedding of (previous, current) token pairs, added to the token's own; 0: none */
    int bigram_buckets, bigram_mul_prev, bigram_mul_cur;
    CUdeviceptr d_tokens; /* the sequence's token ids by position [max_ctx] (decode steps enter theirs only where the embedding needs them) */
    int globals_loaded;
    /* activations */
    CUdeviceptr X, xn, in_out, mix_out, mlp_m, logits, d_token, d_pos, d_next, cand_val, cand_idx;
    int* h_next; /* pinned */
    int host_pos;  /* position the next step will decode, as the host knows it: set_input's value plus the steps issued since */
    uint64_t weight_bytes;
    lb_graph* graph;
    int step_kernels;
    lb_comm* comm;   /* tensor parallel: exchange buffers */
    int vocab_s;     /* vocabulary rows on this shard */
    int ar_count;    /* all-reduces issued so far in the step being built (slot parity) */
    int use_chain;   /* consecutive GEMVs of the step go out as one persistent launch (lb_gemv_chain) */
    CUdeviceptr tp_params[2]; /* tensor parallel: lb_tp_params of the two exchange slots in device memory, for the chain */
    lb_chain_op pend[LB_CHAIN_MAX_OPS]; /* GEMVs and DeltaNet mixers collected since the last stand-alone kernel */
    int n_pend;
    float temperature; int top_k; uint64_t sample_seed; /* top_k == 0: greedy (arg-max); else temperature / top-k sampling */
    struct lb_prefill_ws* ws; /* prompt-pass buffers (lb_prefill.c), NULL until the first prefill */
};


/* prompt-pass workspace (allocated by the first lb_model_prefill) */
typedef struct lb_prefill_ws lb_prefill_ws;

int lb_model_is_fa(const lb_model_cfg* c, int l);
int lb_model_launch_sampler(lb_model* m);
int lb_model_embed_bigram(lb_model* m, CUdeviceptr token, CUdeviceptr pos_ptr, int pos0, int n, CUdeviceptr out);
int lb_model_alloc_common(lb_model* m); /* the buffers every architecture uses; cfg and vocab_s must be set */
pf_set* lb_prefill_set(lb_model* m, int s);    /* buffers of prompt stream s (after a prompt pass) */
int lb_dalloc(lb_model* m, CUdeviceptr* p, size_t bytes);
int lb_upload(lb_model* m, CUdeviceptr* p, const void* src, size_t bytes);
#endif
