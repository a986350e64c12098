/* The Vobunex design: config.json and tensor names -> the stack's description (lb_stack.h).
 * Layers of two mixers (latent attention with a learned soft-max sink and YaRN-scaled rotation; Mamba-2), then a feed-forward (squared ReLU, or
 * experts that a table gives every token id), each behind a layer norm; embeddings of tokens and of token pairs. */
#include "lb_stack.h"
#include "../kernels/params.h"

#define EXPERT_ALPHA 1.702

static int latent(lb_ctx* c, const lb_json* m, int i, lb_stack_layer* L) {
    const lb_json *rot = lb_json_get(m, "rot"), *yarn = rot ? lb_json_get(rot, "scaling") : NULL;
    int dims = 0;
    L->mixer = LB_MIX_LATENT;
    L->sink = 1;
    LB_TRY(lb_cfg_int(c, m, "dim", 1, 65536, i, &L->dim));
    LB_TRY(lb_cfg_int(c, m, "rot_dim", 2, 65536, i, &L->rot_dim));
    LB_TRY(lb_cfg_int(c, m, "q_rank", 1, 1 << 20, i, &L->q_rank));
    LB_TRY(lb_cfg_int(c, m, "kv_rank", 1, 1 << 20, i, &L->kv_rank));
    LB_TRY(lb_cfg_num(c, m, "scale", i, &L->scale));
    LB_TRY(lb_cfg_num(c, rot, "base", i, &L->rot_base));
    LB_TRY(lb_cfg_int(c, rot, "dims", 2, 65536, i, &dims));
    if (dims != L->rot_dim) return lb_fail(c, LB_ERR_INVALID, "config: layer %d: all of rot_dim is rotated (rot.dims %d, rot_dim %d)", i, dims, L->rot_dim);
    if (yarn && yarn->type == LB_JSON_OBJECT) {
        LB_TRY(lb_cfg_num(c, yarn, "factor", i, &L->yarn.factor));
        LB_TRY(lb_cfg_num(c, yarn, "original", i, &L->yarn.original));
        LB_TRY(lb_cfg_num(c, yarn, "fast", i, &L->yarn.fast));
        LB_TRY(lb_cfg_num(c, yarn, "slow", i, &L->yarn.slow));
        if (!(L->yarn.factor > 0 && L->yarn.original > 0 && L->yarn.fast > 0 && L->yarn.slow > 0))
            return lb_fail(c, LB_ERR_INVALID, "config: layer %d: rot.scaling needs positive numbers", i);
    }
    static const struct { int role; const char* name; } t[] = {{LB_T_DQ, "dq"}, {LB_T_DQ_NORM, "dq.norm"}, {LB_T_UQ, "uq"}, {LB_T_DKV, "dkv"},
        {LB_T_DKV_NORM, "dkv.norm"}, {LB_T_UK, "uk"}, {LB_T_UV, "uv"}, {LB_T_SINK, "sink"}};
    for (size_t k = 0; k < sizeof t / sizeof t[0]; k++) snprintf(L->tensor[t[k].role], sizeof L->tensor[0], "l%d.mix.%s", i, t[k].name);
    return LB_OK;
}

static int mamba2(lb_ctx* c, const lb_json* m, int i, lb_stack_layer* L) {
    L->mixer = LB_MIX_SSM;
    LB_TRY(lb_cfg_int(c, m, "state", 1, 65536, i, &L->state));
    LB_TRY(lb_cfg_int(c, m, "groups", 1, 65536, i, &L->groups));
    LB_TRY(lb_cfg_int(c, m, "conv", 1, 65536, i, &L->taps));
    LB_TRY(lb_cfg_int(c, m, "norm_groups", 1, 1 << 24, i, &L->norm_groups));
    static const struct { int role; const char* name; } t[] = {{LB_T_IN, "in"}, {LB_T_CONV, "conv"}, {LB_T_CONV_B, "conv.b"}, {LB_T_DT_BIAS, "dt_bias"},
        {LB_T_A_LOG, "A_log"}, {LB_T_D, "D"}, {LB_T_HEAD_NORM, "norm"}};
    for (size_t k = 0; k < sizeof t / sizeof t[0]; k++) snprintf(L->tensor[t[k].role], sizeof L->tensor[0], "l%d.mix.%s", i, t[k].name);
    return LB_OK;
}

static int feed_forward(lb_ctx* c, const lb_json* f, int i, lb_stack_layer* L) {
    const char* kind = lb_json_str(f, "kind");
#define NAME(role, ...) snprintf(L->tensor[role], sizeof L->tensor[role], __VA_ARGS__)
    NAME(LB_T_NORM2, "l%d.norm2", i);
    NAME(LB_T_NORM2_B, "l%d.norm2.b", i);
    if (kind && !strcmp(kind, "dense")) {
        L->ff_kind = LB_FF_RELU2;
        LB_TRY(lb_cfg_int(c, f, "ff", 1, 1 << 24, i, &L->ff));
        NAME(LB_T_FF_UP, "l%d.mlp.up", i);
        NAME(LB_T_FF_DOWN, "l%d.mlp.down", i);
    } else if (kind && !strcmp(kind, "moe")) {
        const lb_json *e = lb_json_get(f, "expert"), *r = lb_json_get(f, "router");
        L->ff_kind = LB_FF_EXPERTS;
        L->alpha = EXPERT_ALPHA;
        LB_TRY(lb_cfg_int(c, e, "ff", 1, 1 << 24, i, &L->ff));
        LB_TRY(lb_cfg_num(c, e, "limit", i, &L->limit));
        LB_TRY(lb_cfg_int(c, r, "experts", 1, 65536, i, &L->experts));
        LB_TRY(lb_cfg_int(c, r, "top", 1, L->experts, i, &L->top));
        NAME(LB_T_FF_GATE, "l%d.mlp.e%%d.gate", i);
        NAME(LB_T_FF_UP, "l%d.mlp.e%%d.up", i);
        NAME(LB_T_FF_DOWN, "l%d.mlp.e%%d.down", i);
        NAME(LB_T_TABLE, "l%d.mlp.table", i);
    } else return lb_fail(c, LB_ERR_INVALID, "config: layer %d: unknown feed-forward '%s'", i, kind ? kind : "(none)");
    return LB_OK;
}

int lb_vobunex_describe(lb_ctx* c, const lb_json* cfg, const lb_weight_source* src, lb_stack_desc* d) {
    const lb_json *layers = lb_json_get(cfg, "layers"), *emb = lb_json_get(cfg, "embedding"), *pair = emb ? lb_json_get(emb, "bigram") : NULL;
    if (!layers || layers->type != LB_JSON_ARRAY || layers->n < 1) return lb_fail(c, LB_ERR_INVALID, "config: 'layers' is not a list of layers");
    d->design = "Vobunex";
    d->n_layers = layers->n;
    d->serial = 1;
    d->norm = LB_NORM_LAYER;
    d->residual_mult = 1.0;
    LB_TRY(lb_cfg_int(c, cfg, "width", 1, 1 << 20, -1, &d->width));
    LB_TRY(lb_cfg_int(c, cfg, "vocab", 1, 1 << 28, -1, &d->vocab));
    LB_TRY(lb_cfg_num(c, lb_json_get(cfg, "norm"), "eps", -1, &d->eps));
    if (pair && pair->type == LB_JSON_OBJECT) {
        LB_TRY(lb_cfg_int(c, pair, "buckets", 1, 1 << 28, -1, &d->bigram.buckets));
        LB_TRY(lb_cfg_int(c, pair, "mul_prev", 0, 0x7fffffff, -1, &d->bigram.mul_prev));
        LB_TRY(lb_cfg_int(c, pair, "mul_cur", 0, 0x7fffffff, -1, &d->bigram.mul_cur));
        snprintf(d->bigram.name, sizeof d->bigram.name, "bigram");
    }
    snprintf(d->embed, sizeof d->embed, "embed");
    snprintf(d->head, sizeof d->head, "head");
    snprintf(d->final_norm, sizeof d->final_norm, "final.norm");
    snprintf(d->final_norm_b, sizeof d->final_norm_b, "final.norm.b");
    d->layer = (lb_stack_layer*)calloc((size_t)d->n_layers, sizeof *d->layer);
    if (!d->layer) return LB_ERR_NOMEM;
    for (int i = 0; i < d->n_layers; i++) {
        const lb_json *e = &layers->item[i], *m = lb_json_get(e, "mixer"), *f = lb_json_get(e, "mlp");
        const char* type = lb_json_str(e, "type");
        lb_stack_layer* L = &d->layer[i];
        if (!type || !m) return lb_fail(c, LB_ERR_INVALID, "config: layer %d has no type or no mixer", i);
        L->kv_from = -1;
        LB_TRY(lb_cfg_int(c, m, "heads", 1, 65536, i, &L->heads));
        LB_TRY(lb_cfg_int(c, m, "vdim", 1, 65536, i, &L->vdim));
        NAME(LB_T_NORM1, "l%d.norm1", i);
        NAME(LB_T_NORM1_B, "l%d.norm1.b", i);
        NAME(LB_T_O, "l%d.mix.o", i);
        if (!strcmp(type, "latent_attention")) LB_TRY(latent(c, m, i, L));
        else if (!strcmp(type, "mamba2")) LB_TRY(mamba2(c, m, i, L));
        else return lb_fail(c, LB_ERR_INVALID, "config: layer %d: unknown mixer '%s'", i, type);
        if (f && f->type == LB_JSON_OBJECT) LB_TRY(feed_forward(c, f, i, L));
    }
#undef NAME
    return LB_OK;
}
