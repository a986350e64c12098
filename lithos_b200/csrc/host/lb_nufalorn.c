/* The Nufalorn design: config.json and tensor names -> the stack's description (lb_stack.h).
 * Layers of three mixers (attention over blocks of positions with rotated values and a soft-max sink; HGRN2; GLA), mixer and
 * ReLU-gated feed-forward side by side on two norms of the same residual, x += m (mixer + feed-forward), soft-capped logits. */
#include "lb_stack.h"
#include "lb_safetensors.h"
#include "../kernels/params.h"
#include <math.h>

int lb_nufalorn_describe(lb_ctx* c, const lb_json* cfg, const lb_weight_source* src, lb_stack_desc* d) {
    const lb_json* layers = lb_json_get(cfg, "layers");
    if (!layers || layers->type != LB_JSON_ARRAY || layers->n < 1) return lb_fail(c, LB_ERR_INVALID, "config: 'layers' is not a list of layers");
    d->design = "Nufalorn";
    d->n_layers = layers->n;
    LB_TRY(lb_cfg_int(c, cfg, "width", 1, 1 << 20, -1, &d->width));
    LB_TRY(lb_cfg_int(c, cfg, "vocab", 1, 1 << 28, -1, &d->vocab));
    LB_TRY(lb_cfg_num(c, lb_json_get(cfg, "norm"), "eps", -1, &d->eps));
    d->residual_mult = 1.0;
    if (lb_json_has(cfg, "residual_mult")) LB_TRY(lb_cfg_num(c, cfg, "residual_mult", -1, &d->residual_mult));
    if (lb_json_has(cfg, "logit_softcap")) LB_TRY(lb_cfg_num(c, cfg, "logit_softcap", -1, &d->logit_softcap)); /* else 0: no cap */
    snprintf(d->embed, sizeof d->embed, "embed");
    snprintf(d->head, sizeof d->head, "head");
    snprintf(d->final_norm, sizeof d->final_norm, "final.norm");
    d->layer = (lb_stack_layer*)calloc((size_t)d->n_layers, sizeof *d->layer);
    if (!d->layer) return LB_ERR_NOMEM;
    for (int i = 0; i < d->n_layers; i++) {
        const lb_json *e = &layers->item[i], *m = lb_json_get(e, "mixer"), *f = lb_json_get(e, "mlp");
        const char* type = lb_json_str(e, "type");
        lb_stack_layer* L = &d->layer[i];
#define NAME(role, ...) snprintf(L->tensor[role], sizeof L->tensor[role], __VA_ARGS__)
        if (!type || !m) return lb_fail(c, LB_ERR_INVALID, "config: layer %d has no type or no mixer", i);
        L->kv_from = -1;
        LB_TRY(lb_cfg_int(c, m, "heads", 1, 65536, i, &L->heads));
        LB_TRY(lb_cfg_int(c, m, "dim", 1, 65536, i, &L->dim));
        LB_TRY(lb_cfg_int(c, m, "vdim", 1, 65536, i, &L->vdim));
        L->kv_heads = L->heads;
        NAME(LB_T_NORM1, "l%d.norm1", i);
        NAME(LB_T_Q, "l%d.mix.q", i);
        NAME(LB_T_O, "l%d.mix.o", i);
        if (!strcmp(type, "attention")) {
            const lb_json *rot = lb_json_get(m, "rot"), *mask = lb_json_get(m, "mask");
            L->mixer = LB_MIX_ATTENTION;
            L->v_norm = L->v_rot = L->sink = 1;
            if (lb_json_has(m, "kv_heads")) LB_TRY(lb_cfg_int(c, m, "kv_heads", 1, L->heads, i, &L->kv_heads));
            L->rot_dims = L->dim;
            if (lb_json_has(rot, "dims")) LB_TRY(lb_cfg_int(c, rot, "dims", 0, L->dim, i, &L->rot_dims));
            LB_TRY(lb_cfg_num(c, rot, "base", i, &L->rot_base));
            if (mask && mask->type == LB_JSON_OBJECT) LB_TRY(lb_cfg_int(c, mask, "size", 1, 1 << 30, i, &L->block)); /* else 0: every earlier position */
            LB_TRY(lb_cfg_num(c, m, "scale", i, &L->scale));
            if (lb_json_has(m, "kv_from")) LB_TRY(lb_cfg_int(c, m, "kv_from", 0, i - 1, i, &L->kv_from));
            if (L->kv_from < 0) {
                NAME(LB_T_K, "l%d.mix.k", i);
                NAME(LB_T_V, "l%d.mix.v", i);
            }
        } else if (!strcmp(type, "hgrn2") || !strcmp(type, "gla")) {
            L->mixer = LB_MIX_DECAY;
            NAME(LB_T_V, "l%d.mix.v", i);
            NAME(LB_T_HEAD_NORM, "l%d.mix.norm", i);
            if (type[0] == 'h') {
                L->decay = LB_DA_HGRN2;
                NAME(LB_T_F, "l%d.mix.f", i);
                NAME(LB_T_GATE_BIAS, "l%d.mix.f.b", i);
                NAME(LB_T_LOWER, "l%d.mix.lower", i);
            } else {
                L->decay = LB_DA_GLA;
                LB_TRY(lb_cfg_num(c, m, "tau", i, &L->tau));
                NAME(LB_T_K, "l%d.mix.k", i);
                NAME(LB_T_G, "l%d.mix.g", i);
                NAME(LB_T_A1, "l%d.mix.a1", i);
                NAME(LB_T_A2, "l%d.mix.a2", i);
                NAME(LB_T_GATE_BIAS, "l%d.mix.a2.b", i);
                L->rank = 16; /* generated weights; a checkpoint's tensor says */
                if (src->files) {
                    const lb_st_tensor* a1 = lb_st_find((const lb_st_set*)src->files, L->tensor[LB_T_A1]);
                    if (!a1 || a1->ndim != 2 || a1->dim[0] < 1) return lb_fail(c, LB_ERR_IO, "tensor %s is missing or not a matrix", L->tensor[LB_T_A1]);
                    L->rank = (int)a1->dim[0];
                }
            }
        } else return lb_fail(c, LB_ERR_INVALID, "config: layer %d: unknown mixer '%s'", i, type);
        if (f && f->type == LB_JSON_OBJECT) {
            const char* kind = lb_json_str(f, "kind");
            if (kind && strcmp(kind, "dense")) return lb_fail(c, LB_ERR_INVALID, "config: layer %d: unknown feed-forward '%s'", i, kind);
            LB_TRY(lb_cfg_int(c, f, "ff", 1, 1 << 24, i, &L->ff));
            NAME(LB_T_NORM2, "l%d.norm2", i);
            NAME(LB_T_FF_GATE, "l%d.mlp.gate", i);
            NAME(LB_T_FF_UP, "l%d.mlp.up", i);
            NAME(LB_T_FF_DOWN, "l%d.mlp.down", i);
        }
#undef NAME
    }
    return LB_OK;
}
