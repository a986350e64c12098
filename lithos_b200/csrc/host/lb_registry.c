/* The model registry: config.json's "architecture" picks the model class; its loader builds the model, with weights from the
 * directory or (no directory) from the seeded generator. */
#include "lb_model_priv.h"
#include "lb_json.h"
#include "lb_safetensors.h"
#include "lb_stack.h"
#include <sys/stat.h>

typedef int (*open_fn)(lb_ctx* c, const lb_json* cfg, const char* dir, int max_ctx, int dtype, uint64_t seed, lb_model** out);

static int open_stack(lb_ctx* c, const lb_json* cfg, const char* dir, int max_ctx, int dtype, uint64_t seed, lb_model** out,
                      int (*describe)(lb_ctx*, const lb_json*, const lb_weight_source*, lb_stack_desc*)) {
    lb_st_set files;
    lb_weight_source src = {NULL, seed, 0};
    if (dir) {
        LB_TRY(lb_st_open(dir, &files, c->err, sizeof c->err));
        src.files = &files;
    }
    lb_stack_desc d;
    memset(&d, 0, sizeof d);
    int st = describe(c, cfg, &src, &d);
    if (st == LB_OK) {
        d.max_ctx = max_ctx;
        d.dtype = dtype;
        st = lb_stack_create(c, &d, &src, out);
    }
    free(d.layer);
    if (dir) lb_st_close(&files);
    return st;
}
static int open_nufalorn(lb_ctx* c, const lb_json* cfg, const char* dir, int max_ctx, int dtype, uint64_t seed, lb_model** out) {
    return open_stack(c, cfg, dir, max_ctx, dtype, seed, out, lb_nufalorn_describe);
}

static int open_vobunex(lb_ctx* c, const lb_json* cfg, const char* dir, int max_ctx, int dtype, uint64_t seed, lb_model** out) {
    return open_stack(c, cfg, dir, max_ctx, dtype, seed, out, lb_vobunex_describe);
}

/* the int4 hybrid: config.json with the fields of lb_model_cfg; weights through weight_index.bin, which is written over the
 * directory's safetensors files when it is not there yet */
static int open_hybrid(lb_ctx* c, const lb_json* cfg, const char* dir, int max_ctx, int dtype, uint64_t seed, lb_model** out) {
    if (dtype != LB_DTYPE_BF16) return lb_fail(c, LB_ERR_INVALID, "the hybrid runs with int4 weights and 16-bit activations only");
    lb_model_cfg m;
    memset(&m, 0, sizeof m);
    struct { const char* key; int32_t* v; int dflt; } f[] = {
        {"n_layers", &m.n_layers, 0}, {"hidden", &m.hidden, 0}, {"inter", &m.inter, 0}, {"vocab", &m.vocab, 0}, {"dn_k_heads", &m.dn_k_heads, 0},
        {"dn_v_heads", &m.dn_v_heads, 0}, {"dn_dim", &m.dn_dim, 128}, {"conv_taps", &m.conv_taps, 4}, {"fa_q_heads", &m.fa_q_heads, 0},
        {"fa_kv_heads", &m.fa_kv_heads, 0}, {"fa_dim", &m.fa_dim, 256}, {"rot_dims", &m.rot_dims, 64}, {"group", &m.group, 128}, {"fa_period", &m.fa_period, 4}};
    for (size_t i = 0; i < sizeof f / sizeof f[0]; i++) {
        *f[i].v = (int32_t)lb_json_num(cfg, f[i].key, f[i].dflt);
        if (*f[i].v < 1) return lb_fail(c, LB_ERR_INVALID, "config: '%s' is missing or not positive", f[i].key);
    }
    m.eps = (float)lb_json_num(cfg, "eps", 1e-6);
    m.rope_theta = (float)lb_json_num(cfg, "rope_theta", 1e7);
    m.max_ctx = max_ctx;
    LB_TRY(lb_model_create(c, &m, 0, 1, out));
    if (!dir) return lb_model_fill_synthetic(*out, seed);
    char path[1536];
    struct stat sb;
    snprintf(path, sizeof path, "%s/weight_index.bin", dir);
    if (stat(path, &sb) != 0) LB_TRY(lb_weight_index_from_safetensors(dir, &m, c->err, sizeof c->err));
    return lb_load_weights(c, dir, *out);
}

static const struct { const char* architecture; open_fn open; const char* images; } k_registry[] = {
    {"Nufalorn", open_nufalorn, "small prefill rows_gemv dense_gemm window_attention decay_attention"},
    {"Vobunex", open_vobunex, "small prefill rows_gemv dense_gemm window_attention latent_attention ssm"},
    {"Qwen3.5-hybrid", open_hybrid, "gemv chain batched batched_tc deltanet attention attention_mma small comm prefill"},
};

static int find(const lb_json* cfg, char* err, size_t errlen) {
    const char* name = lb_json_str(cfg, "architecture");
    for (size_t i = 0; name && i < sizeof k_registry / sizeof k_registry[0]; i++)
        if (!strcmp(k_registry[i].architecture, name)) return (int)i;
    if (err) snprintf(err, errlen, "config: no model class for architecture '%s'", name ? name : "(none)");
    return -1;
}

LB_API const char* lb_registry_name(int i) { return i >= 0 && (size_t)i < sizeof k_registry / sizeof k_registry[0] ? k_registry[i].architecture : NULL; }

LB_API const char* lb_config_images(const char* config_json) {
    if (!config_json) return NULL;
    lb_json* cfg = lb_json_parse(config_json, strlen(config_json), NULL, 0);
    const int i = cfg ? find(cfg, NULL, 0) : -1;
    lb_json_free(cfg);
    return i < 0 ? NULL : k_registry[i].images;
}

static int open_text(lb_ctx* c, const char* text, size_t len, const char* dir, int max_ctx, int dtype, uint64_t seed, lb_model** out) {
    if (max_ctx < 1) return lb_fail(c, LB_ERR_INVALID, "model: the context must hold at least one token");
    if (dtype != LB_DTYPE_BF16 && dtype != LB_DTYPE_F32) return lb_fail(c, LB_ERR_INVALID, "model: unknown number format %d", dtype);
    char why[200];
    lb_json* cfg = lb_json_parse(text, len, why, sizeof why);
    if (!cfg) return lb_fail(c, LB_ERR_INVALID, "config.json: %s", why);
    const int i = find(cfg, c->err, sizeof c->err);
    int st = LB_ERR_INVALID;
    if (i >= 0) st = k_registry[i].open(c, cfg, dir, max_ctx, dtype, seed, out);
    lb_json_free(cfg);
    if (st != LB_OK && *out) { /* nothing half-built is handed out */
        lb_model_destroy(*out);
        *out = NULL;
    }
    return st;
}

LB_API int lb_model_open(lb_ctx* c, const char* model_dir, int max_ctx, int dtype, lb_model** out) {
    if (!c || !model_dir || !out) return LB_ERR_INVALID;
    *out = NULL;
    char path[1536];
    snprintf(path, sizeof path, "%s/config.json", model_dir);
    size_t n = 0;
    FILE* f = fopen(path, "rb");
    if (!f) return lb_fail(c, LB_ERR_IO, "cannot read %s", path);
    fseek(f, 0, SEEK_END);
    n = (size_t)ftell(f);
    fseek(f, 0, SEEK_SET);
    char* text = (char*)malloc(n + 1);
    if (!text || fread(text, 1, n, f) != n) { free(text); fclose(f); return lb_fail(c, LB_ERR_IO, "cannot read %s", path); }
    fclose(f);
    const int st = open_text(c, text, n, model_dir, max_ctx, dtype, 0, out);
    free(text);
    return st;
}

LB_API int lb_model_open_synthetic(lb_ctx* c, const char* config_json, int max_ctx, int dtype, uint64_t seed, lb_model** out) {
    if (!c || !config_json || !out) return LB_ERR_INVALID;
    *out = NULL;
    return open_text(c, config_json, strlen(config_json), NULL, max_ctx, dtype, seed, out);
}
