/* Models described by a list of layers (lb_stack.h): weights, caches and states, the decode step and a prompt chunk.
 *
 * A layer: x += m (mixer(norm1 x) + feed-forward(norm2 x)).  The projections of both sides read the same row, and the two output
 * projections add into the same row, so a layer of the decode step is three launches:
 *   [both norms + mixer's input projections | gate, up projections + ReLU gating]   rows_gemv, two matrices
 *   [mixer: rotations, cache append, attention over the cache | gates, state update, read-out]   wattn_rows_* | da_step_*
 *   [per-head norm and gate + (W_o | W_down) as one matrix over (mixer, feed-forward) + residual]   rows_gemv, one matrix
 * and of a prompt chunk: norm_rows2, one product launch for all input projections, the mixer's kernels, one product launch for the
 * outputs (gemm_bf16_tc, tcgen05; gemm_f32_simt when the model runs in fp32).
 *
 * Device layout: the mixer's input projections are stacked along rows ([q | k | v], [q | f | v], [q | k | v | g | a1]); gate and up rows
 * alternate; W_o and W_down stand side by side.  Columns are padded to a multiple of 64 with zeros, so any size is a whole number of
 * 128-byte operand rows.  Caches hold max_ctx rows [kv_heads, dim rounded up to 16] per attention layer that has keys of its own.
 */
#include "lb_model_priv.h"
#include "lb_safetensors.h"
#include "lb_stack.h"
#include <math.h>

#define ST_CHUNK 1024 /* largest chunk of a prompt; stack_chunk picks the model's */
#define ST_STREAMS 4
#define ST_SEG 128     /* tokens of a chunk a recurrence walks one after the other; segments run side by side */

typedef struct {
    CUdeviceptr w;
    int rows, K; /* rows with a result; padded columns */
    CUtensorMap tmap;
} st_mat;

typedef struct {
    st_mat in, ff, out; /* mixer's inputs, (gate, up) pairs, (W_o | W_down) */
    CUdeviceptr norm1, norm2, a2, bias, lower, head_norm;
    CUdeviceptr k_cache, v_cache; /* of this layer, or of the layer it reads */
    CUdeviceptr freq_k, freq_v;
    CUdeviceptr state, snap;
    int q_off, k_off, v_off, g_off, a1_off; /* sections of the mixer's projections; -1: absent */
    int n_mix, n_mix_pad, dim_p, vdim_p, dk_p;
    int splits; /* decode attention: slices of the visible positions */
} st_layer;

typedef struct {
    lb_stack_desc d; /* layer array owned */
    st_layer* L;
    st_mat head;
    int Kw; /* width padded to 64 columns */
    int esz; /* bytes of an activation / cache element: 2 (bf16) or 4 (fp32) */
    int max_in, max_cat, max_mix, max_ff, max_q, max_dk, max_o;
    size_t max_state;
    CUdeviceptr proj, mix, act;        /* decode step: fp32 */
    CUdeviceptr scratch, counters;
} stack_t;

static size_t state_bytes(const lb_stack_layer* D) { return (size_t)D->heads * D->dim * D->vdim * 4; }
static int pad_to(int n, int m) { return (n + m - 1) / m * m; }
static stack_t* S_of(const lb_model* m) { return (stack_t*)m->impl; }

/* ---- weights ------------------------------------------------------------------------------------------------ */
/* tensor `name` [rows, cols] (rows alone: a vector) as bf16 into dst: row r at dst + r * row_stride */
static int read_rows(lb_ctx* c, lb_weight_source* src, const char* name, int rows, int cols, uint16_t* dst, size_t row_stride, float gen_mean, float gen_std) {
    if (!src->files) { /* generated: uniform with the given mean and standard deviation, a function of (seed, order, element) */
        const uint64_t stream = ++src->stream, seed = src->seed;
        const float half = gen_std * 1.7320508f;
#pragma omp parallel for schedule(static)
        for (int r = 0; r < rows; r++) {
            for (int i = 0; i < cols; i += 4) {
                uint64_t u = lb_rng_u64(seed, stream, ((uint64_t)r * (uint64_t)cols + (uint64_t)i) / 4 + (uint64_t)r);
                for (int e = 0; e < 4 && i + e < cols; e++, u >>= 16)
                    dst[(size_t)r * row_stride + i + e] = lb_f32_to_bf16(gen_mean + half * ((float)(u & 0xffff) * (2.0f / 65535.0f) - 1.0f));
            }
        }
        return LB_OK;
    }
    const lb_st_tensor* t = lb_st_find((const lb_st_set*)src->files, name);
    if (!t) return lb_fail(c, LB_ERR_IO, "tensor %s is not in the checkpoint", name);
    const int64_t count = (int64_t)rows * cols;
    const int shape_ok = (t->ndim == 2 && t->dim[0] == rows && t->dim[1] == cols) || (t->ndim == 1 && count == t->dim[0] && (rows == 1 || cols == 1));
    if (strcmp(t->dtype, "BF16") || !shape_ok || t->size != (uint64_t)count * 2)
        return lb_fail(c, LB_ERR_IO, "tensor %s: bf16 [%d, %d] expected, the file has %s with %d dimensions [%lld, %lld]", name, rows, cols, t->dtype, t->ndim,
                       (long long)t->dim[0], (long long)t->dim[1]);
    for (int r = 0; r < rows; r++) memcpy(dst + (size_t)r * row_stride, (const uint16_t*)t->data + (size_t)r * cols, (size_t)cols * 2);
    return LB_OK;
}

static int load_vec(lb_model* m, lb_weight_source* src, const char* name, int rows, int cols, CUdeviceptr* out, float mean, float std) {
    uint16_t* h = (uint16_t*)malloc((size_t)rows * cols * 2);
    if (!h) return lb_fail(m->c, LB_ERR_NOMEM, "model: host staging");
    int st = read_rows(m->c, src, name, rows, cols, h, (size_t)cols, mean, std);
    if (st == LB_OK) st = lb_upload(m, out, h, (size_t)rows * cols * 2);
    free(h);
    return st;
}

static int map_rows(lb_ctx* c, CUtensorMap* tm, CUdeviceptr p, int rows, int K, int box_rows) {
    cuuint64_t dims[2] = {(cuuint64_t)K, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)K * 2};
    cuuint32_t box[2] = {LB_DG_KB, (cuuint32_t)box_rows}, es[2] = {1, 1};
    LB_CU(c, lb_drv.TensorMapEncodeTiled(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void*)p, dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE));
    return LB_OK;
}

/* where part of a device matrix comes from: tensor rows r go to device row row0 + r * row_step, columns from col0 */
typedef struct { const char* name; int rows, cols, row0, row_step, col0; } st_part;

static int build_mat(lb_model* m, lb_weight_source* src, st_mat* w, int rows, int K, const st_part* parts, int n_parts) {
    const int alloc_rows = pad_to(rows, 2);
    const size_t bytes = (size_t)alloc_rows * K * 2;
    uint16_t* h = (uint16_t*)calloc((size_t)alloc_rows * K, 2);
    if (!h) return lb_fail(m->c, LB_ERR_NOMEM, "model: host staging");
    int st = LB_OK;
    for (int i = 0; i < n_parts && st == LB_OK; i++)
        st = read_rows(m->c, src, parts[i].name, parts[i].rows, parts[i].cols, h + (size_t)parts[i].row0 * K + parts[i].col0, (size_t)parts[i].row_step * K, 0.f,
                       1.0f / sqrtf((float)parts[i].cols));
    if (st == LB_OK) st = lb_upload(m, &w->w, h, bytes);
    free(h);
    if (st != LB_OK) return st;
    w->rows = rows;
    w->K = K;
    m->weight_bytes += bytes;
    return map_rows(m->c, &w->tmap, w->w, rows, K, LB_DG_ROWS);
}

static int upload_freqs(lb_model* m, CUdeviceptr* out, int dims, double base) {
    double f[LB_WA_MAX_DIM / 2];
    for (int i = 0; i < dims / 2; i++) f[i] = pow(base, -2.0 * i / dims);
    return lb_upload(m, out, f, sizeof(double) * (size_t)(dims > 1 ? dims / 2 : 1));
}

static int check_layer(lb_ctx* c, const lb_stack_desc* d, int i) {
    const lb_stack_layer* L = &d->layer[i];
    if (L->mixer == LB_MIX_ATTENTION) {
        if (L->heads % L->kv_heads || L->dim > LB_WA_MAX_DIM || L->vdim > LB_WA_MAX_DIM || L->vdim % 2 || L->rot_dims % 2 || L->rot_dims > L->dim)
            return lb_fail(c, LB_ERR_INVALID, "layer %d: attention needs heads a multiple of kv_heads, head sizes up to %d, even vdim and rotated size", i, LB_WA_MAX_DIM);
        if (L->kv_from >= 0) {
            const lb_stack_layer* o = &d->layer[L->kv_from];
            if (L->kv_from >= i || o->mixer != LB_MIX_ATTENTION || o->kv_from >= 0 || o->kv_heads != L->kv_heads || o->dim != L->dim || o->vdim != L->vdim)
                return lb_fail(c, LB_ERR_INVALID, "layer %d: layer %d has no keys and values of these sizes to share", i, L->kv_from);
        }
    } else {
        if (L->dim > 256) return lb_fail(c, LB_ERR_INVALID, "layer %d: a recurrent head holds up to 256 key channels", i);
        if (L->decay == LB_DA_GLA && (!(L->tau > 0) || L->rank > 256)) return lb_fail(c, LB_ERR_INVALID, "layer %d: bad gate", i);
    }
    return LB_OK;
}

static int load_layer(lb_model* m, lb_weight_source* src, int i) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    const lb_stack_layer* D = &d->layer[i];
    st_layer* L = &S->L[i];
    const int W = d->width, Kw = S->Kw;
    st_part part[8];
    int np = 0, rows = 0;
    L->k_off = L->v_off = L->g_off = L->a1_off = -1;
#define SECTION(role, n, off)                                                          \
    do {                                                                               \
        part[np++] = (st_part){D->tensor[role], (n), W, rows, 1, 0};                   \
        (off) = rows;                                                                  \
        rows += (n);                                                                   \
    } while (0)
    const int nq = D->heads * D->dim;
    L->n_mix = D->heads * D->vdim;
    SECTION(LB_T_Q, nq, L->q_off);
    if (D->mixer == LB_MIX_ATTENTION) {
        if (D->kv_from < 0) {
            SECTION(LB_T_K, D->kv_heads * D->dim, L->k_off);
            SECTION(LB_T_V, D->kv_heads * D->vdim, L->v_off);
        }
    } else {
        SECTION(D->decay == LB_DA_HGRN2 ? LB_T_F : LB_T_K, nq, L->k_off);
        SECTION(LB_T_V, L->n_mix, L->v_off);
        if (D->decay == LB_DA_GLA) {
            SECTION(LB_T_G, L->n_mix, L->g_off);
            SECTION(LB_T_A1, D->rank, L->a1_off);
        }
    }
#undef SECTION
    LB_TRY(build_mat(m, src, &L->in, rows, Kw, part, np));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_NORM1], 1, W, &L->norm1, 0.f, 0.02f));
    L->n_mix_pad = pad_to(L->n_mix, 64);
    const int ff_pad = pad_to(D->ff, 64);
    if (D->ff) {
        const st_part gu[2] = {{D->tensor[LB_T_FF_GATE], D->ff, W, 0, 2, 0}, {D->tensor[LB_T_FF_UP], D->ff, W, 1, 2, 0}};
        LB_TRY(build_mat(m, src, &L->ff, 2 * D->ff, Kw, gu, 2));
        LB_TRY(load_vec(m, src, D->tensor[LB_T_NORM2], 1, W, &L->norm2, 0.f, 0.02f));
    }
    const st_part ou[2] = {{D->tensor[LB_T_O], W, L->n_mix, 0, 1, 0}, {D->tensor[LB_T_FF_DOWN], W, D->ff, 0, 1, L->n_mix_pad}};
    LB_TRY(build_mat(m, src, &L->out, W, L->n_mix_pad + ff_pad, ou, D->ff ? 2 : 1));
    if (D->mixer == LB_MIX_ATTENTION) {
        L->dim_p = pad_to(D->dim, 16);
        L->vdim_p = pad_to(D->vdim, 16);
        if (D->kv_from < 0) {
            const size_t rows_kv = (size_t)d->max_ctx * D->kv_heads;
            LB_TRY(lb_dalloc(m, &L->k_cache, rows_kv * L->dim_p * S->esz));
            LB_TRY(lb_dalloc(m, &L->v_cache, rows_kv * L->vdim_p * S->esz));
            LB_CU(m->c, lb_drv.MemsetD8Async(L->k_cache, 0, rows_kv * L->dim_p * S->esz, m->c->stream)); /* padding columns stay zero */
            LB_CU(m->c, lb_drv.MemsetD8Async(L->v_cache, 0, rows_kv * L->vdim_p * S->esz, m->c->stream));
        } else {
            L->k_cache = S->L[D->kv_from].k_cache;
            L->v_cache = S->L[D->kv_from].v_cache;
        }
        LB_TRY(upload_freqs(m, &L->freq_k, D->rot_dims, D->rot_base));
        if (D->v_rot) LB_TRY(upload_freqs(m, &L->freq_v, D->vdim, D->rot_base));
    } else {
        const size_t sb = (size_t)D->heads * D->dim * D->vdim * 4;
        L->dk_p = D->dim <= 64 ? 64 : D->dim <= 128 ? 128 : 256;
        LB_TRY(lb_dalloc(m, &L->state, sb));
        LB_TRY(load_vec(m, src, D->tensor[LB_T_HEAD_NORM], 1, D->vdim, &L->head_norm, 1.f, 0.02f));
        LB_TRY(load_vec(m, src, D->tensor[LB_T_GATE_BIAS], 1, nq, &L->bias, 2.f, 1.f));
        if (D->decay == LB_DA_HGRN2) LB_TRY(load_vec(m, src, D->tensor[LB_T_LOWER], 1, nq, &L->lower, 0.4f, 0.2f));
        else LB_TRY(load_vec(m, src, D->tensor[LB_T_A2], nq, D->rank, &L->a2, 0.f, 1.0f / sqrtf((float)D->rank)));
    }
    return LB_OK;
}

/* ---- kernel choice and launch blocks ----------------------------------------------------------------------------- */
static int heads_per_cta(const lb_stack_layer* D) { const int G = D->heads / D->kv_heads; return G <= 2 ? 2 : G <= 4 ? 4 : 8; }
static int head_groups(const lb_stack_layer* D) { const int G = D->heads / D->kv_heads, g = heads_per_cta(D); return (G + g - 1) / g; }

static int rows_smem(int gh, int warps, int dim_p, int vdim_p, int esz) { /* as wattn_rows lays it out */
    return gh * dim_p * 4 + warps * gh * vdim_p * 4 + (dim_p + vdim_p) * esz + warps * 32 * ((dim_p + vdim_p) * esz + 32);
}
static int rows_warps(const stack_t* S, const lb_stack_layer* D, int dim_p, int vdim_p) { /* 4, or as many as shared memory holds tiles for */
    int w = 4;
    while (w > 1 && rows_smem(heads_per_cta(D), w, dim_p, vdim_p, S->esz) > 200 * 1024) w--;
    return w;
}

static void fill_wattn(const lb_model* m, int i, lb_wattn_params* p, CUdeviceptr proj) {
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    memset(p, 0, sizeof *p);
    p->proj = (const float*)proj; p->ld = L->in.rows;
    p->k_cache = (void*)L->k_cache; p->v_cache = (void*)L->v_cache;
    p->freq_k = (const double*)L->freq_k; p->freq_v = (const double*)L->freq_v;
    p->q_off = L->q_off; p->k_off = L->k_off; p->v_off = L->v_off;
    p->H = D->heads; p->KV = D->kv_heads; p->dim = D->dim; p->vdim = D->vdim; p->dim_p = L->dim_p; p->vdim_p = L->vdim_p;
    p->rot_dims = D->rot_dims; p->block = D->block; p->v_norm = D->v_norm; p->sink = D->sink;
    p->max_ctx = S->d.max_ctx; p->splits = 1; p->T = 1;
    p->scale = (float)D->scale; p->eps = (float)S->d.eps;
    p->scratch = (float*)S->scratch; p->counters = (uint32_t*)S->counters;
    p->status = (uint32_t*)m->c->dev_status;
}
static int launch_wattn_rows(lb_model* m, int i, const lb_wattn_params* p) {
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const int gh = heads_per_cta(D), wide = p->vdim_p > 128, f32 = S->esz == 4;
    static const int k[2][2][3] = {{{LBK_wattn_rows_b2n2, LBK_wattn_rows_b4n2, LBK_wattn_rows_b8n2}, {LBK_wattn_rows_b2n4, LBK_wattn_rows_b4n4, LBK_wattn_rows_b8n4}},
                                   {{LBK_wattn_rows_f2n2, LBK_wattn_rows_f4n2, LBK_wattn_rows_f8n2}, {LBK_wattn_rows_f2n4, LBK_wattn_rows_f4n4, LBK_wattn_rows_f8n4}}};
    const int warps = rows_warps(S, D, p->dim_p, p->vdim_p);
    const unsigned smem = (unsigned)rows_smem(gh, warps, p->dim_p, p->vdim_p, S->esz);
    void* params[] = {(void*)p};
    return lb_launch(m->c, k[f32][wide][gh == 2 ? 0 : gh == 4 ? 1 : 2], (unsigned)(D->kv_heads * head_groups(D)), (unsigned)p->splits, (unsigned)p->T, (unsigned)(32 * warps), smem, params, 1);
}

static void fill_decay(const lb_model* m, int i, lb_decay_params2* p, CUdeviceptr proj) {
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    memset(p, 0, sizeof *p);
    p->proj = (const float*)proj; p->ld = L->in.rows;
    p->a2 = (const uint16_t*)L->a2; p->bias = (const uint16_t*)L->bias; p->lower = (const uint16_t*)L->lower; p->head_w = (const uint16_t*)L->head_norm;
    p->state = (float*)L->state;
    p->kind = D->decay; p->q_off = L->q_off; p->k_off = L->k_off; p->v_off = L->v_off; p->g_off = L->g_off; p->a1_off = L->a1_off; p->rank = D->rank;
    p->H = D->heads; p->dk = D->dim; p->dv = D->vdim; p->dk_p = L->dk_p; p->T = 1;
    p->q_scale = (float)(1.0 / sqrt((double)D->dim)); p->inv_tau = D->decay == LB_DA_GLA ? (float)(1.0 / D->tau) : 0.f; p->eps = (float)S->d.eps;
}

/* one launch of rows_gemv: ring depth and row splitting from what shared memory holds; two CTAs per row where one vector would leave the
 * ring fewer than five stages (the mixer's part must lie in the first half) */
static int launch_rows(lb_model* m, lb_rows_gemv_params* p) {
    lb_ctx* c = m->c;
    int P = 0;
    for (int i = 0; i < p->n_mat; i++) P += (p->mat[i].rows + 1) / 2;
    const int n_vec = p->x_mode == LB_RG_X_NORM ? p->n_mat : 1, limit = c->max_smem_optin - ((c->fn_static_smem[LBK_rows_gemv] + 1023) & ~1023);
    p->segs = (p->K + LB_RG_SEG - 1) / LB_RG_SEG;
    p->status = (uint32_t*)c->dev_status;
    const int can_halve = p->x_mode == LB_RG_X_CAT && p->n_mix_pad <= p->segs / 2 * LB_RG_SEG && c->sm_count % 2 == 0;
    size_t smem = 0;
    int ks = 1;
    for (ks = 1; ks <= 1 + can_halve; ks++) {
        const int ctas = c->sm_count / ks, max_pairs = (P + ctas - 1) / ctas, segs = (p->segs + ks - 1) / ks;
        p->x_cols = ks == 1 ? p->K : segs * LB_RG_SEG;
        p->split = max_pairs >= 64 ? 1 : segs;
        for (p->stages = 5; p->stages >= 1; p->stages--) {
            smem = (size_t)LB_RG_WARPS * p->stages * LB_RG_SEG * 4 + (size_t)n_vec * p->x_cols * 4 + (p->gate ? (size_t)((p->n_mix + 3) & ~3) * 4 : 0) +
                   (size_t)2 * max_pairs * p->split * 4 + 40 * 4 + ((size_t)LB_RG_WARPS * p->stages + 1) * 8;
            if ((int)smem <= limit) break;
        }
        if (p->stages == 5) break;
    }
    if (ks > 1 + can_halve) ks = 1 + can_halve;
    if (p->stages < 1) return lb_fail(c, LB_ERR_INVALID, "model: a row of %d columns does not fit the decode step's shared memory", p->K);
    void* params[] = {p};
    return lb_launch_cluster(c, LBK_rows_gemv, (unsigned)(c->sm_count / ks), (unsigned)ks, 1, LB_RG_THREADS, (unsigned)smem, params, 1, (unsigned)ks);
}

/* Tokens per product tile, and what a product then costs in units of one wave of 256-token tiles: fewer tokens per tile make more tiles
 * for narrow matrices, at a lower rate per tile (measured: the operands' trip through shared memory bounds small tiles). */
static double product_cost(const lb_ctx* c, int row_tiles, int T, int* nt_out) {
    static const struct { int nt; double cost; } k[] = {{256, 1.0}, {128, 0.55}, {64, 0.38}, {32, 0.34}, {16, 0.33}};
    double best = 1e30;
    for (int i = 0; i < 5; i++) {
        const int tiles = row_tiles * ((T + k[i].nt - 1) / k[i].nt);
        const double v = (double)((tiles + c->sm_count - 1) / c->sm_count) * k[i].cost;
        if (v < best) { best = v; *nt_out = k[i].nt; }
    }
    return best;
}

/* one or two products Y = X W^T of a chunk (w[1] may be NULL) */
typedef struct { const st_mat* w; CUdeviceptr x; CUdeviceptr y; int y_mode, ld_y; } st_prod;
static int launch_products(lb_model* m, const st_prod* pr, int n, int T) {
    lb_ctx* c = m->c;
    const stack_t* S = S_of(m);
    lb_dgemm_params p;
    memset(&p, 0, sizeof p);
    p.T = T; p.K = pr[0].w->K; p.ld_x = p.K;
    p.mult = (float)S->d.residual_mult; p.cap = (float)S->d.logit_softcap;
    p.status = (uint32_t*)c->dev_status;
    for (int i = 0; i < n; i++) {
        p.rows[i] = pr[i].w->rows; p.w[i] = (const uint16_t*)pr[i].w->w; p.x[i] = (const void*)pr[i].x;
        p.y[i] = (void*)pr[i].y; p.y_mode[i] = pr[i].y_mode; p.ld_y[i] = pr[i].ld_y; p.y_f32[i] = S->esz == 4;
        p.tiles[i] = (p.rows[i] + LB_DG_ROWS - 1) / LB_DG_ROWS;
    }
    product_cost(c, p.tiles[0] + p.tiles[1], T, &p.NT);
    p.t_tiles = (T + p.NT - 1) / p.NT;
    void* params[] = {&p};
    if (S->esz == 4)
        return lb_launch(c, LBK_gemm_f32_simt, (unsigned)((p.rows[0] + 63) / 64 + (p.rows[1] + 63) / 64), (unsigned)((T + 63) / 64), 1, 256, 0, params, 1);
    for (int i = 0; i < n; i++) {
        CUtensorMap tm;
        memcpy(p.tmap_w[i], &pr[i].w->tmap, sizeof tm);
        LB_TRY(map_rows(c, &tm, pr[i].x, T, p.K, p.NT));
        memcpy(p.tmap_x[i], &tm, sizeof tm);
    }
    const int stage = LB_DG_ROWS * LB_DG_KB * 2 + p.NT * LB_DG_KB * 2;
    p.stages = 200 * 1024 / stage;
    if (p.stages > LB_DG_MAX_STAGES) p.stages = LB_DG_MAX_STAGES;
    p.tmem_cols = 2 * p.NT < 32 ? 32 : 2 * p.NT;
    const int tiles = (p.tiles[0] + p.tiles[1]) * p.t_tiles;
    return lb_launch(c, LBK_gemm_bf16_tc, (unsigned)(tiles < c->sm_count ? tiles : c->sm_count), 1, 1, LB_DG_THREADS, (unsigned)(p.stages * stage), params, 1);
}

/* ---- the decode step ------------------------------------------------------------------------------------------------ */
static int stack_step_layers(lb_model* m) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    for (int i = 0; i < d->n_layers; i++) {
        const lb_stack_layer* D = &d->layer[i];
        const st_layer* L = &S->L[i];
        lb_rows_gemv_params g;
        memset(&g, 0, sizeof g);
        g.x_mode = LB_RG_X_NORM; g.x = (const float*)m->X; g.width = d->width; g.K = S->Kw; g.eps = (float)d->eps;
        g.n_mat = D->ff ? 2 : 1;
        g.mat[0] = (lb_rg_mat){(const uint16_t*)L->in.w, (const uint16_t*)L->norm1, (float*)S->proj, L->in.rows, LB_DY_STORE};
        if (D->ff) g.mat[1] = (lb_rg_mat){(const uint16_t*)L->ff.w, (const uint16_t*)L->norm2, (float*)S->act, L->ff.rows, LB_DY_RELU_GLU};
        LB_TRY(launch_rows(m, &g));
        memset(&g, 0, sizeof g);
        if (D->mixer == LB_MIX_ATTENTION) {
            lb_wattn_params p;
            fill_wattn(m, i, &p, S->proj);
            p.out = (float*)S->mix; p.pos_ptr = (const int32_t*)m->d_pos; p.splits = L->splits;
            LB_TRY(launch_wattn_rows(m, i, &p));
        } else {
            lb_decay_params2 p;
            fill_decay(m, i, &p, S->proj);
            p.o = (float*)S->mix;
            void* params[] = {&p};
            LB_TRY(lb_launch(m->c, L->dk_p == 64 ? LBK_da_step_64 : L->dk_p == 128 ? LBK_da_step_128 : LBK_da_step_256, (unsigned)D->heads,
                             (unsigned)((D->vdim + 31) / 32), 1, 128, D->decay == LB_DA_GLA ? (unsigned)(D->dim * D->rank * 2) : 0u, params, 1));
            g.head_w = (const uint16_t*)L->head_norm; g.vdim = D->vdim;
            if (L->g_off >= 0) g.gate = (const float*)(S->proj + (size_t)L->g_off * 4);
        }
        g.x_mode = LB_RG_X_CAT; g.K = L->out.K; g.eps = (float)d->eps; g.mult = (float)d->residual_mult; g.n_mat = 1;
        g.mix = (const float*)S->mix; g.n_mix = L->n_mix; g.n_mix_pad = L->n_mix_pad; g.act = (const float*)S->act; g.n_act = D->ff;
        g.mat[0] = (lb_rg_mat){(const uint16_t*)L->out.w, NULL, (float*)m->X, L->out.rows, LB_DY_RESIDUAL};
        LB_TRY(launch_rows(m, &g));
    }
    return LB_OK;
}

static int stack_head(lb_model* m, CUdeviceptr x_row) {
    const stack_t* S = S_of(m);
    lb_rows_gemv_params g;
    memset(&g, 0, sizeof g);
    g.x_mode = LB_RG_X_NORM; g.x = (const float*)x_row; g.width = S->d.width; g.K = S->Kw; g.eps = (float)S->d.eps; g.cap = (float)S->d.logit_softcap;
    g.n_mat = 1;
    g.mat[0] = (lb_rg_mat){(const uint16_t*)S->head.w, (const uint16_t*)m->final_norm, (float*)m->logits, S->head.rows, LB_DY_SOFTCAP};
    g.part_val = (float*)m->cand_val; g.part_idx = (int32_t*)m->cand_idx;
    return launch_rows(m, &g);
}
static int stack_head_ctas(lb_model* m) { return m->c->sm_count; }

/* ---- a prompt chunk --------------------------------------------------------------------------------------------------- */
static int norm_rows(lb_model* m, CUdeviceptr x, CUdeviceptr w0, CUdeviceptr h0, CUdeviceptr w1, CUdeviceptr h1, int T) {
    const stack_t* S = S_of(m);
    lb_norm2_params p;
    memset(&p, 0, sizeof p);
    p.x = (const float*)x; p.w[0] = (const uint16_t*)w0; p.h[0] = (void*)h0; p.w[1] = (const uint16_t*)w1; p.h[1] = (void*)h1;
    p.width = S->d.width; p.ld = S->Kw; p.f32 = S->esz == 4; p.eps = (float)S->d.eps;
    void* params[] = {&p};
    return lb_launch(m->c, LBK_norm_rows2, (unsigned)T, 1, 1, 256, 0, params, 1);
}

static int stack_pf_layer(lb_model* m, pf_set* w, int i, int pos0, int T) {
    lb_ctx* c = m->c;
    stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    const int f32 = S->esz == 4;
    LB_TRY(norm_rows(m, w->st.X, L->norm1, w->st.h1, D->ff ? L->norm2 : 0, D->ff ? w->st.h2 : 0, T));
    st_prod pr[2] = {{&L->in, w->st.h1, w->st.proj, LB_DY_STORE, L->in.rows},
                     {&L->ff, w->st.h2, w->st.cat + (size_t)L->n_mix_pad * S->esz, LB_DY_RELU_GLU, L->out.K}};
    LB_TRY(launch_products(m, pr, D->ff ? 2 : 1, T));
    if (D->mixer == LB_MIX_ATTENTION) {
        lb_wattn_params p;
        fill_wattn(m, i, &p, w->st.proj);
        p.pos0 = pos0; p.T = T; p.cat = (void*)w->st.cat; p.cat_ld = L->out.K;
        void* params[] = {&p};
        if (f32) {
            if (L->k_off >= 0) LB_TRY(lb_launch(c, LBK_wattn_prepare_f32, (unsigned)T, 1, 1, 256, 0, params, 1));
            p.k_off = -1; /* the chunk's rows are in the cache */
            LB_TRY(launch_wattn_rows(m, i, &p));
        } else {
            p.qh = (uint16_t*)w->st.q; p.ql = (uint16_t*)w->st.k;
            LB_TRY(lb_launch(c, LBK_wattn_prepare_bf16, (unsigned)T, 1, 1, 256, 0, params, 1));
            const int rows = T * (D->heads / D->kv_heads);
            const unsigned smem = (unsigned)(2 * LB_WA_ROWS * (2 * L->dim_p + 16) + 2 * LB_WA_KV * (2 * L->dim_p + 2 * L->vdim_p + 32));
            LB_TRY(lb_launch(c, L->vdim_p <= 64 ? LBK_wattn_chunk_64 : L->vdim_p <= 128 ? LBK_wattn_chunk_128 : LBK_wattn_chunk_256,
                             (unsigned)((rows + LB_WA_ROWS - 1) / LB_WA_ROWS), (unsigned)D->kv_heads, 1, LB_WA_THREADS, smem, params, 1));
        }
    } else {
        lb_decay_params2 p;
        fill_decay(m, i, &p, w->st.proj);
        p.T = T; p.q = (float*)w->st.q; p.k = (float*)w->st.k; p.a = (float*)w->st.a; p.o = (float*)w->st.o;
        p.cat = (void*)w->st.cat; p.cat_ld = L->out.K; p.cat_f32 = f32;
        void* params[] = {&p};
        LB_TRY(lb_launch(c, LBK_da_inputs, (unsigned)((D->heads * L->dk_p + 255) / 256), (unsigned)((T + 7) / 8), 1, 256, (unsigned)(8 * (D->rank > 0 ? D->rank : 1) * 4), params, 1));
        const int part = L->dk_p / 16, tok = 3 * 16 * (part == 4 ? 4 : part + 4) + 64; /* floats a token's operands take in a stage */
        const int dki = L->dk_p == 64 ? 0 : L->dk_p == 128 ? 1 : 2;
        static const int k_scan[3] = {LBK_da_scan_64, LBK_da_scan_128, LBK_da_scan_256}, k_local[3] = {LBK_da_local_64, LBK_da_local_128, LBK_da_local_256};
        const unsigned slabs = (unsigned)((D->vdim + 63) / 64), threads = dki == 2 ? 256 : 128, smem = (unsigned)(3 * 4 * tok * 4), segs = (unsigned)((T + ST_SEG - 1) / ST_SEG);
        p.seg = ST_SEG; p.seg_state = (float*)w->st.seg_state; p.seg_decay = (float*)w->st.seg_decay;
        if (segs > 1) LB_TRY(lb_launch(c, k_local[dki], (unsigned)D->heads, slabs, segs, threads, smem, params, 1));
        LB_TRY(lb_launch(c, k_scan[dki], (unsigned)D->heads, slabs, segs, threads, smem, params, 1));
        LB_TRY(lb_launch(c, LBK_da_finish, (unsigned)T, (unsigned)((D->heads + 3) / 4), 1, 128, 0, params, 1));
    }
    const st_prod out = {&L->out, w->st.cat, w->st.X, LB_DY_RESIDUAL, S->d.width};
    return launch_products(m, &out, 1, T);
}

static int stack_head_rows(lb_model* m, CUdeviceptr rows, int n, CUdeviceptr logits) {
    stack_t* S = S_of(m);
    pf_set* w = lb_prefill_set(m, 0); /* the chunk streams have been joined: their buffers are free */
    LB_TRY(norm_rows(m, rows, m->final_norm, w->st.h1, 0, 0, n));
    const st_prod pr = {&S->head, w->st.h1, logits, LB_DY_SOFTCAP, S->head.rows};
    return launch_products(m, &pr, 1, n);
}

static void stack_pf_sizes(const lb_model* m, size_t bytes[LB_PF_MAX_BUFS]) {
    const stack_t* S = S_of(m);
    const size_t T = (size_t)m->pf_chunk, e = (size_t)S->esz, q = (size_t)S->max_dk * 4 > (size_t)S->max_q * 2 ? (size_t)S->max_dk * 4 : (size_t)S->max_q * 2;
    const size_t b[] = {T * (size_t)S->d.width * 4, T * (size_t)S->Kw * e, T * (size_t)S->Kw * e, T * (size_t)S->max_in * 4, T * (size_t)S->max_cat * e,
                        T * q, T * q, T * (size_t)S->max_dk * 4, T * (size_t)S->max_o * 4,
                        (T + ST_SEG - 1) / ST_SEG * S->max_state, (T + ST_SEG - 1) / ST_SEG * (size_t)S->max_dk * 4};
    memcpy(bytes, b, sizeof b); /* in the order of pf_set.st */
}

/* ---- state ---------------------------------------------------------------------------------------------------------------- */
static int stack_reset_state(lb_model* m) { /* cache rows past the position are never read: only the recurrent states start over */
    const stack_t* S = S_of(m);
    for (int i = 0; i < S->d.n_layers; i++)
        if (S->L[i].state) LB_CU(m->c, lb_drv.MemsetD8Async(S->L[i].state, 0, state_bytes(&S->d.layer[i]), m->c->stream));
    return LB_OK;
}
static int stack_snapshot(lb_model* m, int restore) {
    lb_ctx* c = m->c;
    stack_t* S = S_of(m);
    for (int i = 0; i < S->d.n_layers; i++) {
        st_layer* L = &S->L[i];
        if (!L->state) continue;
        const size_t n = state_bytes(&S->d.layer[i]);
        if (!L->snap) {
            if (restore) return lb_fail(c, LB_ERR_STATE, "lb_model_rollback: no checkpoint taken");
            LB_TRY(lb_dalloc(m, &L->snap, n));
        }
        LB_CU(c, lb_drv.MemcpyDtoDAsync(restore ? L->state : L->snap, restore ? L->snap : L->state, n, c->stream));
    }
    return LB_OK;
}
static int stack_state_ptr(lb_model* m, int i, int which, uint64_t* dptr, size_t* bytes) {
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    if (D->mixer == LB_MIX_ATTENTION) {
        *dptr = which ? L->v_cache : L->k_cache;
        *bytes = (size_t)S->d.max_ctx * D->kv_heads * (which ? L->vdim_p : L->dim_p) * S->esz;
    } else {
        if (which) return lb_fail(m->c, LB_ERR_INVALID, "layer %d has one state buffer", i);
        *dptr = L->state;
        *bytes = state_bytes(D);
    }
    return LB_OK;
}

static void stack_destroy(lb_model* m) {
    stack_t* S = S_of(m);
    if (!S) return;
    for (int i = 0; S->L && i < S->d.n_layers; i++) {
        st_layer* L = &S->L[i];
        const int own = S->d.layer[i].kv_from < 0;
        CUdeviceptr p[] = {L->in.w, L->ff.w, L->out.w, L->norm1, L->norm2, L->a2, L->bias, L->lower, L->head_norm, own ? L->k_cache : 0, own ? L->v_cache : 0,
                           L->freq_k, L->freq_v, L->state, L->snap};
        for (size_t k = 0; k < sizeof p / sizeof p[0]; k++) if (p[k]) lb_drv.MemFree(p[k]);
    }
    CUdeviceptr g[] = {S->head.w, S->proj, S->mix, S->act, S->scratch, S->counters};
    for (size_t k = 0; k < sizeof g / sizeof g[0]; k++) if (g[k]) lb_drv.MemFree(g[k]);
    free(S->L);
    free(S->d.layer);
    S->L = NULL;
    S->d.layer = NULL;
}

static const lb_arch k_stack = {"stack", ST_STREAMS, stack_reset_state, stack_snapshot, stack_state_ptr, stack_step_layers, stack_head,
                                stack_head_ctas, stack_head_rows, stack_pf_sizes, stack_pf_layer, stack_destroy};

/* tokens per prompt chunk: the multiple of 256 whose products fill whole waves of SMs best */
static int stack_chunk(const lb_model* m) {
    const stack_t* S = S_of(m);
    double best = 1e30;
    int chunk = 256;
    for (int T = 256; T <= ST_CHUNK; T += 256) {
        double cost = 0;
        for (int i = 0; i < S->d.n_layers; i++) {
            const st_layer* L = &S->L[i];
            int nt;
            cost += L->in.K * product_cost(m->c, (L->in.rows + LB_DG_ROWS - 1) / LB_DG_ROWS + (L->ff.rows + LB_DG_ROWS - 1) / LB_DG_ROWS, T, &nt) +
                    L->out.K * product_cost(m->c, (L->out.rows + LB_DG_ROWS - 1) / LB_DG_ROWS, T, &nt);
        }
        cost /= T;
        if (T < 512) cost *= 1.05; /* weights read once per chunk */
        if (cost < best * 0.999) { best = cost; chunk = T; }
    }
    return chunk;
}

static int stack_build(lb_model* m, const lb_stack_desc* d, lb_weight_source* src) {
    lb_ctx* c = m->c;
    stack_t* S = S_of(m);
    LB_CU(c, lb_drv.CtxSetCurrent(c->cu_ctx));
    S->d = *d;
    S->d.layer = (lb_stack_layer*)malloc((size_t)d->n_layers * sizeof *d->layer);
    S->L = (st_layer*)calloc((size_t)d->n_layers, sizeof *S->L);
    if (!S->d.layer || !S->L) return LB_ERR_NOMEM;
    memcpy(S->d.layer, d->layer, (size_t)d->n_layers * sizeof *d->layer);
    S->Kw = pad_to(d->width, 64);
    S->esz = d->dtype == LB_DTYPE_F32 ? 4 : 2;
    m->cfg.n_layers = d->n_layers; m->cfg.hidden = d->width; m->cfg.vocab = d->vocab; m->cfg.max_ctx = d->max_ctx; m->cfg.eps = (float)d->eps;
    m->tp_size = 1; m->vocab_s = d->vocab;
    for (int i = 0; i < d->n_layers; i++) LB_TRY(check_layer(c, d, i));
    LB_TRY(lb_model_alloc_common(m));
    size_t scratch = 0;
    int groups_max = 1;
    for (int i = 0; i < d->n_layers; i++) {
        const lb_stack_layer* D = &d->layer[i];
        st_layer* L = &S->L[i];
        LB_TRY(load_layer(m, src, i));
#define MAX(a, b) do { if ((b) > (a)) (a) = (b); } while (0)
        MAX(S->max_in, L->in.rows); MAX(S->max_cat, L->out.K); MAX(S->max_mix, L->n_mix); MAX(S->max_ff, D->ff);
        if (D->mixer == LB_MIX_ATTENTION) {
            MAX(S->max_q, D->heads * L->dim_p);
            /* slices of the decode attention: one tile of 32 rows per warp each, as many as keep one CTA per SM */
            const int groups = D->kv_heads * head_groups(D), seen = D->block && D->block < d->max_ctx ? D->block : d->max_ctx;
            const int slice = 32 * rows_warps(S, D, L->dim_p, L->vdim_p);
            L->splits = (seen + slice - 1) / slice;
            if (L->splits > LB_WA_MAX_SPLITS) L->splits = LB_WA_MAX_SPLITS;
            if (L->splits * groups > c->sm_count) L->splits = c->sm_count / groups;
            if (L->splits < 1) L->splits = 1;
            const size_t n = (size_t)groups * L->splits * heads_per_cta(D) * (L->vdim_p + 2) * 4;
            if (n > scratch) scratch = n;
            MAX(groups_max, groups);
        } else {
            MAX(S->max_dk, D->heads * L->dk_p);
            MAX(S->max_state, state_bytes(D));
            MAX(S->max_o, D->heads * D->vdim);
        }
#undef MAX
    }
    uint16_t* e = (uint16_t*)malloc((size_t)d->vocab * d->width * 2);
    if (!e) return lb_fail(c, LB_ERR_NOMEM, "model: host staging");
    int st = read_rows(c, src, d->embed, d->vocab, d->width, e, (size_t)d->width, 0.f, 1.f);
    if (st == LB_OK) st = lb_upload(m, &m->embed, e, (size_t)d->vocab * d->width * 2);
    free(e);
    LB_TRY(st);
    const st_part hp = {d->head, d->vocab, d->width, 0, 1, 0};
    LB_TRY(build_mat(m, src, &S->head, d->vocab, S->Kw, &hp, 1));
    LB_TRY(load_vec(m, src, d->final_norm, 1, d->width, &m->final_norm, 0.f, 0.02f));
    LB_TRY(lb_dalloc(m, &S->proj, (size_t)S->max_in * 4));
    LB_TRY(lb_dalloc(m, &S->mix, (size_t)S->max_mix * 4));
    LB_TRY(lb_dalloc(m, &S->act, (size_t)(S->max_ff ? S->max_ff : 1) * 4));
    LB_TRY(lb_dalloc(m, &S->scratch, scratch));
    LB_TRY(lb_dalloc(m, &S->counters, (size_t)groups_max * 4));
    LB_CU(c, lb_drv.MemsetD8Async(S->counters, 0, (size_t)groups_max * 4, c->stream));
    m->globals_loaded = 1;
    m->pf_chunk = stack_chunk(m);
    return lb_model_reset_state(m);
}

int lb_stack_create(lb_ctx* c, const lb_stack_desc* d, const lb_weight_source* src, lb_model** out) {
    lb_model* m = (lb_model*)calloc(1, sizeof *m);
    stack_t* S = (stack_t*)calloc(1, sizeof *S);
    if (!m || !S) { free(m); free(S); return LB_ERR_NOMEM; }
    m->c = c; m->arch = &k_stack; m->impl = S; m->tp_size = 1;
    *out = m;
    lb_weight_source s = *src;
    return stack_build(m, d, &s);
}
