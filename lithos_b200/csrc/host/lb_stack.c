/* Models described by a list of layers (lb_stack.h): weights, caches and states, the decode step and a prompt chunk.
 *
 * A layer whose two sides read the same row: x += m (mixer(norm1 x) + feed-forward(norm2 x)).  The projections of both sides read the same row, and the two output
 * projections add into the same row, so a layer of the decode step is three launches:
 *   [both norms + mixer's input projections | gate, up projections + ReLU gating]   rows_gemv, two matrices
 *   [mixer: rotations, cache append, attention over the cache | gates, state update, read-out]   wattn_rows_* | da_step_*
 *   [per-head norm and gate + (W_o | W_down) as one matrix over (mixer, feed-forward) + residual]   rows_gemv, one matrix
 * and of a prompt chunk: norm_rows2, one product launch for all input projections, the mixer's kernels, one product launch for the
 * outputs (gemm_bf16_tc, tcgen05; gemm_f32_simt when the model runs in fp32).
 * A serial layer (x += m mixer(norm1 x), then x += m ff(norm2 x)) runs the same kernels side by side of one another's product: the mixer's input
 * products, the mixer, W_o + residual, then the feed-forward's two products.  Experts are one matrix stacked by expert: a decode step reads the
 * chosen ones' rows (and columns) only; a prompt chunk sorts its (token, expert) assignments by expert, multiplies tile by tile of one expert's
 * tokens, and the next norm adds a token's results to its residual row.
 *
 * Device layout: the mixer's input projections are stacked along rows ([q | k | v], [q | f | v], [q | k | v | g | a1]); gate and up rows
 * alternate; W_o and W_down stand side by side.  Columns are padded to a multiple of 64 with zeros, so any size is a whole number of
 * 128-byte operand rows.  Caches hold max_ctx rows [kv_heads, dim rounded up to 16] per attention layer that has keys of its own, rows [latent rounded up to 64 | shared key part rounded up to
 * 16] per latent attention layer; a state-space layer has its state and the last inputs of its convolution.
 */
#include "lb_model_priv.h"
#include "lb_safetensors.h"
#include "lb_stack.h"
#include <math.h>

#define ST_CHUNK 1024 /* largest chunk of a prompt; stack_chunk picks the model's */
#define ST_CHUNK_EXPERTS 2048 /* ... where the weights of experts are read once per chunk */
#define ST_STREAMS 4
#define ST_LAT_ABSORB 16 /* latent attention: portions of fewer tokens do not make keys and values of every cached position */
#define ST_MOE_TILE 64 /* token tile of the fp32 expert products */
#define ST_SSM_SEGS 8  /* most segments of a chunk through a state-space recurrence */
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
    /* serial layers */
    st_mat down, uq, uk, uv; /* feed-forward output; latent attention's second query product, keys and values of the latent */
    CUdeviceptr norm1_b, norm2_b, cq_norm, c_norm, sink, conv, conv_b, dt_bias, a_log, dskip, table;
    CUdeviceptr ring, snap_ring; /* last inputs of the convolution */
    int ff_p, q_rank_p, rank_p, rot_p, N_p, V_p;
    float rot_mul;
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
    /* serial layers */
    CUdeviceptr final_b, lq, lat_q, lat_part;
    int max_h2, max_lq, max_latq, max_rec, max_xbc, max_heads, max_act, max_top, max_experts, max_actp; /* max_actp: act elements per token of a chunk */
    int max_kx, max_vx, max_part_rows; /* expanded keys / values per position; slices x rows of a decode step or a short portion */
    int lat_full;                      /* a chunk may take the absorbed way whatever its length */
} stack_t;

static size_t state_bytes(const lb_stack_layer* D) { return (size_t)D->heads * (D->mixer == LB_MIX_SSM ? D->state : D->dim) * D->vdim * 4; }
static int conv_channels(const lb_stack_layer* D) { return D->heads * D->vdim + 2 * D->groups * D->state; }
static size_t ring_bytes(const lb_stack_layer* D) { return (size_t)D->taps * conv_channels(D) * 4; }
static int pad_to(int n, int m) { return (n + m - 1) / m * m; }
static stack_t* S_of(const lb_model* m) { return (stack_t*)m->impl; }

/* ---- configuration ------------------------------------------------------------------------------------------ */
int lb_cfg_int(lb_ctx* c, const lb_json* j, const char* key, int lo, int hi, int layer, int* out) {
    const double v = lb_json_num(j, key, NAN);
    if (!(v >= lo && v <= hi) || v != floor(v)) return lb_fail(c, LB_ERR_INVALID, "config: layer %d: '%s' is missing or not an integer in [%d, %d]", layer, key, lo, hi);
    *out = (int)v;
    return LB_OK;
}
int lb_cfg_num(lb_ctx* c, const lb_json* j, const char* key, int layer, double* out) {
    *out = lb_json_num(j, key, NAN);
    if (!isfinite(*out)) return lb_fail(c, LB_ERR_INVALID, "config: layer %d: '%s' is missing or not a number", layer, key);
    return LB_OK;
}

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

/* the experts of every token id */
static int load_table(lb_model* m, lb_weight_source* src, const char* name, int vocab, int top, int experts, CUdeviceptr* out) {
    lb_ctx* c = m->c;
    const size_t n = (size_t)vocab * top;
    int32_t* h = (int32_t*)malloc(n * 4);
    if (!h) return lb_fail(c, LB_ERR_NOMEM, "model: host staging");
    int st = LB_OK;
    if (!src->files) {
        const uint64_t stream = ++src->stream;
        for (int v = 0; v < vocab; v++) { /* different experts: a random first one, then on by random steps that stay inside one round */
            int e = (int)(lb_rng_u64(src->seed, stream, (uint64_t)v * (uint64_t)top) % (uint64_t)experts), left = experts - top;
            for (int k = 0; k < top; k++) {
                h[(size_t)v * top + k] = e;
                const int step = left > 0 ? (int)(lb_rng_u64(src->seed, stream, (uint64_t)v * (uint64_t)top + (uint64_t)k + 1) % (uint64_t)(left + 1)) : 0;
                e = (e + 1 + step) % experts;
                left -= step;
            }
        }
    } else {
        const lb_st_tensor* t = lb_st_find((const lb_st_set*)src->files, name);
        if (!t || strcmp(t->dtype, "I32") || t->ndim != 2 || t->dim[0] != vocab || t->dim[1] != top || t->size != n * 4)
            st = lb_fail(c, LB_ERR_IO, "tensor %s is missing or not int32 [%d, %d]", name, vocab, top);
        else memcpy(h, t->data, n * 4);
        for (size_t i = 0; i < n && st == LB_OK; i++)
            if (h[i] < 0 || h[i] >= experts) st = lb_fail(c, LB_ERR_IO, "tensor %s names expert %d of %d", name, h[i], experts);
    }
    if (st == LB_OK) st = lb_upload(m, out, h, n * 4);
    free(h);
    return st;
}

/* a matrix whose rows are `ld` elements apart */
static int map_rows_ld(lb_ctx* c, CUtensorMap* tm, CUdeviceptr p, int rows, int K, int ld, int box_rows) {
    cuuint64_t dims[2] = {(cuuint64_t)K, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    cuuint32_t box[2] = {LB_DG_KB, (cuuint32_t)box_rows}, es[2] = {1, 1};
    LB_CU(c, lb_drv.TensorMapEncodeTiled(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void*)p, dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE));
    return LB_OK;
}
static int map_rows(lb_ctx* c, CUtensorMap* tm, CUdeviceptr p, int rows, int K, int box_rows) { return map_rows_ld(c, tm, p, rows, K, K, box_rows); }

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

/* YaRN: pairs that turn often over the original length keep their frequency, pairs that turn seldom are slowed down by `factor`, a ramp between
 * them; cosines and sines are scaled */
static int upload_yarn_freqs(lb_model* m, const lb_stack_layer* D, CUdeviceptr* out, float* mul) {
    const int dims = D->rot_dim;
    double f[LB_LA_MAX_ROT / 2], lo = 0, hi = 0;
    const double factor = D->yarn.factor;
    *mul = 1.f;
    if (factor > 0) {
        const double pi = 3.14159265358979323846, k = dims / (2.0 * log(D->rot_base));
        lo = floor(k * log(D->yarn.original / (2.0 * pi * D->yarn.fast)));
        hi = ceil(k * log(D->yarn.original / (2.0 * pi * D->yarn.slow)));
        if (lo < 0) lo = 0;
        if (hi > dims - 1) hi = dims - 1;
        *mul = (float)(0.1 * log(factor) + 1.0);
    }
    for (int i = 0; i < dims / 2; i++) {
        f[i] = pow(D->rot_base, -2.0 * i / dims);
        if (factor > 0) {
            double ramp = (i - lo) / (hi - lo > 0.001 ? hi - lo : 0.001);
            ramp = ramp < 0 ? 0 : ramp > 1 ? 1 : ramp;
            f[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp);
        }
    }
    return lb_upload(m, out, f, sizeof(double) * (size_t)(dims / 2));
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
    } else if (L->mixer == LB_MIX_LATENT) {
        if (L->kv_rank > LB_LA_MAX_RANK || L->dim > 256 || L->rot_dim > LB_LA_MAX_ROT || L->rot_dim % 2 || !(L->rot_base > 0) || L->rot_base == 1.0)
            return lb_fail(c, LB_ERR_INVALID, "layer %d: latent attention needs a latent of up to %d, head sizes up to 256 and an even rotated part of up to %d", i,
                           LB_LA_MAX_RANK, LB_LA_MAX_ROT);
    } else if (L->mixer == LB_MIX_SSM) {
        if (L->heads % L->groups || (L->heads * L->vdim) % L->norm_groups || L->state > LB_SSM_MAX_STATE || L->taps > LB_SSM_MAX_TAPS ||
            L->heads * L->vdim / L->norm_groups > 50000)
            return lb_fail(c, LB_ERR_INVALID, "layer %d: a state-space mixer needs heads a multiple of groups, channels a multiple of norm groups, up to %d state rows and %d taps",
                           i, LB_SSM_MAX_STATE, LB_SSM_MAX_TAPS);
    } else {
        if (L->dim > 256) return lb_fail(c, LB_ERR_INVALID, "layer %d: a recurrent head holds up to 256 key channels", i);
        if (L->decay == LB_DA_GLA && (!(L->tau > 0) || L->rank > 256)) return lb_fail(c, LB_ERR_INVALID, "layer %d: bad gate", i);
    }
    if (L->ff && L->ff_kind == LB_FF_EXPERTS && (L->experts > LB_MOE_MAX_EXPERTS || L->top > LB_RG_MAX_PARTS))
        return lb_fail(c, LB_ERR_INVALID, "layer %d: up to %d experts, %d of them per token", i, LB_MOE_MAX_EXPERTS, LB_RG_MAX_PARTS);
    return LB_OK;
}

/* feed-forward of a serial layer: [gate, up] pairs or up rows; the output matrix; experts stacked one after the other */
static int load_serial_ff(lb_model* m, lb_weight_source* src, int i) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    const lb_stack_layer* D = &d->layer[i];
    st_layer* L = &S->L[i];
    const int W = d->width, F = D->ff, W2 = pad_to(W, 2);
    L->ff_p = pad_to(F, 64);
    LB_TRY(load_vec(m, src, D->tensor[LB_T_NORM2], 1, W, &L->norm2, 1.f, 0.02f));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_NORM2_B], 1, W, &L->norm2_b, 0.f, 0.02f));
    if (D->ff_kind == LB_FF_RELU2) {
        const st_part up = {D->tensor[LB_T_FF_UP], F, W, 0, 1, 0}, down = {D->tensor[LB_T_FF_DOWN], W, F, 0, 1, 0};
        LB_TRY(build_mat(m, src, &L->ff, F, S->Kw, &up, 1));
        return build_mat(m, src, &L->down, W, L->ff_p, &down, 1);
    }
    const int E = D->experts;
    char(*name)[48] = (char(*)[48])malloc((size_t)E * 3 * 48);
    st_part* part = (st_part*)malloc((size_t)E * 3 * sizeof *part);
    int st = name && part ? LB_OK : LB_ERR_NOMEM;
    for (int e = 0; e < E && st == LB_OK; e++) {
        static const int role[3] = {LB_T_FF_GATE, LB_T_FF_UP, LB_T_FF_DOWN};
        for (int k = 0; k < 3; k++) snprintf(name[3 * e + k], 48, D->tensor[role[k]], e);
        part[2 * e] = (st_part){name[3 * e], F, W, 2 * F * e, 2, 0};
        part[2 * e + 1] = (st_part){name[3 * e + 1], F, W, 2 * F * e + 1, 2, 0};
        part[2 * E + e] = (st_part){name[3 * e + 2], W, F, W2 * e, 1, 0};
    }
    if (st == LB_OK) st = build_mat(m, src, &L->ff, 2 * F * E, S->Kw, part, 2 * E);
    if (st == LB_OK) st = build_mat(m, src, &L->down, W2 * E, L->ff_p, part + 2 * E, E);
    free(name);
    free(part);
    LB_TRY(st);
    return load_table(m, src, D->tensor[LB_T_TABLE], d->vocab, D->top, E, &L->table);
}

static int load_latent(lb_model* m, lb_weight_source* src, int i) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    const lb_stack_layer* D = &d->layer[i];
    st_layer* L = &S->L[i];
    const int W = d->width, H = D->heads;
    L->q_rank_p = pad_to(D->q_rank, 64);
    L->rank_p = pad_to(D->kv_rank, 64);
    L->rot_p = pad_to(D->rot_dim, 16);
    L->dim_p = pad_to(D->dim, 16);
    L->vdim_p = pad_to(D->vdim, 16);
    const st_part in[2] = {{D->tensor[LB_T_DQ], D->q_rank, W, 0, 1, 0}, {D->tensor[LB_T_DKV], D->kv_rank + D->rot_dim, W, D->q_rank, 1, 0}};
    const st_part uq = {D->tensor[LB_T_UQ], H * (D->dim + D->rot_dim), D->q_rank, 0, 1, 0}, uk = {D->tensor[LB_T_UK], H * D->dim, D->kv_rank, 0, 1, 0},
                  uv = {D->tensor[LB_T_UV], H * D->vdim, D->kv_rank, 0, 1, 0};
    L->q_off = 0;
    L->k_off = D->q_rank;
    LB_TRY(build_mat(m, src, &L->in, D->q_rank + D->kv_rank + D->rot_dim, S->Kw, in, 2));
    LB_TRY(build_mat(m, src, &L->uq, H * (D->dim + D->rot_dim), L->q_rank_p, &uq, 1));
    LB_TRY(build_mat(m, src, &L->uk, H * D->dim, L->rank_p, &uk, 1));
    LB_TRY(build_mat(m, src, &L->uv, H * D->vdim, L->rank_p, &uv, 1));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_DQ_NORM], 1, D->q_rank, &L->cq_norm, 1.f, 0.02f));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_DKV_NORM], 1, D->kv_rank, &L->c_norm, 1.f, 0.02f));
    if (D->sink) LB_TRY(load_vec(m, src, D->tensor[LB_T_SINK], 1, H, &L->sink, 0.f, 1.f));
    LB_TRY(upload_yarn_freqs(m, D, &L->freq_k, &L->rot_mul));
    const size_t bytes = (size_t)d->max_ctx * (L->rank_p + L->rot_p) * S->esz;
    LB_TRY(lb_dalloc(m, &L->k_cache, bytes));
    LB_CU(m->c, lb_drv.MemsetD8Async(L->k_cache, 0, bytes, m->c->stream)); /* padding columns stay zero */
    return LB_OK;
}

static int load_ssm(lb_model* m, lb_weight_source* src, int i) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    const lb_stack_layer* D = &d->layer[i];
    st_layer* L = &S->L[i];
    const int inner = D->heads * D->vdim, C = conv_channels(D), rows = inner + C + D->heads;
    L->N_p = pad_to(D->state, 16);
    L->V_p = pad_to(D->vdim, LB_SSM_COLS);
    const st_part in = {D->tensor[LB_T_IN], rows, d->width, 0, 1, 0};
    LB_TRY(build_mat(m, src, &L->in, rows, S->Kw, &in, 1));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_CONV], C, D->taps, &L->conv, 0.f, 0.5f));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_CONV_B], 1, C, &L->conv_b, 0.f, 0.1f));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_DT_BIAS], 1, D->heads, &L->dt_bias, -3.f, 1.f));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_A_LOG], 1, D->heads, &L->a_log, 1.5f, 0.7f));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_D], 1, D->heads, &L->dskip, 1.f, 0.1f));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_HEAD_NORM], 1, inner, &L->head_norm, 1.f, 0.02f));
    LB_TRY(lb_dalloc(m, &L->state, state_bytes(D)));
    LB_TRY(lb_dalloc(m, &L->ring, ring_bytes(D)));
    return LB_OK;
}

static int load_serial_layer(lb_model* m, lb_weight_source* src, int i) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    const lb_stack_layer* D = &d->layer[i];
    st_layer* L = &S->L[i];
    const int W = d->width;
    LB_TRY(load_vec(m, src, D->tensor[LB_T_NORM1], 1, W, &L->norm1, 1.f, 0.02f));
    LB_TRY(load_vec(m, src, D->tensor[LB_T_NORM1_B], 1, W, &L->norm1_b, 0.f, 0.02f));
    LB_TRY(D->mixer == LB_MIX_LATENT ? load_latent(m, src, i) : load_ssm(m, src, i));
    L->n_mix = D->heads * D->vdim;
    L->n_mix_pad = pad_to(L->n_mix, 64);
    const st_part o = {D->tensor[LB_T_O], W, L->n_mix, 0, 1, 0};
    LB_TRY(build_mat(m, src, &L->out, W, L->n_mix_pad, &o, 1));
    return D->ff ? load_serial_ff(m, src, i) : LB_OK;
}

static int load_layer(lb_model* m, lb_weight_source* src, int i) {
    stack_t* S = S_of(m);
    if (S->d.serial) return load_serial_layer(m, src, i);
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
    const int normed = p->x_mode == LB_RG_X_NORM;
    const int kernel = p->sel ? LBK_rows_gemv_experts : normed && p->norm == LB_NORM_LAYER ? LBK_rows_gemv_ln : normed && p->norm == LB_NORM_RMS ? LBK_rows_gemv_rms : LBK_rows_gemv;
    int P = 0;
    if (p->sel && normed && p->norm != LB_NORM_LAYER) return lb_fail(c, LB_ERR_INVALID, "model: experts behind another norm than layer norm");
    for (int i = 0; i < p->n_mat; i++) P += (p->mat[i].rows + 1) / 2;
    const int n_vec = p->x_mode == LB_RG_X_NORM ? p->n_mat : 1, limit = c->max_smem_optin - ((c->fn_static_smem[kernel] + 1023) & ~1023);
    const int by_columns = p->sel && p->x_mode == LB_RG_X_CAT; /* experts side by side along K */
    if (!p->sel) p->parts = 1;
    if (!by_columns) p->k_part = p->K;
    p->segs_part = (p->k_part + LB_RG_SEG - 1) / LB_RG_SEG;
    p->segs = by_columns ? p->parts * p->segs_part : p->segs_part;
    p->status = (uint32_t*)c->dev_status;
    const int can_halve = !p->sel && p->x_mode == LB_RG_X_CAT && p->n_mix_pad <= p->segs / 2 * LB_RG_SEG && c->sm_count % 2 == 0;
    size_t smem = 0;
    int ks = 1;
    for (ks = 1; ks <= 1 + can_halve; ks++) {
        const int ctas = c->sm_count / ks, max_pairs = (P + ctas - 1) / ctas, segs = (p->segs + ks - 1) / ks;
        p->x_cols = ks == 1 ? p->K : segs * LB_RG_SEG;
        p->split = max_pairs >= LB_RG_WARPS ? 1 : segs; /* pieces, each with its sum over the warp, only where warps would have no row pair at all */
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
    return lb_launch_cluster(c, kernel, (unsigned)(c->sm_count / ks), (unsigned)ks, 1, LB_RG_THREADS, (unsigned)smem, params, 1, (unsigned)ks);
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

static int launch_tc(lb_ctx* c, lb_dgemm_params* p, int tiles) { /* operand stages, accumulator columns, CTAs */
    const int stage = LB_DG_ROWS * LB_DG_KB * 2 + p->NT * LB_DG_KB * 2;
    p->stages = 200 * 1024 / stage;
    if (p->stages > LB_DG_MAX_STAGES) p->stages = LB_DG_MAX_STAGES;
    for (p->tmem_cols = 32; p->tmem_cols < 2 * p->NT;) p->tmem_cols *= 2;
    void* params[] = {p};
    return lb_launch(c, LBK_gemm_bf16_tc, (unsigned)(tiles < c->sm_count ? tiles : c->sm_count), 1, 1, LB_DG_THREADS, (unsigned)(p->stages * stage), params, 1);
}

/* one or two products Y = X W^T of a chunk (w[1] may be NULL) */
typedef struct { const st_mat* w; CUdeviceptr x; CUdeviceptr y; int y_mode, ld_y; int ld_x, head, head_p; } st_prod; /* ld_x 0: K; head: LB_DY_HEADS */
static int launch_products(lb_model* m, const st_prod* pr, int n, int T) {
    lb_ctx* c = m->c;
    const stack_t* S = S_of(m);
    lb_dgemm_params p;
    memset(&p, 0, sizeof p);
    p.T = T; p.K = pr[0].w->K; p.ld_x = pr[0].ld_x ? pr[0].ld_x : p.K;
    p.mult = (float)S->d.residual_mult; p.cap = (float)S->d.logit_softcap;
    p.status = (uint32_t*)c->dev_status;
    for (int i = 0; i < n; i++) {
        p.rows[i] = pr[i].w->rows; p.w[i] = (const uint16_t*)pr[i].w->w; p.x[i] = (const void*)pr[i].x;
        p.y[i] = (void*)pr[i].y; p.y_mode[i] = pr[i].y_mode; p.ld_y[i] = pr[i].ld_y; p.y_f32[i] = S->esz == 4;
        p.tiles[i] = (p.rows[i] + LB_DG_ROWS - 1) / LB_DG_ROWS;
        p.head[i] = pr[i].head; p.head_p[i] = pr[i].head_p;
    }
    product_cost(c, p.tiles[0] + p.tiles[1], T, &p.NT);
    p.t_tiles = (T + p.NT - 1) / p.NT;
    void* params[] = {&p};
    if (S->esz == 4)
        return lb_launch(c, LBK_gemm_f32_simt, (unsigned)((p.rows[0] + 63) / 64 + (p.rows[1] + 63) / 64), (unsigned)((T + 63) / 64), 1, 256, 0, params, 1);
    for (int i = 0; i < n; i++) {
        CUtensorMap tm;
        memcpy(p.tmap_w[i], &pr[i].w->tmap, sizeof tm);
        LB_TRY(map_rows_ld(c, &tm, pr[i].x, T, p.K, p.ld_x, p.NT));
        memcpy(p.tmap_x[i], &tm, sizeof tm);
    }
    return launch_tc(c, &p, (p.tiles[0] + p.tiles[1]) * p.t_tiles);
}

/* the expert products of a chunk: `n` assignments sorted by expert, tile by tile of the plan */
static double tile_cost(int nt) { const double c = 0.1 + 0.9 * nt / 256.0; return c < 0.33 ? 0.33 : c; } /* the table of product_cost, any width */
static int moe_tile(const stack_t* S, const lb_stack_layer* D, int T) { /* assignments per tile: an expert's share and some more, in as few tiles as pays */
    if (S->esz == 4) return ST_MOE_TILE;
    const double share = (double)T * D->top / D->experts, want = share + 2.0 * sqrt(share);
    double best = 1e30;
    int nt = 256;
    for (int k = (int)(want / 256.0) + 1, n = 0; n < 3; n++, k++) {
        const int w = pad_to((int)ceil(want / k), 16), c = w > 256 ? 256 : w;
        if (k * tile_cost(c) < best) { best = k * tile_cost(c); nt = c; }
    }
    return nt;
}
static size_t plan_ints(int T, int top, int experts, int nt) { return (size_t)pad_to(T * top, 4) + 4 + 4 * (size_t)(experts + T * top / nt + 1); }
static int launch_experts(lb_model* m, const lb_stack_layer* D, const st_mat* w, int rows, int expert_rows, CUdeviceptr x, CUdeviceptr y, int y_mode, int ld_y, int T,
                          CUdeviceptr plan) {
    lb_ctx* c = m->c;
    const stack_t* S = S_of(m);
    lb_dgemm_params p;
    memset(&p, 0, sizeof p);
    const int n = T * D->top, f32 = S->esz == 4;
    p.NT = moe_tile(S, D, T);
    const int max_tt = D->experts + n / p.NT < n ? D->experts + n / p.NT : n; /* token tiles the plan can have */
    p.T = n; p.K = w->K; p.ld_x = p.K; p.limit = (float)D->limit; p.alpha = (float)D->alpha;
    p.status = (uint32_t*)c->dev_status;
    p.rows[0] = rows; p.expert_rows = expert_rows; p.w[0] = (const uint16_t*)w->w; p.x[0] = (const void*)x; p.y[0] = (void*)y; p.y_mode[0] = y_mode; p.ld_y[0] = ld_y;
    p.y_f32[0] = f32;
    p.head[0] = p.head_p[0] = rows;
    p.tiles[0] = (rows + LB_DG_ROWS - 1) / LB_DG_ROWS;
    p.plan_n = (const int32_t*)(plan + (size_t)pad_to(n, 4) * 4);
    p.plan_tiles = p.plan_n + 4;
    void* params[] = {&p};
    if (f32) return lb_launch(c, LBK_gemm_f32_simt, (unsigned)((rows + 63) / 64), (unsigned)max_tt, 1, 256, 0, params, 1);
    CUtensorMap tm;
    memcpy(p.tmap_w[0], &w->tmap, sizeof tm);
    LB_TRY(map_rows(c, &tm, x, n, p.K, p.NT));
    memcpy(p.tmap_x[0], &tm, sizeof tm);
    return launch_tc(c, &p, max_tt * p.tiles[0]);
}
static int launch_plan(lb_model* m, int i, int pos0, int T, CUdeviceptr plan) {
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    lb_moe_plan_params p;
    memset(&p, 0, sizeof p);
    p.tokens = (const int32_t*)(m->d_tokens + (size_t)pos0 * 4); p.table = (const int32_t*)S->L[i].table;
    p.place = (int32_t*)plan; p.n_tiles = p.place + pad_to(T * D->top, 4); p.tiles = p.n_tiles + 4;
    p.T = T; p.top = D->top; p.experts = D->experts; p.NT = moe_tile(S, D, T);
    void* params[] = {&p};
    return lb_launch(m->c, LBK_moe_plan, 1, 1, 1, 1024, 0, params, 1);
}

static void fill_latent(const lb_model* m, int i, lb_latent_params* p, CUdeviceptr proj, CUdeviceptr q, CUdeviceptr lat_q, CUdeviceptr lat_part) {
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    memset(p, 0, sizeof *p);
    p->proj = (const float*)proj; p->ld = L->in.rows; p->kv_off = L->k_off; p->q = (const float*)q;
    p->uk = (const uint16_t*)L->uk.w; p->uv = (const uint16_t*)L->uv.w; p->c_norm = (const uint16_t*)L->c_norm; p->sink = (const uint16_t*)L->sink;
    p->freq = (const double*)L->freq_k; p->cache = (void*)L->k_cache; p->ql = (float*)lat_q; p->part = (float*)lat_part;
    p->status = (uint32_t*)m->c->dev_status;
    p->H = D->heads; p->dim = D->dim; p->dim_p = L->dim_p; p->vdim = D->vdim; p->rank = D->kv_rank; p->rank_p = L->rank_p; p->rot = D->rot_dim; p->rot_p = L->rot_p;
    p->T = 1; p->max_ctx = S->d.max_ctx; p->splits = 1; p->stages = 1;
    p->rot_mul = L->rot_mul; p->scale = (float)D->scale; p->eps = (float)S->d.eps;
}
/* slices of the cache: as many as keep one CTA per SM, one staged block of rows each at least */
static int latent_splits(const lb_ctx* c, const stack_t* S, const lb_stack_layer* D, int T) {
    const int groups = S->esz == 4 ? T * ((D->heads + 7) / 8) : (T * D->heads + 15) / 16, blocks = (S->d.max_ctx + LB_LA_KEYS - 1) / LB_LA_KEYS;
    int n = c->sm_count / groups;
    if (n > blocks) n = blocks;
    if (n > LB_LA_MAX_SPLITS) n = LB_LA_MAX_SPLITS;
    return n < 1 ? 1 : n;
}
/* the absorbed way: T tokens from p's position on; queries, slices, output */
static int launch_latent_absorbed(lb_model* m, int i, lb_latent_params* p) {
    lb_ctx* c = m->c;
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const int f32 = S->esz == 4, ld_c = p->rank_p + p->rot_p, row = 2 * ld_c + 16;
    const unsigned tg = (unsigned)((p->T + LB_LA_TOKENS - 1) / LB_LA_TOKENS);
    p->splits = latent_splits(c, S, D, p->T);
    void* params[] = {p};
    LB_TRY(lb_launch(c, f32 ? LBK_lat_query_f32 : LBK_lat_query_bf16, (unsigned)D->heads + 1, (unsigned)((p->rank_p + 127) / 128), tg, 256, 0, params, 1));
    if (f32) {
        LB_TRY(lb_launch(c, LBK_lat_rows_f32, (unsigned)(p->T * ((D->heads + 7) / 8)), (unsigned)p->splits, 1, 128, (unsigned)((8 * ld_c + 32 * (ld_c + 4)) * 4), params, 1));
    } else {
        const int fixed = 32 * row + 32 * 144;
        p->stages = fixed + 2 * LB_LA_KEYS * row <= 220 * 1024 ? 2 : 1;
        LB_TRY(lb_launch(c, p->rank_p <= 128 ? LBK_lat_rows_128 : p->rank_p <= 256 ? LBK_lat_rows_256 : LBK_lat_rows_512, (unsigned)((p->T * D->heads + 15) / 16),
                         (unsigned)p->splits, 1, 128, (unsigned)(fixed + p->stages * LB_LA_KEYS * row), params, 1));
    }
    return lb_launch(c, f32 ? LBK_lat_out_f32 : LBK_lat_out_bf16, (unsigned)D->heads, (unsigned)((D->vdim + 31) / 32), tg, 256, 0, params, 1);
}

static void fill_ssm(const lb_model* m, int i, lb_ssm_params* p, CUdeviceptr proj) {
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    memset(p, 0, sizeof *p);
    p->proj = (const float*)proj; p->ld = L->in.rows;
    p->conv_w = (const uint16_t*)L->conv; p->conv_b = (const uint16_t*)L->conv_b; p->dt_bias = (const uint16_t*)L->dt_bias; p->a_log = (const uint16_t*)L->a_log;
    p->d = (const uint16_t*)L->dskip; p->norm_w = (const uint16_t*)L->head_norm; p->state = (float*)L->state; p->ring = (float*)L->ring;
    p->H = D->heads; p->V = D->vdim; p->V_p = L->V_p; p->N = D->state; p->N_p = L->N_p; p->G = D->groups; p->taps = D->taps; p->channels = conv_channels(D);
    p->ld_xbc = D->heads * L->V_p + 2 * D->groups * L->N_p; p->norm_groups = D->norm_groups; p->T = 1; p->f32 = S->esz == 4; p->eps = (float)S->d.eps;
}
static int state_size(const lb_stack_layer* D) { return D->state <= 64 ? 0 : D->state <= 128 ? 1 : 2; }

/* ---- the decode step ------------------------------------------------------------------------------------------------ */
/* rows of W (two at most) against the normed residual, or against one vector */
static void rows_norm(const stack_t* S, lb_rows_gemv_params* g, CUdeviceptr x, int width, int K, int norm) {
    memset(g, 0, sizeof *g);
    g->x_mode = LB_RG_X_NORM; g->x = (const float*)x; g->width = width; g->K = K; g->norm = norm; g->eps = (float)S->d.eps; g->n_mat = 1;
}
static void rows_cat(const lb_model* m, lb_rows_gemv_params* g, const st_mat* w, int rows, double mult) { /* ... added to the residual */
    memset(g, 0, sizeof *g);
    g->x_mode = LB_RG_X_CAT; g->K = w->K; g->eps = (float)S_of(m)->d.eps; g->mult = (float)mult; g->n_mat = 1;
    g->mat[0] = (lb_rg_mat){(const uint16_t*)w->w, NULL, NULL, (float*)m->X, rows, LB_DY_RESIDUAL};
}

static int serial_step_ff(lb_model* m, int i) {
    const stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    const lb_stack_layer* D = &d->layer[i];
    const st_layer* L = &S->L[i];
    const int moe = D->ff_kind == LB_FF_EXPERTS;
    lb_rows_gemv_params g;
    rows_norm(S, &g, m->X, d->width, S->Kw, d->norm);
    g.mat[0] = (lb_rg_mat){(const uint16_t*)L->ff.w, (const uint16_t*)L->norm2, (const uint16_t*)L->norm2_b, (float*)S->act, moe ? 2 * D->ff * D->top : D->ff,
                           moe ? LB_DY_CLAMP_GLU : LB_DY_RELU2};
    if (moe) {
        g.sel = (const int32_t*)L->table; g.sel_row = (const int32_t*)m->d_token; g.parts = D->top; g.sel_rows = 2 * D->ff; g.y_part = L->ff_p;
        g.limit = (float)D->limit; g.alpha = (float)D->alpha;
    }
    LB_TRY(launch_rows(m, &g));
    rows_cat(m, &g, &L->down, d->width, moe ? d->residual_mult / D->top : d->residual_mult);
    g.act = (const float*)S->act; g.n_act = D->ff;
    if (moe) {
        g.sel = (const int32_t*)L->table; g.sel_row = (const int32_t*)m->d_token; g.parts = D->top; g.k_part = L->ff_p;
        g.K = D->top * L->ff_p; g.n_act = g.K;
    }
    return launch_rows(m, &g);
}

static int serial_step_layer(lb_model* m, int i) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    const lb_stack_layer* D = &d->layer[i];
    const st_layer* L = &S->L[i];
    lb_rows_gemv_params g;
    rows_norm(S, &g, m->X, d->width, S->Kw, d->norm);
    g.mat[0] = (lb_rg_mat){(const uint16_t*)L->in.w, (const uint16_t*)L->norm1, (const uint16_t*)L->norm1_b, (float*)S->proj, L->in.rows, LB_DY_STORE};
    LB_TRY(launch_rows(m, &g));
    if (D->mixer == LB_MIX_LATENT) {
        rows_norm(S, &g, S->proj, D->q_rank, L->q_rank_p, LB_NORM_RMS);
        g.mat[0] = (lb_rg_mat){(const uint16_t*)L->uq.w, (const uint16_t*)L->cq_norm, NULL, (float*)S->lq, L->uq.rows, LB_DY_STORE};
        LB_TRY(launch_rows(m, &g));
        lb_latent_params p;
        fill_latent(m, i, &p, S->proj, S->lq, S->lat_q, S->lat_part);
        p.out = (float*)S->mix; p.pos_ptr = (const int32_t*)m->d_pos;
        LB_TRY(launch_latent_absorbed(m, i, &p));
        rows_cat(m, &g, &L->out, d->width, d->residual_mult);
    } else {
        lb_ssm_params p;
        fill_ssm(m, i, &p, S->proj);
        p.y = (float*)S->mix; p.pos_ptr = (const int32_t*)m->d_pos;
        static const int k[3] = {LBK_ssm_step_64, LBK_ssm_step_128, LBK_ssm_step_256};
        void* params[] = {&p};
        LB_TRY(lb_launch(m->c, k[state_size(D)], (unsigned)D->heads, (unsigned)(L->V_p / LB_SSM_COLS), 1, 128, 0, params, 1));
        rows_cat(m, &g, &L->out, d->width, d->residual_mult);
        g.gate = (const float*)S->proj; g.gate_first = 1; g.head_w = (const uint16_t*)L->head_norm; g.vdim = L->n_mix / D->norm_groups;
    }
    g.mix = (const float*)S->mix; g.n_mix = L->n_mix; g.n_mix_pad = L->n_mix_pad;
    LB_TRY(launch_rows(m, &g));
    return D->ff ? serial_step_ff(m, i) : LB_OK;
}

static int stack_step_layers(lb_model* m) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    for (int i = 0; d->serial && i < d->n_layers; i++) LB_TRY(serial_step_layer(m, i));
    if (d->serial) return LB_OK;
    for (int i = 0; i < d->n_layers; i++) {
        const lb_stack_layer* D = &d->layer[i];
        const st_layer* L = &S->L[i];
        lb_rows_gemv_params g;
        memset(&g, 0, sizeof g);
        g.x_mode = LB_RG_X_NORM; g.x = (const float*)m->X; g.width = d->width; g.K = S->Kw; g.eps = (float)d->eps;
        g.n_mat = D->ff ? 2 : 1;
        g.mat[0] = (lb_rg_mat){(const uint16_t*)L->in.w, (const uint16_t*)L->norm1, NULL, (float*)S->proj, L->in.rows, LB_DY_STORE};
        if (D->ff) g.mat[1] = (lb_rg_mat){(const uint16_t*)L->ff.w, (const uint16_t*)L->norm2, NULL, (float*)S->act, L->ff.rows, LB_DY_RELU_GLU};
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
        g.mat[0] = (lb_rg_mat){(const uint16_t*)L->out.w, NULL, NULL, (float*)m->X, L->out.rows, LB_DY_RESIDUAL};
        LB_TRY(launch_rows(m, &g));
    }
    return LB_OK;
}

static int stack_head(lb_model* m, CUdeviceptr x_row) {
    const stack_t* S = S_of(m);
    lb_rows_gemv_params g;
    rows_norm(S, &g, x_row, S->d.width, S->Kw, S->d.norm);
    g.cap = (float)S->d.logit_softcap;
    g.mat[0] = (lb_rg_mat){(const uint16_t*)S->head.w, (const uint16_t*)m->final_norm, (const uint16_t*)S->final_b, (float*)m->logits, S->head.rows, LB_DY_SOFTCAP};
    g.part_val = (float*)m->cand_val; g.part_idx = (int32_t*)m->cand_idx;
    return launch_rows(m, &g);
}
static int stack_head_ctas(lb_model* m) { return m->c->sm_count; }

/* ---- a prompt chunk --------------------------------------------------------------------------------------------------- */
/* norms of a chunk's rows (the design's kind); callers add to it what a launch does besides */
static lb_norm2_params norm_params(const lb_model* m, CUdeviceptr x, CUdeviceptr w, CUdeviceptr b, CUdeviceptr h) {
    const stack_t* S = S_of(m);
    lb_norm2_params p;
    memset(&p, 0, sizeof p);
    p.x = (float*)x; p.w[0] = (const uint16_t*)w; p.b[0] = (const uint16_t*)b; p.h[0] = (void*)h;
    p.width = p.ld_x = S->d.width; p.ld = S->Kw; p.f32 = S->esz == 4; p.norm = S->d.norm; p.eps = (float)S->d.eps;
    return p;
}
static int launch_norm(lb_model* m, lb_norm2_params* p, int T) {
    void* params[] = {p};
    const int plain = p->norm == LB_NORM_RMS_1P && p->ld_x == p->width && !p->y && !p->scatter;
    return lb_launch(m->c, plain ? LBK_norm_rows2 : LBK_norm_rows_any, (unsigned)T, 1, 1, 256, 0, params, 1);
}
static int norm_rows(lb_model* m, CUdeviceptr x, CUdeviceptr w0, CUdeviceptr h0, CUdeviceptr w1, CUdeviceptr h1, int T) {
    lb_norm2_params p = norm_params(m, x, w0, 0, h0);
    p.w[1] = (const uint16_t*)w1; p.h[1] = (void*)h1;
    return launch_norm(m, &p, T);
}

/* what the experts of layer i left in ye joins the residual in the norm that follows */
static void norm_adds(const lb_model* m, const pf_set* w, int i, lb_norm2_params* p) {
    const stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    p->y = (const void*)w->st.ye; p->y_place = (const int32_t*)w->st.plan; p->y_top = D->top; p->ld_y = S->d.width;
    p->y_mult = (float)(S->d.residual_mult / D->top);
}
static int has_experts(const stack_t* S, int i) { return i >= 0 && S->d.layer[i].ff && S->d.layer[i].ff_kind == LB_FF_EXPERTS; }

static int pf_latent(lb_model* m, pf_set* w, int i, int pos0, int T) {
    lb_ctx* c = m->c;
    stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    const int kd = L->dim_p + L->rot_p, ld_c = L->rank_p + L->rot_p;
    lb_norm2_params n = norm_params(m, w->st.proj, L->cq_norm, 0, w->st.h2);
    n.width = D->q_rank; n.ld_x = L->in.rows; n.ld = L->q_rank_p; n.norm = LB_NORM_RMS;
    LB_TRY(launch_norm(m, &n, T));
    const st_prod uq = {&L->uq, w->st.h2, w->st.lq, LB_DY_STORE, L->uq.rows, 0, 0, 0};
    LB_TRY(launch_products(m, &uq, 1, T));
    lb_latent_params p;
    fill_latent(m, i, &p, w->st.proj, w->st.lq, w->st.lat_q, w->st.lat_part);
    p.pos0 = pos0; p.T = T; p.cat = (void*)w->st.cat; p.cat_ld = L->out.K;
    if (!L->splits || T < ST_LAT_ABSORB) return launch_latent_absorbed(m, i, &p);
    /* every seen position's keys and values from its latent, then attention on the tensor cores, one KV head per head */
    p.qh = (uint16_t*)w->st.q; p.ql16 = (uint16_t*)w->st.k;
    void* params[] = {&p};
    LB_TRY(lb_launch(c, LBK_lat_prepare, (unsigned)T, 1, 1, 256, 0, params, 1));
    const st_prod kv[2] = {{&L->uk, L->k_cache, w->st.kx, LB_DY_HEADS, D->heads * L->dim_p, ld_c, D->dim, L->dim_p},
                           {&L->uv, L->k_cache, w->st.vx, LB_DY_HEADS, D->heads * L->vdim_p, ld_c, D->vdim, L->vdim_p}};
    LB_TRY(launch_products(m, kv, 2, pos0 + T));
    lb_wattn_params a;
    memset(&a, 0, sizeof a);
    a.k_cache = (void*)w->st.kx; a.v_cache = (void*)w->st.vx; a.qh = (uint16_t*)w->st.q; a.ql = (uint16_t*)w->st.k;
    a.k_tail = (const uint16_t*)(L->k_cache + (size_t)L->rank_p * 2); a.tail_p = L->rot_p; a.tail_ld = ld_c;
    a.sink = D->sink; a.sink_w = (const uint16_t*)L->sink; a.status = (uint32_t*)c->dev_status;
    a.H = a.KV = D->heads; a.dim = D->dim + D->rot_dim; a.dim_p = kd; a.vdim = D->vdim; a.vdim_p = L->vdim_p;
    a.pos0 = pos0; a.T = T; a.max_ctx = S->d.max_ctx; a.cat = (void*)w->st.cat; a.cat_ld = L->out.K;
    void* aparams[] = {&a};
    const unsigned smem = (unsigned)(2 * LB_WA_ROWS * (2 * kd + 16) + 2 * LB_WA_KV * (2 * kd + 2 * L->vdim_p + 32));
    return lb_launch(c, L->vdim_p <= 64 ? LBK_wattn_chunk_64 : L->vdim_p <= 128 ? LBK_wattn_chunk_128 : LBK_wattn_chunk_256,
                     (unsigned)((T + LB_WA_ROWS - 1) / LB_WA_ROWS), (unsigned)D->heads, 1, LB_WA_THREADS, smem, aparams, 1);
}

static int pf_ssm(lb_model* m, pf_set* w, int i, int pos0, int T) {
    lb_ctx* c = m->c;
    stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    lb_ssm_params p;
    fill_ssm(m, i, &p, w->st.proj);
    p.pos0 = pos0; p.T = T; p.xbc = (void*)w->st.xbc; p.dt = (float*)w->st.dt; p.y = (float*)w->st.o; p.cat = (void*)w->st.cat; p.cat_ld = L->out.K;
    void* params[] = {&p};
    LB_TRY(lb_launch(c, LBK_ssm_conv, (unsigned)((p.ld_xbc + D->heads + 255) / 256), (unsigned)((T + LB_SSM_CONV_TOKENS - 1) / LB_SSM_CONV_TOKENS), 1, 256, 0, params, 1));
    static const int k_f32[3] = {LBK_ssm_scan_f32_64, LBK_ssm_scan_f32_128, LBK_ssm_scan_f32_256}, k_tc[3] = {LBK_ssm_chunk_64, LBK_ssm_chunk_128, LBK_ssm_chunk_256};
    const int row = 2 * L->N_p + 16, smem = 2 * LB_SSM_SEG * row + (row >= 240 ? 1 : 4) * LB_SSM_SEG * 80 + 3 * L->N_p * 80 + 2 * LB_SSM_SEG * 4; /* as ssm_chunk lays it out */
    static const int k_local[3] = {LBK_ssm_local_64, LBK_ssm_local_128, LBK_ssm_local_256};
    const unsigned slabs = (unsigned)(L->V_p / LB_SSM_COLS), heads = (unsigned)D->heads;
    if (S->esz == 4) LB_TRY(lb_launch(c, k_f32[state_size(D)], heads, slabs, 1, 128, 0, params, 1));
    else {
        /* as many segments side by side as CTAs fit on the SMs, four blocks of tokens each at least */
        const int blocks = (T + LB_SSM_SEG - 1) / LB_SSM_SEG, fit = c->sm_count * (L->N_p <= 128 ? 3 : 1) / (int)(heads * slabs);
        int P = fit < blocks / 4 ? fit : blocks / 4;
        if (P > ST_SSM_SEGS) P = ST_SSM_SEGS;
        if (P < 1) P = 1;
        p.seg = (blocks + P - 1) / P * LB_SSM_SEG;
        P = (T + p.seg - 1) / p.seg;
        p.seg_state = (float*)w->st.seg_state; p.seg_decay = (float*)w->st.seg_decay;
        if (P > 1) LB_TRY(lb_launch(c, k_local[state_size(D)], heads, slabs, (unsigned)P - 1, 128, (unsigned)smem, params, 1));
        LB_TRY(lb_launch(c, k_tc[state_size(D)], heads, slabs, (unsigned)P, 128, (unsigned)smem, params, 1));
    }
    return lb_launch(c, LBK_ssm_finish, (unsigned)T, (unsigned)D->norm_groups, 1, 128, (unsigned)(L->n_mix / D->norm_groups * 4), params, 1);
}

static int pf_serial_ff(lb_model* m, pf_set* w, int i, int pos0, int T) {
    stack_t* S = S_of(m);
    const lb_stack_desc* d = &S->d;
    const lb_stack_layer* D = &d->layer[i];
    const st_layer* L = &S->L[i];
    lb_norm2_params n = norm_params(m, w->st.X, L->norm2, L->norm2_b, w->st.h1);
    if (D->ff_kind != LB_FF_EXPERTS) {
        LB_TRY(launch_norm(m, &n, T));
        const st_prod up = {&L->ff, w->st.h1, w->st.act, LB_DY_RELU2, L->ff_p, 0, 0, 0}, down = {&L->down, w->st.act, w->st.X, LB_DY_RESIDUAL, d->width, 0, 0, 0};
        LB_TRY(launch_products(m, &up, 1, T));
        return launch_products(m, &down, 1, T);
    }
    n.h[0] = (void*)w->st.xg; n.scatter = (const int32_t*)w->st.plan; n.top = D->top;
    LB_TRY(launch_norm(m, &n, T));
    LB_TRY(launch_experts(m, D, &L->ff, 2 * D->ff, 2 * D->ff, w->st.xg, w->st.act, LB_DY_CLAMP_GLU, L->ff_p, T, w->st.plan));
    LB_TRY(launch_experts(m, D, &L->down, d->width, pad_to(d->width, 2), w->st.act, w->st.ye, S->esz == 4 ? LB_DY_STORE : LB_DY_HEADS, d->width, T, w->st.plan));
    if (i + 1 < d->n_layers) return LB_OK;
    lb_norm2_params last = norm_params(m, w->st.X, 0, 0, 0); /* nothing follows that would add them */
    norm_adds(m, w, i, &last);
    return launch_norm(m, &last, T);
}

static int pf_serial_layer(lb_model* m, pf_set* w, int i, int pos0, int T) {
    stack_t* S = S_of(m);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    lb_norm2_params n = norm_params(m, w->st.X, L->norm1, L->norm1_b, w->st.h1);
    if (has_experts(S, i - 1)) norm_adds(m, w, i - 1, &n);
    LB_TRY(launch_norm(m, &n, T));
    if (has_experts(S, i)) LB_TRY(launch_plan(m, i, pos0, T, w->st.plan)); /* the previous layer's places have been read */
    const st_prod in = {&L->in, w->st.h1, w->st.proj, LB_DY_STORE, L->in.rows, 0, 0, 0};
    LB_TRY(launch_products(m, &in, 1, T));
    LB_TRY(D->mixer == LB_MIX_LATENT ? pf_latent(m, w, i, pos0, T) : pf_ssm(m, w, i, pos0, T));
    const st_prod out = {&L->out, w->st.cat, w->st.X, LB_DY_RESIDUAL, S->d.width, 0, 0, 0};
    LB_TRY(launch_products(m, &out, 1, T));
    return D->ff ? pf_serial_ff(m, w, i, pos0, T) : LB_OK;
}

static int stack_pf_layer(lb_model* m, pf_set* w, int i, int pos0, int T) {
    lb_ctx* c = m->c;
    stack_t* S = S_of(m);
    if (S->d.serial) return pf_serial_layer(m, w, i, pos0, T);
    const lb_stack_layer* D = &S->d.layer[i];
    const st_layer* L = &S->L[i];
    const int f32 = S->esz == 4;
    LB_TRY(norm_rows(m, w->st.X, L->norm1, w->st.h1, D->ff ? L->norm2 : 0, D->ff ? w->st.h2 : 0, T));
    st_prod pr[2] = {{&L->in, w->st.h1, w->st.proj, LB_DY_STORE, L->in.rows, 0, 0, 0},
                     {&L->ff, w->st.h2, w->st.cat + (size_t)L->n_mix_pad * S->esz, LB_DY_RELU_GLU, L->out.K, 0, 0, 0}};
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
    const st_prod out = {&L->out, w->st.cat, w->st.X, LB_DY_RESIDUAL, S->d.width, 0, 0, 0};
    return launch_products(m, &out, 1, T);
}

static int stack_head_rows(lb_model* m, CUdeviceptr rows, int n, CUdeviceptr logits) {
    stack_t* S = S_of(m);
    pf_set* w = lb_prefill_set(m, 0); /* the chunk streams have been joined: their buffers are free */
    lb_norm2_params p = norm_params(m, rows, m->final_norm, S->final_b, w->st.h1);
    LB_TRY(launch_norm(m, &p, n));
    const st_prod pr = {&S->head, w->st.h1, logits, LB_DY_SOFTCAP, S->head.rows, 0, 0, 0};
    return launch_products(m, &pr, 1, n);
}

static void stack_pf_sizes(const lb_model* m, size_t bytes[LB_PF_MAX_BUFS]) {
    const stack_t* S = S_of(m);
    const int absorbed = S->lat_full ? m->pf_chunk : m->pf_chunk < ST_LAT_ABSORB ? m->pf_chunk : ST_LAT_ABSORB;
    const size_t T = (size_t)m->pf_chunk, C = (size_t)S->d.max_ctx, e = (size_t)S->esz, q = (size_t)S->max_dk * 4 > (size_t)S->max_q * 2 ? (size_t)S->max_dk * 4 : (size_t)S->max_q * 2;
    const size_t b[] = {T * (size_t)S->d.width * 4, T * (size_t)S->Kw * e, T * (size_t)S->max_h2 * e, T * (size_t)S->max_in * 4, T * (size_t)S->max_cat * e,
                        T * q, T * q, T * (size_t)S->max_dk * 4, T * (size_t)S->max_o * 4,
                        (T + ST_SEG - 1) / ST_SEG * S->max_state, (T + ST_SEG - 1) / ST_SEG * (size_t)S->max_dk * 4,
                        T * (size_t)S->max_lq * 4, C * (size_t)S->max_kx * 2, C * (size_t)S->max_vx * 2, (size_t)absorbed * (size_t)S->max_latq * 4,
                        S->max_rec ? ((size_t)absorbed * (size_t)S->max_heads + (size_t)S->max_part_rows) * (size_t)S->max_rec * 4 : 0, T * (size_t)S->max_xbc * e,
                        T * (size_t)S->max_heads * 4, T * (size_t)S->max_actp * e, T * (size_t)S->max_top * (size_t)S->Kw * e,
                        T * (size_t)S->max_top * (size_t)S->d.width * e, S->max_top ? plan_ints(m->pf_chunk, S->max_top, S->max_experts, 16) * 4 : 0};
    memcpy(bytes, b, sizeof b); /* in the order of pf_set.st */
}

/* ---- state ---------------------------------------------------------------------------------------------------------------- */
static int stack_reset_state(lb_model* m) { /* cache rows past the position are never read: only the recurrent states start over */
    const stack_t* S = S_of(m);
    for (int i = 0; i < S->d.n_layers; i++)
        if (S->L[i].state) LB_CU(m->c, lb_drv.MemsetD8Async(S->L[i].state, 0, state_bytes(&S->d.layer[i]), m->c->stream));
    return LB_OK; /* a convolution's last inputs are taken as zero before position 0 */
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
        if (!L->ring) continue;
        const size_t r = ring_bytes(&S->d.layer[i]);
        if (!L->snap_ring) LB_TRY(lb_dalloc(m, &L->snap_ring, r));
        LB_CU(c, lb_drv.MemcpyDtoDAsync(restore ? L->ring : L->snap_ring, restore ? L->snap_ring : L->ring, r, c->stream));
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
    } else if (D->mixer == LB_MIX_SSM && which) {
        *dptr = L->ring;
        *bytes = ring_bytes(D);
    } else {
        if (which) return lb_fail(m->c, LB_ERR_INVALID, "layer %d has one state buffer", i);
        if (D->mixer == LB_MIX_LATENT) {
            *dptr = L->k_cache;
            *bytes = (size_t)S->d.max_ctx * (L->rank_p + L->rot_p) * S->esz;
            return LB_OK;
        }
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
                           L->freq_k, L->freq_v, L->state, L->snap, L->down.w, L->uq.w, L->uk.w, L->uv.w, L->norm1_b, L->norm2_b, L->cq_norm, L->c_norm,
                           L->sink, L->conv, L->conv_b, L->dt_bias, L->a_log, L->dskip, L->table, L->ring, L->snap_ring};
        for (size_t k = 0; k < sizeof p / sizeof p[0]; k++) if (p[k]) lb_drv.MemFree(p[k]);
    }
    CUdeviceptr g[] = {S->head.w, S->proj, S->mix, S->act, S->scratch, S->counters, S->final_b, S->lq, S->lat_q, S->lat_part};
    for (size_t k = 0; k < sizeof g / sizeof g[0]; k++) if (g[k]) lb_drv.MemFree(g[k]);
    free(S->L);
    free(S->d.layer);
    S->L = NULL;
    S->d.layer = NULL;
}

static const lb_arch k_stack = {"stack", ST_STREAMS, stack_reset_state, stack_snapshot, stack_state_ptr, stack_step_layers, stack_head,
                                stack_head_ctas, stack_head_rows, stack_pf_sizes, stack_pf_layer, stack_destroy};

/* the expert products of a chunk in the units of product_cost: full tiles (the rate does not fall as much as a dense product's, the tiles of an
 * expert read the same operands), or the time to read every expert's weights from HBM (a wave of tiles takes as long as HBM_ROWS rows of them) */
#define HBM_ROWS 14000.0
static double experts_cost(const lb_model* m, const lb_stack_layer* D, int rows, int K, int T) {
    const stack_t* S = S_of(m);
    const int nt = moe_tile(S, D, T), tiles = D->experts * ((T * D->top / D->experts + nt - 1) / nt) * ((rows + LB_DG_ROWS - 1) / LB_DG_ROWS);
    const double flops = (double)((tiles + m->c->sm_count - 1) / m->c->sm_count) * tile_cost(nt), bytes = D->experts * (double)rows / HBM_ROWS;
    return K * (flops > bytes ? flops : bytes);
}

/* tokens per prompt chunk: the multiple of 256 whose products fill whole waves of SMs best */
static int stack_chunk(const lb_model* m) {
    const stack_t* S = S_of(m);
    double best = 1e30;
    int chunk = 256;
    if (S->esz == 4 && S->max_latq) return chunk; /* an absorbed chunk keeps a latent query per token and head */
    for (int T = 256; T <= (S->max_top ? ST_CHUNK_EXPERTS : ST_CHUNK); T += 256) {
        double cost = 0;
        for (int i = 0; i < S->d.n_layers; i++) {
            const st_layer* L = &S->L[i];
            int nt;
            if (S->d.serial) {
                const st_mat* w[] = {&L->in, &L->uq, &L->out, &L->ff, &L->down};
                const int moe = has_experts(S, i);
                if (moe) cost += experts_cost(m, &S->d.layer[i], 2 * S->d.layer[i].ff, L->ff.K, T) + experts_cost(m, &S->d.layer[i], S->d.width, L->down.K, T);
                for (int k = 0; k < (moe ? 3 : 5); k++)
                    if (w[k]->w) cost += w[k]->K * product_cost(m->c, (w[k]->rows + LB_DG_ROWS - 1) / LB_DG_ROWS, T, &nt);
                continue;
            }
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
    S->max_h2 = S->Kw;
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
        if (D->ff_kind != LB_FF_RELU_GLU) {
            MAX(S->max_ff, D->ff_kind == LB_FF_EXPERTS ? D->top * L->ff_p : L->ff_p);
            MAX(S->max_actp, D->ff_kind == LB_FF_EXPERTS ? D->top * L->ff_p : L->ff_p);
            MAX(S->max_top, D->top); MAX(S->max_experts, D->experts);
        }
        if (D->mixer == LB_MIX_LATENT) {
            const int kd = L->dim_p + L->rot_p, rows = c->sm_count * 16;
            L->splits = S->esz == 2 && kd <= LB_WA_MAX_DIM && L->vdim_p <= LB_WA_MAX_DIM; /* chunks can take the expanded way */
            if (!L->splits) S->lat_full = 1;
            MAX(S->max_h2, L->q_rank_p); MAX(S->max_lq, L->uq.rows); MAX(S->max_latq, D->heads * (L->rank_p + L->rot_p)); MAX(S->max_rec, L->rank_p + 2);
            MAX(S->max_heads, D->heads);
            MAX(S->max_part_rows, rows);
            if (L->splits) {
                MAX(S->max_q, D->heads * kd); MAX(S->max_kx, D->heads * L->dim_p); MAX(S->max_vx, D->heads * L->vdim_p);
            }
        } else if (D->mixer == LB_MIX_SSM) {
            MAX(S->max_state, state_bytes(D));
            MAX(S->max_heads, D->heads); MAX(S->max_dk, D->heads); MAX(S->max_xbc, D->heads * L->V_p + 2 * D->groups * L->N_p); MAX(S->max_o, D->heads * D->vdim);
        } else if (D->mixer == LB_MIX_ATTENTION) {
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
    LB_TRY(load_vec(m, src, d->final_norm, 1, d->width, &m->final_norm, d->norm == LB_NORM_RMS_1P ? 0.f : 1.f, 0.02f));
    if (d->norm == LB_NORM_LAYER) LB_TRY(load_vec(m, src, d->final_norm_b, 1, d->width, &S->final_b, 0.f, 0.02f));
    if (d->bigram.buckets) {
        LB_TRY(load_vec(m, src, d->bigram.name, d->bigram.buckets + 1, d->width, &m->bigram, 0.f, 1.f));
        m->bigram_buckets = d->bigram.buckets; m->bigram_mul_prev = d->bigram.mul_prev; m->bigram_mul_cur = d->bigram.mul_cur;
    }
    if (S->max_latq) {
        LB_TRY(lb_dalloc(m, &S->lq, (size_t)S->max_lq * 4));
        LB_TRY(lb_dalloc(m, &S->lat_q, (size_t)S->max_latq * 4));
        LB_TRY(lb_dalloc(m, &S->lat_part, ((size_t)S->max_heads + (size_t)S->max_part_rows) * (size_t)S->max_rec * 4));
    }
    LB_TRY(lb_dalloc(m, &S->proj, (size_t)S->max_in * 4));
    LB_TRY(lb_dalloc(m, &S->mix, (size_t)S->max_mix * 4));
    LB_TRY(lb_dalloc(m, &S->act, (size_t)(S->max_ff ? S->max_ff : 1) * 4));
    LB_CU(c, lb_drv.MemsetD8Async(S->act, 0, (size_t)(S->max_ff ? S->max_ff : 1) * 4, c->stream)); /* columns that only pad a layer's width stay finite */
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
