/* Kernel parameter blocks shared by the host layer (C) and the kernels (CUDA).
 * Every struct is passed by value as the single kernel parameter, so the
 * layout here IS the launch ABI of the primary entry points.  (The entry
 * points that keep the reference's own positional parameter blocks live under
 * csrc/compat/, one source per cubin, and do not use these structs.) */
#ifndef LB_KERNEL_PARAMS_H
#define LB_KERNEL_PARAMS_H
#include <stdint.h>

/* ---- int4 GEMV ---------------------------------------------------------- */
#define LB_GEMV_TILE_N 256   /* columns per CTA tile: eight 32-column TMA boxes */
#define LB_GEMV_GROUP 128    /* GPTQ group size along K */
#define LB_GEMV_ROWS 16      /* packed rows per group */
#define LB_GEMV_THREADS 160  /* 4 consumer warps (one 32-column box each) + 1 producer warp */
#define LB_GEMV_STAGE_BYTES 16384 /* one pipeline stage: 16 packed rows (one group) x 256 columns */

/* how the activation vector is produced from p.x */
enum {
    LB_X_F16 = 0,          /* x fp16 [K] */
    LB_X_F32 = 1,          /* x fp32 [K], rounded to fp16 */
    LB_X_F32_RMSNORM = 2,  /* x fp32 [K]; h = x*rsqrt(mean x^2+eps)*(1+w), w = aux0 bf16 [K] */
    LB_X_F32_HEADNORM_SILU = 3 /* x fp32 [K] in heads of 128; h = x*rsqrt(mean_head x^2+eps)*w[i]*silu(z),
                                  w = aux0 fp32 [128], z = aux1 fp32 [K] */
};
/* what is done with the N results */
enum {
    LB_Y_F16 = 0,       /* y fp16 [N] = result */
    LB_Y_F32 = 1,       /* y fp32 [N] = result */
    LB_Y_F32_ACCUM = 2, /* y fp32 [N] += result (residual add) */
    LB_Y_SWIGLU_F16 = 3, /* columns come in interleaved 64-wide blocks (gate block, up block, gate block, ...);
                           y fp16 [N/2] = silu(gate)*up */
    LB_Y_TP_ALLREDUCE = 4 /* persistent chain under tensor parallelism only: the fp32 results are this rank's partial sums of a
                           row-parallel projection; y (the residual stream) += their sum over all ranks, exchanged inside the
                           epilogue as (value, generation) words stored straight into every rank's buffer (ext = lb_tp_params) */
};

typedef struct {
    /* CUtensorMap over qweight viewed as [N/32][K/8][32] uint32: box 8 x 16 x 32, 128-byte swizzle */
    unsigned char tmap[128] __attribute__((aligned(64)));
    /* scales as fp16 [K/128, N], box = groups_per_split x 256; qzeros as u32 [K/128, N/8], box = groups_per_split x 32 */
    unsigned char tmap_sc[128] __attribute__((aligned(64)));
    unsigned char tmap_zr[128] __attribute__((aligned(64)));
    const uint32_t* qweight; /* [K/8, N] */
    const uint16_t* scales;  /* fp16 [K/128, N] */
    const uint32_t* qzeros;  /* [K/128, N/8] or NULL: zero-point 8 */
    const void* x;
    void* y;
    const void* aux0;
    const void* aux1;
    uint16_t* x_out;    /* optional fp16 [K]: the activation vector as the kernel used it */
    uint32_t* status;   /* device status word (bounded waits) */
    int32_t K, N;
    int32_t ksplit;           /* gridDim.y = cluster size along y */
    int32_t groups_per_split; /* ceil(K/128 / ksplit) */
    int32_t stages;           /* TMA ring depth */
    int32_t x_mode, y_mode;
    float eps;
} lb_gemv_params;

/* ---- chain of int4 GEMVs in ONE persistent launch (chain.cu) ------------------------------
 * One CTA per SM; CTA c owns a strip of whole columns of every GEMV (all of K), so no partial sums
 * cross CTAs.  The weights are read from a strip-packed copy made once by gemv_pack_strips:
 *   column unit = an octet of 8 columns (for the SwiGLU epilogue a unit is two octets: gate, up);
 *   CTA c owns octets [start(c), start(c+1)), start(c) = floor(c * units / G) * octets_per_unit,
 *   taken two at a time (a pair = the 16 rows of one tensor-core step; a strip with an odd number
 *   of octets ends with a single);
 *   per (octet, K-group) one 544-byte record
 *     [32 lanes x 16 B : lane (g = column in octet, t) holds the packed words of rows t, t+4, t+8, t+12 of the group]
 *     [8 x (fp16 scale, fp16 zero-point)];
 *   the strip is contiguous and pair-major: strip base = start(c) * KG * 544, then for every pair all
 *   K-groups in order, each group as [record of the first octet][record of the second octet].
 * A pipeline stage is LB_CHAIN_GC consecutive K-groups of one pair (4352 bytes), brought by one 1-D
 * bulk copy and consumed by ONE warp. */
#define LB_CHAIN_MAX_OPS 32
#define LB_CHAIN_PACK_VERSION 1      /* bumped whenever the strip-packed byte layout changes */
#define LB_CHAIN_OP_GEMV 0
#define LB_CHAIN_OP_DELTANET 1      /* the DeltaNet mixer of one layer (deltanet_core.cuh); ext = lb_dn_layer_params in device memory */

#define LB_CHAIN_WARPS 16            /* consumer warps; every warp streams its own stages */
#define LB_CHAIN_THREADS (LB_CHAIN_WARPS * 32)
#define LB_CHAIN_RECORD 544          /* bytes per (octet, K-group) */
#define LB_CHAIN_GC 4                /* K-groups per stage */
#define LB_CHAIN_STAGE_BYTES (LB_CHAIN_GC * 2 * LB_CHAIN_RECORD)
#define LB_CHAIN_MAX_OCTETS 32       /* octets one CTA may own */
#define LB_CHAIN_GROUP_BYTES 448     /* shared-memory bytes of one K-group's block of the activation table (chain.cu) */
#define LB_CHAIN_MAIL_WORDS 17408    /* 8-byte words of one entry's mailbox: fp32 results one per word, fp16 results two per word */

typedef struct {
    const unsigned char* packed; /* strip-packed weights (gemv_pack_strips) */
    const void* x;
    void* y;
    const void* aux0;
    const void* aux1;
    uint16_t* x_out;
    int32_t K, N;
    int32_t kg;       /* K / 128 */
    int32_t units;    /* column units: N/8 octets, or N/16 pairs for the SwiGLU epilogue */
    int32_t upo;      /* octets per unit: 1 or 2 */
    int32_t x_mode, y_mode;
    float eps;
    int32_t type;     /* LB_CHAIN_OP_* */
    int32_t early_gate; /* set by the launcher (LB_X_F32_HEADNORM_SILU): the entry right before this one does not write the gate
                           vector aux1, so its silu is taken before this entry's grid barrier */
    const void* ext;  /* parameters of a non-GEMV entry, in device memory */
    int32_t x_src;    /* set by the launcher: index + 1 of the entry of this launch whose tagged results are this GEMV's x
                         (then x is read from that entry's mailbox and NO grid barrier precedes this entry); 0 = read p.x */
    int32_t mail;     /* set by the launcher: this GEMV also publishes its results as (value, tag) words in its mailbox */
} lb_chain_op;

typedef struct {
    lb_chain_op op[LB_CHAIN_MAX_OPS];
    uint32_t* status;
    uint32_t* sync;       /* [0] grid-barrier arrivals, [1] CTAs that left; both zero between launches; [2] tag base, advanced
                             by LB_CHAIN_MAX_OPS per launch */
    int32_t n_ops;
    int32_t slots;        /* ring slots per warp */
    int32_t table_rows;   /* packed rows (K/8) the activation table holds: the largest K of the chain */
    int32_t red_slots;    /* 16-float slots for per-stage column sums: the most stages any CTA has in one GEMV of the chain */
    int32_t trigger_op;   /* griddepcontrol.launch_dependents is issued when this GEMV starts */
    int32_t tab_len;      /* entries of a CTA's stage list: the stages of the busiest CTA, all GEMVs of the chain */
    int32_t pad_[2];
    unsigned long long* mail; /* mailboxes: LB_CHAIN_MAX_OPS regions of LB_CHAIN_MAIL_WORDS 8-byte words (see chain.cu) */
    unsigned long long* timeline; /* optional [gridDim.x][LB_CHAIN_MAX_OPS][8] stamps of thread 0.  [0] %globaltimer (ns) when the entry
                                     is reached (the one stamp that compares across SMs); the rest are the SM's cycle counter:
                                     [1] entry reached, [2] grid barrier left, [3] input vector arrived, [4] activation table ready,
                                     [5] every stage of the strip consumed, [6] column sums ready, [7] entry finished (epilogue and,
                                     under tensor parallelism, the exchange); a mixer or all-reduce entry stamps [3..7] when it ends */
} lb_chain_params;

/* gemv_pack_strips: reference format -> strip-packed (one thread per 32-bit word of the output) */
typedef struct {
    const uint32_t* qweight; /* [K/8, N] */
    const uint16_t* scales;  /* fp16 [K/128, N] */
    const uint32_t* qzeros;  /* [K/128, N/8] or NULL: zero-point 8 */
    uint32_t* out;           /* N/8 * K/128 records of 136 words */
    int32_t K, N;
    int32_t swiglu;          /* input columns are interleaved 64-wide (gate, up) blocks; output units are (gate octet, up octet) pairs */
    int32_t G;               /* CTAs the strips are cut for */
} lb_pack_params;

/* ---- batched int4 projection: Y[B,N] = X[B,K] W ------------------------- */
typedef struct {
    /* gemm_int4_tc: CUtensorMap over X [B, K] fp16, box 64 k x NT tokens, 128-byte swizzle */
    unsigned char tmap_x[128] __attribute__((aligned(64)));
    const uint32_t* qweight; /* [K/8, N] */
    const uint16_t* scales;  /* fp16 [K/128, N] */
    const uint32_t* qzeros;  /* [K/128, N/8] or NULL: zero-point 8 */
    const uint16_t* x;       /* fp16 [B, K] */
    void* y;                 /* fp32 or fp16 [B, N] */
    int32_t K, N, B;
    int32_t y_f32;
    uint32_t* status; /* device status word for bounded waits (the host layer always passes the context's) */
    int32_t reserved;
} lb_bgemm_params;

/* ---- dense bf16 [N,K] x vector ------------------------------------------ */
typedef struct {
    const uint16_t* w; /* bf16 [N,K] row-major */
    const void* x;     /* fp16 or fp32 [K] */
    float* y;          /* fp32 [N] */
    const void* norm_w; /* bf16 [K] when x_mode == LB_X_F32_RMSNORM */
    int32_t N, K;
    int32_t x_mode; /* LB_X_F16 | LB_X_F32 | LB_X_F32_RMSNORM */
    float eps;
    float* part_val;  /* optional [gridDim.x]: largest y of the rows this CTA produced ... */
    int32_t* part_idx; /* ... and its row (smallest row on ties), for the greedy-sampling reduction */
    uint32_t* status;  /* device status word: set when a bounded wait for a weight row runs out (the rows left stay unwritten) */
} lb_dense_params;

/* ---- gated DeltaNet step -------------------------------------------------- */
typedef struct {
    float* state;      /* fp32 [HV,128,128] updated in place */
    const void* q;     /* [HK,128] bf16 or fp32 */
    const void* k;     /* [HK,128] */
    const void* v;     /* [HV,128] */
    const float* z;    /* fp32 [HV,128] or NULL: no silu(z) output gate */
    const float* g;    /* fp32 [HV] decay */
    const float* beta; /* fp32 [HV] */
    float* out;        /* fp32 [HV,128] */
    int32_t HV, HK;
} lb_deltanet_params;

typedef struct {
    const float* a;        /* [n] in_proj_a output */
    const float* a_log;    /* [n] */
    const float* dt_bias;  /* [n] */
    const float* b;        /* [n] in_proj_b output */
    float* g;              /* [n] decay out */
    float* beta;           /* [n] beta out */
    int32_t n;
} lb_decay_params;

/* ---- whole DeltaNet mixer of one layer (between the qkvz projection and the out projection) */
typedef struct {
    const float* qkvz;       /* fp32 [2*HK*128 + 2*HV*128]: q | k | v | z from the fused projection */
    const uint16_t* xn;      /* fp16 [hidden]: the normalised layer input (as the projection used it) */
    const uint16_t* proj_a;  /* bf16 [HV, hidden] in_proj_a */
    const uint16_t* proj_b;  /* bf16 [HV, hidden] in_proj_b */
    const float* a_log;      /* fp32 [HV] */
    const uint16_t* dt_bias; /* bf16 [HV] */
    const uint16_t* conv_w;  /* bf16 [4, C] planar, tap 0 = current token; C = 2*HK*128 + HV*128 */
    float* conv_ring;        /* fp32 [4, C]: slot (pos & 3) receives the current token's pre-conv values */
    float* state;            /* fp32 [HV,128,128] */
    float* out;              /* fp32 [HV,128] read-out (before the per-head norm and z gate) */
    const int* pos;          /* device int: position of the token being decoded */
    int32_t HV, HK, hidden;
    int32_t h0;              /* first global value head of this shard (tensor parallel), for nothing but clarity */
} lb_dn_layer_params;

/* ---- causal attention of a prompt chunk (pf_attn_prepare, pf_attn_chunk) --- */
typedef struct {
    const float* proj;        /* fp32 [T, ld]: per token, per head 256 query then 256 gate columns | k [HKV,256] | v [HKV,256] */
    const uint16_t* q_norm_w; /* bf16 [256] */
    const uint16_t* k_norm_w; /* bf16 [256] */
    uint16_t* k_cache;        /* bf16 [ctx,HKV,256]: rows pos0 .. pos0+T-1 are written by pf_attn_prepare */
    uint16_t* v_cache;
    uint16_t* qh;             /* bf16 [T,HQ,256]: the normalised, rotated, pre-scaled queries, leading term */
    uint16_t* ql;             /* bf16 [T,HQ,256]: what the rounding of qh left over */
    uint16_t* out;            /* fp16 [T,HQ,256]: attention output x sigmoid(gate), the o projection's input */
    int32_t ld, HQ, HKV, pos0, T, rot_dims;
    float eps;
    double rope_freq[64];     /* theta^(-i/(rot_dims/2)), computed on the host in double */
} lb_pf_attn_params;
/* pf_attn_chunk: query rows per CTA (16 per warp), threads, dynamic shared memory (two query tiles of ROWS x 528 B, two
 * stages of 32 K rows + 32 V rows x 528 B) */
#define LB_PF_ATTN_ROWS 32
#define LB_PF_ATTN_THREADS 64
#define LB_PF_ATTN_SMEM (2 * LB_PF_ATTN_ROWS * 528 + 2 * 2 * 32 * 528)

/* ---- GQA decode attention ------------------------------------------------- */
typedef struct {
    const void* q;        /* [HQ,256] bf16 or fp32 (raw, before norm) */
    const void* k_new;    /* [HKV,256] raw new key */
    const void* v_new;    /* [HKV,256] new value */
    const void* gate;     /* [HQ,256] or NULL */
    const uint16_t* q_norm_w; /* bf16 [256] or NULL: skip q/k norm */
    const uint16_t* k_norm_w; /* bf16 [256] */
    uint16_t* k_cache;    /* bf16 [ctx,HKV,256] */
    uint16_t* v_cache;
    float* out;           /* fp32 [HQ,256] */
    float* scratch;       /* split partials: [HKV][splits][G][(256 acc) + m + l] */
    uint32_t* counters;   /* one per kv head, zero between launches */
    const int* pos_ptr;   /* when non-NULL the position is read from device memory (graph replay) */
    int32_t pos;          /* position of the new token; rows [0,pos] are attended */
    int32_t HQ, HKV;
    int32_t splits;
    int32_t in_dtype;     /* 0 = bf16 inputs, 1 = fp32 inputs */
    int32_t gate_stride;  /* elements between consecutive heads of gate (256, or 512 when interleaved with q) */
    int32_t q_stride;     /* elements between consecutive heads of q */
    int32_t rot_dims;
    float rope_theta;
    float eps;
    double rope_freq[64]; /* theta^(-i/(rot_dims/2)), i < rot_dims/2 <= 64, computed on the host in double */
    uint32_t* status;     /* device status word for bounded waits (attn_decode_mma); may be NULL */
    int32_t coop;         /* attn_decode_mma: the grid fits the SMs one CTA each, so the CTAs of a KV head may wait for each
                             other and share the slice merge (counters[kv] arrivals, counters[8 + kv] finished) */
    int32_t max_ctx;      /* rows the caches hold (0 = not checked): a position outside [0, max_ctx) sets status
                             LB_DEV_POS_RANGE and the kernel returns without reading or writing a cache row */
} lb_attn_params;

/* ---- dense bf16 rows x one fp32 vector with fused prologue and epilogue (rows_gemv) ------------------------
 * One or two row-major bf16 matrices [rows, K] against vectors built in shared memory.  Rows are taken two at a time (a
 * pair), pair p of the launch (matrix 0 first) by CTA p % gridDim.x; the number of rows is even (a zero row pads an odd
 * matrix) and K is a multiple of 64. */
#define LB_RG_THREADS 256
#define LB_RG_WARPS 8
#define LB_RG_SEG 1024 /* elements of one row in a pipeline stage */
enum { LB_RG_X_NORM = 0, /* vector of matrix i = norm(x) with that matrix's weights */
       LB_RG_X_CAT = 1   /* one vector: the mixer's output (norm of its parts and gate applied here), then the feed-forward's activations */ };
/* norms in front of a product */
enum { LB_NORM_RMS_1P = 0, /* x / rms(x) * (1 + w) */
       LB_NORM_RMS = 1,    /* x / rms(x) * w */
       LB_NORM_LAYER = 2   /* (x - mean) / sd * w + b */ };
/* epilogues, shared with the matrix products of a prompt chunk (lb_dgemm_params) */
enum { LB_DY_STORE = 0,    /* y[n] = r */
       LB_DY_RELU_GLU = 1, /* rows come as (gate, up) pairs: y[pair] = relu(gate) * up */
       LB_DY_RESIDUAL = 2, /* y[n] += mult * r */
       LB_DY_SOFTCAP = 3,  /* y[n] = cap * tanh(r / cap), cap 0: y[n] = r; with part_val: arg-max candidates */
       LB_DY_RELU2 = 4,    /* y[n] = max(r, 0)^2 */
       LB_DY_CLAMP_GLU = 5, /* (gate, up) pairs: g = min(gate, limit), u = clamp(up, -limit, limit), y[pair] = g sigmoid(alpha g) (u + 1) */
       LB_DY_HEADS = 6     /* prompt: bf16 y[n / head * head_p + n % head] */ };
typedef struct {
    const uint16_t* w;      /* bf16 [rows, K] */
    const uint16_t* norm_w; /* bf16 [width] (LB_RG_X_NORM) */
    const uint16_t* norm_b; /* bf16 [width] (LB_NORM_LAYER) */
    float* y;
    int32_t rows;           /* rows with a result (the allocation holds an even number) */
    int32_t y_mode;
} lb_rg_mat;
typedef struct {
    lb_rg_mat mat[2];
    const float* x;         /* LB_RG_X_NORM: fp32 [width] */
    const float* mix;       /* LB_RG_X_CAT: fp32 [n_mix] */
    const float* gate;      /* fp32 [n_mix]: mix *= silu(gate); NULL = no gate */
    const uint16_t* head_w; /* mix = rmsnorm of each part of vdim values * head_w first (bf16 [vdim]; [n_mix] with gate_first); NULL = none */
    const float* act;       /* fp32 [n_act] */
    float* part_val;        /* [gridDim.x] arg-max candidates (LB_DY_SOFTCAP), or NULL */
    int32_t* part_idx;
    uint32_t* status;
    int32_t n_mat, K, width, x_mode;
    int32_t n_mix, n_mix_pad, vdim, n_act; /* the feed-forward part starts at n_mix_pad */
    int32_t stages;         /* ring stages per warp */
    int32_t split;          /* pieces a row pair is cut into along K: 1, or one per stage segment */
    int32_t segs;           /* ceil(K / LB_RG_SEG) */
    int32_t x_cols;         /* columns of a vector one CTA holds: K, or the longer half where two CTAs share a row */
    int32_t norm;           /* LB_NORM_* (LB_RG_X_NORM) */
    int32_t gate_first;     /* mix is gated before its norm, not after */
    /* experts: a matrix is a stack of `experts`; sel[0..parts) (a row of a table, row *sel_row) names the ones this token uses */
    const int32_t* sel;     /* NULL: no experts */
    const int32_t* sel_row; /* row of sel; written well before the launch in front of this one has started */
    int32_t parts;          /* experts per token (1 without experts) */
    int32_t sel_rows;       /* LB_RG_X_NORM: rows of one expert; mat.rows = parts * sel_rows, results of part i start at y[i * y_part] */
    int32_t y_part;
    int32_t k_part;         /* LB_RG_X_CAT: columns of one expert; K = parts * k_part, expert e is [rows padded to even][k_part].  Else K */
    int32_t segs_part;      /* ceil(k_part / LB_RG_SEG); segs = parts * segs_part */
    float limit, alpha;     /* LB_DY_CLAMP_GLU */
    float eps, mult, cap;
} lb_rows_gemv_params;
#define LB_RG_MAX_PARTS 32

/* ---- dense products of a prompt chunk: Y[T, N] = X[T, K] W[N, K]^T, one or two of them in one launch --------- */
#define LB_DG_ROWS 128  /* weight rows per tile = M of the product */
#define LB_DG_KB 64     /* k per pipeline stage: one 128-byte swizzled row */
#define LB_DG_THREADS 192
#define LB_DG_MAX_STAGES 8
typedef struct {
    unsigned char tmap_w[2][128] __attribute__((aligned(64))); /* bf16 [rows, K], box 64 x 128, 128-byte swizzle */
    unsigned char tmap_x[2][128] __attribute__((aligned(64))); /* bf16 [T, K], box 64 x NT, 128-byte swizzle */
    const uint16_t* w[2]; /* the same operands as pointers (gemm_f32_simt) */
    const void* x[2];
    void* y[2];
    int32_t rows[2], y_mode[2], ld_y[2];
    int32_t tiles[2];     /* row tiles of each product (tiles[1] = 0: one product) */
    int32_t y_f32[2];     /* LB_DY_RELU_GLU: y is fp32 (else bf16) */
    int32_t T, NT, t_tiles, K, ld_x, stages, tmem_cols;
    int32_t head[2], head_p[2]; /* LB_DY_HEADS */
    float mult, cap, limit, alpha;
    uint32_t* status;
    /* experts (one product): w is a stack of experts, x and y have the chunk's (token, expert) assignments sorted by
     * expert; a token tile is plan_tiles[i] = (expert, first assignment, end of the expert's assignments, 0), i < *plan_n */
    const int32_t* plan_tiles; /* NULL: no experts */
    const int32_t* plan_n;
    int32_t expert_rows; /* rows of the stack from one expert to the next */
} lb_dgemm_params;

/* a chunk's (token, expert) assignments sorted by expert (moe_plan) */
typedef struct {
    const int32_t* tokens; /* [T] */
    const int32_t* table;  /* [vocab, top]: the experts of a token id */
    int32_t* place;        /* [T, top]: row of the assignment in sorted order */
    int32_t* tiles;        /* as lb_dgemm_params.plan_tiles */
    int32_t* n_tiles;
    int32_t T, top, experts, NT;
} lb_moe_plan_params;
#define LB_MOE_MAX_EXPERTS 1024

/* norm of a chunk's rows with up to two weights: h_i[t] = norm(x[t]) with w_i (and b_i).  Before it, optionally, x[t] += mult * the sum of the
 * token's rows of y (place: a layer's expert outputs); after it, optionally, the row goes to `scatter` places instead of place t */
typedef struct {
    float* x;            /* fp32 [T, ld_x] */
    const uint16_t* w[2];
    const uint16_t* b[2]; /* LB_NORM_LAYER */
    void* h[2];          /* bf16 (or fp32) [T, ld]; h[1] may be NULL */
    int32_t width, ld, ld_x, f32, norm;
    float eps;
    const void* y;       /* NULL: nothing to add; bf16 (or fp32) [assignments, ld_y] */
    const int32_t* y_place; /* [T, y_top] */
    int32_t y_top, ld_y;
    float y_mult;
    const int32_t* scatter; /* NULL, or [T, top]: h_0[scatter[t, i]] = row */
    int32_t top;
} lb_norm2_params;

/* ---- attention over the current block of positions, general head sizes (window_attention.cu) ---------------- */
#define LB_WA_MAX_DIM 256
#define LB_WA_MAX_SPLITS 64 /* position slices of a decode step */
typedef struct {
    const float* proj;   /* fp32 [T, ld]: q | k | v sections at the given offsets */
    void* k_cache;       /* bf16 (or fp32) [max_ctx, KV, dim_p]: rotated keys; padding columns are zero */
    void* v_cache;       /* [max_ctx, KV, vdim_p]: normed, rotated values */
    const double* freq_k; /* [rot_dims / 2] radians per position */
    const double* freq_v; /* [vdim / 2]; NULL: values are not rotated */
    float* out;          /* fp32 [H * vdim] of one token (decode) ... */
    void* cat;           /* ... or, when not NULL, rows [T, cat_ld] of bf16 / fp32 (prompt) */
    uint16_t* qh;        /* prompt, bf16: rotated queries x scale x log2(e) as two bf16 terms [T, H, dim_p] */
    uint16_t* ql;
    float* scratch;      /* partials of the position slices: [groups][splits][heads per CTA][vdim_p + 2] */
    uint32_t* counters;  /* one per (KV head, head group), zero between launches */
    const int32_t* pos_ptr; /* position of token 0 in device memory, or NULL: pos0 */
    uint32_t* status;
    int32_t ld, q_off, k_off, v_off; /* k_off < 0: the cache belongs to another layer, which has filled it */
    int32_t H, KV, dim, vdim, dim_p, vdim_p, rot_dims;
    int32_t block;       /* position i sees j <= i with the same floor(j / block); 0: every j <= i */
    int32_t v_norm;      /* values are divided by their root mean square */
    int32_t sink;        /* 1 is added to the soft-max denominator */
    int32_t pos0, T, max_ctx, splits, cat_ld;
    float scale, eps;
    /* prompt, bf16: the last tail_p of a key's dim_p values are shared by all heads: k_tail rows (of tail_ld values), k_cache rows without them */
    const uint16_t* k_tail;
    int32_t tail_p, tail_ld;
    const uint16_t* sink_w; /* bf16 [H]: exp(sink_w) is added to the denominator instead of 1 */
} lb_wattn_params;
/* wattn_chunk_*: query rows per CTA (16 per warp), keys per staged block */
#define LB_WA_ROWS 64
#define LB_WA_THREADS 128
#define LB_WA_KV 32

/* ---- linear attention with one decay per key channel (decay_attention.cu) ----------------------------------- */
enum { LB_DA_HGRN2 = 0, LB_DA_GLA = 1 };
typedef struct {
    const float* proj;    /* fp32 [T, ld]: sections at the offsets below */
    const uint16_t* a2;   /* GLA: bf16 [H * dk, rank] */
    const uint16_t* bias; /* bf16 [H * dk]: added to the gate's pre-activation */
    const uint16_t* lower; /* HGRN2: bf16 [H * dk] */
    const uint16_t* head_w; /* bf16 [dv]: per-head norm of the output (prompt: da_finish) */
    float* state;         /* fp32 [H, dk, dv] */
    float* q;             /* prompt: fp32 [T, H, dk_p], likewise k and a (padding columns zero) */
    float* k;
    float* a;
    float* o;             /* fp32 [T, H * dv] */
    void* cat;            /* prompt: bf16 / fp32 rows [T, cat_ld] */
    float* seg_state;     /* prompt in segments: fp32 [segments, H, dk, dv] and ... */
    float* seg_decay;     /* ... [segments, H, dk_p] */
    int32_t kind, ld, q_off, k_off, v_off, g_off; /* k_off: HGRN2 the gate's section; g_off < 0: no output gate */
    int32_t a1_off, rank; /* GLA: section of the low-rank pre-activation */
    int32_t H, dk, dv, dk_p, T, cat_ld, cat_f32;
    int32_t seg;          /* prompt: tokens per segment, a multiple of 4 (T or more: one segment) */
    float q_scale, inv_tau, eps;
} lb_decay_params2;

/* ---- attention over a cached latent (latent_attention.cu) ---------------------------------------------------
 * A position is cached as one row [latent c (rank_p) | rotated key part shared by all heads (rot_p)]; a head's key is [W_uk c | that part],
 * its value W_uv c. */
#define LB_LA_MAX_RANK 512
#define LB_LA_MAX_ROT 128
#define LB_LA_MAX_SPLITS 64
#define LB_LA_TOKENS 8 /* tokens a CTA of lat_query / lat_out walks with one read of its weights */
#define LB_LA_KEYS 64  /* lat_rows_bf16: cache rows per staged block */
typedef struct {
    const float* proj;     /* fp32 [T, ld]: at kv_off the latent (rank) and the shared key part (rot), before norm and rotation */
    const float* q;        /* fp32 [T, H * (dim + rot)] */
    const uint16_t* uk;    /* bf16 [H * dim, rank_p] */
    const uint16_t* uv;    /* bf16 [H * vdim, rank_p] */
    const uint16_t* c_norm; /* bf16 [rank] */
    const uint16_t* sink;  /* bf16 [H]: exp(sink) joins the denominator; NULL: none */
    const double* freq;    /* [rot / 2] radians per position */
    void* cache;           /* bf16 (or fp32) [max_ctx, rank_p + rot_p]; padding columns are zero */
    float* ql;             /* fp32 [T, H, rank_p + rot_p]: (W_uk^T q | rotated q) * scale */
    float* part;           /* fp32 [T * H][splits][rank_p + 2]: weighted sum of latents, maximum, denominator of a slice of positions */
    float* out;            /* fp32 [H * vdim] of one token (decode) ... */
    void* cat;             /* ... or, when not NULL, rows [T, cat_ld] of bf16 / fp32 */
    uint16_t* qh;          /* lat_prepare: queries x scale x log2(e) as two bf16 terms [T, H, dim_p + rot_p]; NULL: cache rows only */
    uint16_t* ql16;
    const int32_t* pos_ptr; /* position of token 0 in device memory, or NULL: pos0 */
    uint32_t* status;
    int32_t ld, kv_off, H, dim, dim_p, vdim, rank, rank_p, rot, rot_p;
    int32_t pos0, T, max_ctx, splits, cat_ld, stages;
    float rot_mul, scale, eps;
} lb_latent_params;

/* ---- state-space recurrence with a scalar decay per head (ssm.cu) -------------------------------------------- */
#define LB_SSM_MAX_TAPS 8
#define LB_SSM_MAX_STATE 256
#define LB_SSM_SEG 64  /* tokens per block of ssm_chunk_* */
#define LB_SSM_COLS 32 /* value columns per CTA */
#define LB_SSM_CONV_TOKENS 16 /* tokens per thread of ssm_conv */
typedef struct {
    const float* proj;      /* fp32 [T, ld]: z [H V] | x [H V] | B [G N] | C [G N] | dt [H] */
    const uint16_t* conv_w; /* bf16 [channels, taps], last column = the current token */
    const uint16_t* conv_b; /* bf16 [channels] */
    const uint16_t* dt_bias; /* bf16 [H] */
    const uint16_t* a_log;
    const uint16_t* d;
    const uint16_t* norm_w; /* bf16 [H V] */
    float* state;           /* fp32 [H, N, V] */
    float* ring;            /* fp32 [taps, channels]: slot position % taps holds that position's values before the convolution */
    float* y;               /* fp32 [T, H V] */
    void* xbc;              /* prompt: x [H, V_p] | B [G, N_p] | C [G, N_p] after the convolution, bf16 (or fp32), padding zero, rows of ld_xbc */
    float* dt;              /* prompt: fp32 [T, H] step sizes */
    float* seg_state;       /* prompt in segments: fp32 [segments, H, N, V] and ... */
    float* seg_decay;       /* ... [segments, H], logarithms */
    void* cat;              /* prompt: gated, normed rows [T, cat_ld] */
    const int32_t* pos_ptr; /* decode: position in device memory */
    int32_t ld, H, V, V_p, N, N_p, G, taps, channels, ld_xbc, norm_groups;
    int32_t pos0, T, cat_ld, f32;
    int32_t seg;            /* ssm_chunk, ssm_local: tokens per segment, a multiple of LB_SSM_SEG (T or more: one segment) */
    float eps;
} lb_ssm_params;

/* ---- tensor-parallel exchange (comm.cu) ----------------------------------------------- */
#define LB_TP_MAX 8
/* Exchange buffer of one rank (every rank maps every peer's): float [2][size][n_max] partial vectors (slot = exchange
 * parity, then the rank that produced the vector), float [n_max] for the sampling record, the flag words, then
 * uint2 [2][size][n_max] (value, generation) words.
 * "Pull" exchanges (tp_allreduce_add): rank q leaves its partial in ITS OWN buffer at (slot, q),
 * raises flag [q] in every peer's flag array (system-scope release), readers load the vector from q's buffer.
 * "Pushed" exchanges (LB_Y_TP_ALLREDUCE): the thread that owns column n on rank q stores the 8-byte word (partial sum,
 * generation) into EVERY rank's word array at (slot, q, n) -- one store, delivered whole, so no fence and no flag -- and
 * then polls its own rank's array until the words of column n from all ranks carry this generation.  The same thread owns
 * column n on every rank (same matrix, same number of SMs), so nothing else has to be synchronised. */
typedef struct {
    float* x;                          /* residual stream [n] on this GPU */
    float* partials[LB_TP_MAX];        /* every rank's exchange buffer (peer pointers) */
    unsigned* peer_flags[LB_TP_MAX];   /* every rank's pull-flag array: unsigned [LB_TP_MAX] */
    unsigned* my_flags;                /* this rank's pull-flag array (local) */
    unsigned* gen;                     /* this rank's generation counter (local, advanced by the kernel) */
    unsigned* status;
    unsigned long long* words[LB_TP_MAX]; /* every rank's (value, generation) word array [2][size][n_max] (peer pointers) */
    int32_t n, n_max, slot, rank, size;
    int32_t pad_;
} lb_tp_params;
/* float offset of partial vector (slot, rank q) inside an exchange buffer; slot 2 is the sampling record */
#define LB_TP_PARTIAL(p, slot_, q) ((size_t)((slot_) == 2 ? 2 * (p).size : (slot_) * (p).size + (q)) * (size_t)(p).n_max)

typedef struct {
    lb_tp_params tp;        /* slot = 2: the record (logit, token) lives at the start of that slot */
    const float* cand_val;  /* this rank's per-CTA candidates from the LM-head kernel */
    const int32_t* cand_idx; /* rows inside this rank's vocabulary shard */
    int32_t n_cand, vocab_offset;
    int32_t* out_idx;
    int32_t* next_token;
    int32_t* pos;
} lb_tp_argmax_params;

#endif
