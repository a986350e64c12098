/* The prompt pass: runs n tokens through the model in chunks (lb_model.pf_chunk tokens each) and leaves the state a
 * token-by-token decode of the same tokens leaves, then the sampled next token (lb_model_prefill) or the logits of chosen
 * tokens (lb_model_forward).  The layer order is that of compiler/megakernel-link.ls:281-525; what a layer does to a chunk is
 * the architecture's pf_layer: every projection is one matrix product per chunk (weights read once), recurrences walk the
 * chunk inside one launch with the state held on chip, attention is one causal tensor-core kernel over the chunk's tokens.
 * Single GPU only.
 *
 * Up to lb_arch.pf_streams chunks are in flight at a time, each on its own stream with its own buffer set: chunk c+1 follows
 * chunk c one layer behind (layer l of chunk c+1 waits for the event recorded after layer l of chunk c: recurrent states,
 * convolution rings and cache rows of a layer pass from chunk to chunk in order).  The kernels of a layer that cannot fill the
 * GPU (recurrences, attention, the element-wise kernels) run beside the other chunks' projections instead of alone.
 */
#include "lb_model_priv.h"

struct lb_prefill_ws {
    pf_set set[LB_PF_MAX_STREAMS]; /* one per stream */
    CUdeviceptr rows, row_logits;  /* residual rows whose logits are wanted, and those logits; grown on demand */
    int rows_cap;
    CUstream stream[LB_PF_MAX_STREAMS];
    CUevent* layer_done[LB_PF_MAX_STREAMS]; /* [n_layers] per stream: recorded after a chunk's layer l */
    CUevent fork, join[LB_PF_MAX_STREAMS];
};

void lb_prefill_ws_free(lb_model* m);

static int ws_fill(lb_model* m) {
    lb_prefill_ws* ws = (lb_prefill_ws*)calloc(1, sizeof *ws);
    if (!ws) return LB_ERR_NOMEM;
    m->ws = ws; /* ws_alloc releases whatever a failure below leaves behind */
    lb_ctx* ctx = m->c;
    const lb_model_cfg* c = &m->cfg;
    size_t bytes[LB_PF_MAX_BUFS] = {0};
    m->arch->pf_sizes(m, bytes);
    for (int s = 0; s < m->arch->pf_streams; s++) {
        for (int i = 0; i < LB_PF_MAX_BUFS; i++) {
            if (!bytes[i]) continue;
            LB_TRY(lb_dalloc(m, &ws->set[s].b[i], bytes[i]));
            LB_CU(ctx, lb_drv.MemsetD8Async(ws->set[s].b[i], 0, bytes[i], ctx->stream)); /* padding columns stay zero */
        }
        LB_CU(ctx, lb_drv.StreamCreate(&ws->stream[s], CU_STREAM_NON_BLOCKING));
        ws->layer_done[s] = (CUevent*)calloc((size_t)c->n_layers, sizeof(CUevent));
        if (!ws->layer_done[s]) return LB_ERR_NOMEM;
        for (int l = 0; l < c->n_layers; l++) LB_CU(ctx, lb_drv.EventCreate(&ws->layer_done[s][l], CU_EVENT_DISABLE_TIMING));
        LB_CU(ctx, lb_drv.EventCreate(&ws->join[s], CU_EVENT_DISABLE_TIMING));
    }
    LB_CU(ctx, lb_drv.EventCreate(&ws->fork, CU_EVENT_DISABLE_TIMING));
    return LB_OK;
}

static int ws_alloc(lb_model* m) {
    if (m->ws) return LB_OK;
    const int st = ws_fill(m);
    if (st != LB_OK) lb_prefill_ws_free(m); /* never leave half a workspace behind for the next call */
    return st;
}

pf_set* lb_prefill_set(lb_model* m, int s) { return &m->ws->set[s]; }

static int rows_reserve(lb_model* m, int n) {
    lb_prefill_ws* ws = m->ws;
    if (n <= ws->rows_cap) return LB_OK;
    LB_CU(m->c, lb_drv.StreamSynchronize(m->c->stream));
    if (ws->rows) lb_drv.MemFree(ws->rows);
    if (ws->row_logits) lb_drv.MemFree(ws->row_logits);
    ws->rows = ws->row_logits = 0;
    ws->rows_cap = 0;
    LB_TRY(lb_dalloc(m, &ws->rows, (size_t)n * m->cfg.hidden * 4));
    LB_TRY(lb_dalloc(m, &ws->row_logits, (size_t)n * m->cfg.vocab * 4));
    ws->rows_cap = n;
    return LB_OK;
}

void lb_prefill_ws_free(lb_model* m) {
    lb_prefill_ws* ws = m->ws;
    if (!ws) return;
    for (int s = 0; s < LB_PF_MAX_STREAMS; s++) {
        if (ws->stream[s]) lb_drv.StreamSynchronize(ws->stream[s]);
        for (int i = 0; i < LB_PF_MAX_BUFS; i++)
            if (ws->set[s].b[i]) lb_drv.MemFree(ws->set[s].b[i]);
        if (ws->layer_done[s]) {
            for (int l = 0; l < m->cfg.n_layers; l++)
                if (ws->layer_done[s][l]) lb_drv.EventDestroy(ws->layer_done[s][l]);
            free(ws->layer_done[s]);
        }
        if (ws->join[s]) lb_drv.EventDestroy(ws->join[s]);
        if (ws->stream[s]) lb_drv.StreamDestroy(ws->stream[s]);
    }
    if (ws->fork) lb_drv.EventDestroy(ws->fork);
    if (ws->rows) lb_drv.MemFree(ws->rows);
    if (ws->row_logits) lb_drv.MemFree(ws->row_logits);
    free(ws);
    m->ws = NULL;
}

/* tokens[0..n) at positions pos0..: every layer; the residual row after the last layer of tokens want[0..n_want) (ascending)
 * goes to rows, one after the other */
static int run_chunks(lb_model* m, const int* tokens, int n, int pos0, const int* want, int n_want, CUdeviceptr rows) {
    lb_ctx* c = m->c;
    const lb_model_cfg* cfg = &m->cfg;
    lb_prefill_ws* ws = m->ws;
    const int H = cfg->hidden, CH = m->pf_chunk, NS = m->arch->pf_streams;
    CUstream main_stream = c->stream;
    LB_CU(c, lb_drv.MemcpyHtoDAsync(m->d_tokens + (size_t)pos0 * 4, tokens, (size_t)n * 4, main_stream));
    LB_CU(c, lb_drv.StreamSynchronize(main_stream)); /* the caller's token array may be pageable */
    /* the chunk streams start behind what the caller's stream holds so far (an earlier decode step, the token copy) */
    LB_CU(c, lb_drv.EventRecord(ws->fork, main_stream));
    for (int s = 0; s < NS; s++) LB_CU(c, lb_drv.StreamWaitEvent(ws->stream[s], ws->fork, 0));
    int st = LB_OK, chunk = 0, wi = 0;
    for (int c0 = 0; c0 < n && st == LB_OK; c0 += CH, chunk++) {
        const int T = n - c0 < CH ? n - c0 : CH, s = chunk % NS, prev = (chunk + NS - 1) % NS;
        pf_set* w = &ws->set[s];
        c->stream = ws->stream[s]; /* every launch below goes to this chunk's stream */
        CUdeviceptr toks = m->d_tokens + (size_t)(pos0 + c0) * 4;
        void* params[] = {&m->embed, &toks, &w->b[0], (void*)&H};
        st = m->bigram ? lb_model_embed_bigram(m, 0, 0, pos0 + c0, T, w->b[0]) : lb_launch(c, LBK_pf_embed, (unsigned)T, 1, 1, 256, 0, params, 1);
        for (int l = 0; l < cfg->n_layers && st == LB_OK; l++) {
            /* layer l's state, ring and cache rows come from the previous chunk's layer l (on the stream before this one) */
            if (chunk > 0 && lb_drv.StreamWaitEvent(c->stream, ws->layer_done[prev][l], 0) != CUDA_SUCCESS) st = LB_ERR_CUDA;
            if (st == LB_OK) st = m->arch->pf_layer(m, w, l, pos0 + c0, T);
            if (st == LB_OK && lb_drv.EventRecord(ws->layer_done[s][l], c->stream) != CUDA_SUCCESS) st = LB_ERR_CUDA;
        }
        while (st == LB_OK && wi < n_want && want[wi] < c0 + T) { /* runs of neighbouring rows are one copy */
            int run = 1;
            while (wi + run < n_want && want[wi + run] == want[wi] + run && want[wi + run] < c0 + T) run++;
            if (lb_drv.MemcpyDtoDAsync(rows + (size_t)wi * H * 4, w->b[0] + (size_t)(want[wi] - c0) * H * 4, (size_t)run * H * 4, c->stream) != CUDA_SUCCESS)
                st = LB_ERR_CUDA;
            wi += run;
        }
    }
    c->stream = main_stream;
    /* the caller's stream continues behind all chunk streams (also after a failed launch: nothing may still be running
     * on buffers the caller is about to reuse) */
    for (int s = 0; s < NS; s++) {
        LB_CU(c, lb_drv.EventRecord(ws->join[s], ws->stream[s]));
        LB_CU(c, lb_drv.StreamWaitEvent(main_stream, ws->join[s], 0));
    }
    return st == LB_ERR_CUDA ? lb_fail(c, LB_ERR_CUDA, "prompt pass: a stream operation failed") : st;
}

static int check_tokens(lb_model* m, const char* who, const int* tokens, int n, int pos0) {
    lb_ctx* c = m->c;
    const lb_model_cfg* cfg = &m->cfg;
    if (m->tp_size != 1) return lb_fail(c, LB_ERR_STATE, "%s: single GPU only (this model is shard %d of %d)", who, m->tp_rank, m->tp_size);
    if (pos0 + n > cfg->max_ctx) return lb_fail(c, LB_ERR_INVALID, "%s: %d tokens from position %d run past the context of %d rows", who, n, pos0, cfg->max_ctx);
    for (int i = 0; i < n; i++)
        if (tokens[i] < 0 || tokens[i] >= cfg->vocab) return lb_fail(c, LB_ERR_INVALID, "%s: token %d at %d out of range", who, tokens[i], i);
    if (!m->globals_loaded) return lb_fail(c, LB_ERR_STATE, "model: globals have no weights");
    return LB_OK;
}

LB_API int lb_model_prefill(lb_model* m, const int* tokens, int n, int pos0, int* next_out) {
    if (!m || !tokens || n < 1 || pos0 < 0) return LB_ERR_INVALID;
    lb_ctx* c = m->c;
    LB_TRY(check_tokens(m, "lb_model_prefill", tokens, n, pos0));
    LB_CU(c, lb_drv.CtxSetCurrent(c->cu_ctx));
    LB_TRY(ws_alloc(m));
    const int last = n - 1;
    LB_TRY(run_chunks(m, tokens, n, pos0, &last, 1, m->X)); /* the last prompt token's hidden state -> final norm, LM head, sample */
    LB_CU(c, lb_drv.MemsetD32Async(m->d_pos, (unsigned)(pos0 + n - 1), 1, c->stream)); /* the sampling kernel advances it */
    LB_TRY(m->arch->head(m, m->X));
    LB_TRY(lb_model_launch_sampler(m));
    m->host_pos = pos0 + n;
    return next_out ? lb_model_read_next(m, next_out) : LB_OK;
}

LB_API int lb_model_forward(lb_model* m, const int* tokens, int n, int pos0, const int* want, int n_want, float* logits_out) {
    if (!m || !tokens || n < 1 || pos0 < 0 || n_want < 0 || (n_want && (!want || !logits_out))) return LB_ERR_INVALID;
    lb_ctx* c = m->c;
    LB_TRY(check_tokens(m, "lb_model_forward", tokens, n, pos0));
    for (int i = 0; i < n_want; i++)
        if (want[i] < 0 || want[i] >= n || (i && want[i] <= want[i - 1])) return lb_fail(c, LB_ERR_INVALID, "lb_model_forward: wanted places must ascend inside the portion");
    LB_CU(c, lb_drv.CtxSetCurrent(c->cu_ctx));
    CUdeviceptr src = 0;
    if (n == 1) { /* one token is a decode step, the one generation replays */
        if (!m->graph) LB_TRY(lb_model_capture(m));
        LB_TRY(lb_model_set_input(m, tokens[0], pos0));
        LB_TRY(lb_model_replay(m, 1));
        src = m->logits;
    } else {
        LB_TRY(ws_alloc(m));
        LB_TRY(rows_reserve(m, n_want));
        lb_prefill_ws* ws = m->ws;
        LB_TRY(run_chunks(m, tokens, n, pos0, want, n_want, ws->rows));
        for (int r = 0; r < n_want; r += m->pf_chunk) {
            const int k = n_want - r < m->pf_chunk ? n_want - r : m->pf_chunk;
            LB_TRY(m->arch->head_rows(m, ws->rows + (size_t)r * m->cfg.hidden * 4, k, ws->row_logits + (size_t)r * m->cfg.vocab * 4));
        }
        src = ws->row_logits;
        m->host_pos = pos0 + n;
    }
    if (n_want) LB_CU(c, lb_drv.MemcpyDtoHAsync(logits_out, src, (size_t)n_want * m->cfg.vocab * 4, c->stream));
    uint32_t word = 0;
    return lb_device_status(c, &word); /* synchronises */
}
