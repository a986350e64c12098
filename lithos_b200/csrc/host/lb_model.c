/* The runtime every model shares: activation and sampling buffers, the decode step (embedding -> the architecture's layers ->
 * LM head -> sampler), its capture as a CUDA graph, sampling settings and the generation loop.
 * C re-expression of the reference's host loop (src/launcher.s:685-1092 decode_one_token, :2981-3136 alloc_buffers);
 * what the layers do is the architecture's (lb_model_priv.h lb_arch). */
#include "lb_model_priv.h"
#include <math.h>

extern void lb_prefill_ws_free(lb_model* m);
extern int lb_comm_fill(const lb_comm* m, lb_tp_params* p, int slot, int n);

int lb_dalloc(lb_model* m, CUdeviceptr* p, size_t bytes) {
    uint64_t d = 0;
    LB_TRY(lb_malloc(m->c, bytes < 16 ? 16 : bytes, &d));
    *p = (CUdeviceptr)d;
    return LB_OK;
}
int lb_upload(lb_model* m, CUdeviceptr* p, const void* src, size_t bytes) {
    LB_TRY(lb_dalloc(m, p, bytes));
    LB_CU(m->c, lb_drv.MemcpyHtoDAsync(*p, src, bytes, m->c->stream));
    LB_CU(m->c, lb_drv.StreamSynchronize(m->c->stream)); /* src may be a temporary */
    return LB_OK;
}

int lb_model_alloc_common(lb_model* m) {
    LB_TRY(lb_dalloc(m, &m->X, (size_t)m->cfg.hidden * 4));
    LB_TRY(lb_dalloc(m, &m->logits, (size_t)m->vocab_s * 4));
    LB_TRY(lb_dalloc(m, &m->d_token, 16));
    LB_TRY(lb_dalloc(m, &m->d_pos, 16));
    LB_TRY(lb_dalloc(m, &m->d_next, 16));
    LB_TRY(lb_dalloc(m, &m->d_tokens, (size_t)m->cfg.max_ctx * 4));
    LB_TRY(lb_dalloc(m, &m->cand_val, (size_t)m->arch->head_ctas(m) * 4));
    LB_TRY(lb_dalloc(m, &m->cand_idx, (size_t)m->arch->head_ctas(m) * 4));
    LB_CU(m->c, lb_drv.MemHostAlloc((void**)&m->h_next, 64, 0));
    return LB_OK;
}

LB_API int lb_model_reset_state(lb_model* m) {
    if (!m) return LB_ERR_INVALID;
    LB_CU(m->c, lb_drv.CtxSetCurrent(m->c->cu_ctx));
    LB_TRY(m->arch->reset_state(m));
    LB_CU(m->c, lb_drv.StreamSynchronize(m->c->stream));
    m->host_pos = 0;
    return LB_OK;
}
LB_API int lb_model_checkpoint(lb_model* m) { return m ? m->arch->snapshot(m, 0) : LB_ERR_INVALID; }
LB_API int lb_model_rollback(lb_model* m) { return m ? m->arch->snapshot(m, 1) : LB_ERR_INVALID; }
LB_API int lb_model_state_ptr(lb_model* m, int layer, int which, uint64_t* dptr, size_t* bytes) {
    if (!m || layer < 0 || layer >= m->cfg.n_layers || !dptr || !bytes || which < 0 || which > 1) return LB_ERR_INVALID;
    return m->arch->state_ptr(m, layer, which, dptr, bytes);
}
LB_API const char* lb_model_arch_name(const lb_model* m) { return m ? m->arch->name : ""; }

LB_API int lb_model_logits_ptr(lb_model* m, uint64_t* dptr) {
    if (!m || !dptr) return LB_ERR_INVALID;
    *dptr = m->logits;
    return LB_OK;
}
LB_API uint64_t lb_model_weight_bytes(const lb_model* m) { return m ? m->weight_bytes : 0; }
LB_API const lb_model_cfg* lb_model_config(const lb_model* m) { return m ? &m->cfg : NULL; }
LB_API int lb_model_step_kernels(const lb_model* m) { return m ? m->step_kernels : 0; }

/* the kernel that turns the LM head's output into the next token (and advances the position on the device) */
int lb_model_launch_sampler(lb_model* m) {
    lb_ctx* c = m->c;
    if (m->tp_size == 1 && m->top_k > 0) { /* temperature / top-k sampling over the full logits; the draw is a function of (seed, position) */
        uint64_t zero = 0;
        int n = m->vocab_s;
        void* params[] = {&m->logits, &n, &m->d_next, &m->d_token, &m->d_pos, &m->temperature, &m->top_k, &m->sample_seed, &zero, &zero, &zero};
        LB_TRY(lb_launch(c, LBK_topk_sample_f32, 1, 1, 1, 1024, 0, params, 1));
    } else if (m->tp_size == 1) {
        int n = m->arch->head_ctas(m); /* one (value, row) candidate per LM-head CTA */
        void* params[] = {&m->cand_val, &n, &m->d_next, &m->d_token, &m->d_pos, &m->cand_idx};
        LB_TRY(lb_launch(c, LBK_argmax_f32, 1, 1, 1, 1024, 0, params, 1));
    } else {
        lb_tp_argmax_params q;
        memset(&q, 0, sizeof q);
        LB_TRY(lb_comm_fill(m->comm, &q.tp, 2, 2));
        q.cand_val = (const float*)m->cand_val; q.cand_idx = (const int32_t*)m->cand_idx;
        q.n_cand = m->arch->head_ctas(m); q.vocab_offset = m->tp_rank * m->vocab_s;
        q.out_idx = (int32_t*)m->d_next; q.next_token = (int32_t*)m->d_token; q.pos = (int32_t*)m->d_pos;
        void* params[] = {&q};
        LB_TRY(lb_launch(c, LBK_tp_argmax_exchange, 1, 1, 1, 1024, 0, params, 1));
    }
    return LB_OK;
}

/* n tokens' embeddings with the pair embedding: one token (given, its position in device memory), or the tokens already in m->d_tokens from pos0 on */
int lb_model_embed_bigram(lb_model* m, CUdeviceptr token, CUdeviceptr pos_ptr, int pos0, int n, CUdeviceptr out) {
    const int H = m->cfg.hidden;
    void* params[] = {&m->embed, &m->bigram, &token, &pos_ptr, &pos0, &m->d_tokens, &out, (void*)&H, &m->bigram_buckets, &m->bigram_mul_prev, &m->bigram_mul_cur};
    return lb_launch(m->c, LBK_embed_bigram, (unsigned)((H + 1023) / 1024), (unsigned)n, 1, 256, 0, params, 1);
}

static int issue_step(lb_model* m) {
    lb_ctx* c = m->c;
    const int H = m->cfg.hidden;
    uint64_t launches0 = c->launches;
    if (m->bigram) LB_TRY(lb_model_embed_bigram(m, m->d_token, m->d_pos, 0, 1, m->X));
    else {
        void* params[] = {&m->embed, &m->d_token, &m->X, (void*)&H};
        LB_TRY(lb_launch(c, LBK_embed_bf16, (unsigned)((H + 1023) / 1024), 1, 1, 256, 0, params, 1));
    }
    LB_TRY(m->arch->step_layers(m));
    if (!m->globals_loaded) return lb_fail(c, LB_ERR_STATE, "model: globals have no weights");
    LB_TRY(m->arch->head(m, m->X));
    LB_TRY(lb_model_launch_sampler(m));
    m->step_kernels = (int)(c->launches - launches0);
    return LB_OK;
}

/* top_k == 0 (default): greedy.  Otherwise the step samples among the top_k largest logits at this temperature; the
 * uniform draw of a step is element (position) of a stream of the seeded generator, so a run can be repeated.  Takes
 * effect at the next lb_model_decode / lb_model_capture.  Single GPU only. */
LB_API int lb_model_set_sampling(lb_model* m, float temperature, int top_k, uint64_t seed) {
    if (!m) return LB_ERR_INVALID;
    if (top_k < 0 || top_k > 64 || (top_k > 0 && !(temperature > 0.f))) return lb_fail(m->c, LB_ERR_INVALID, "model: sampling needs 0 <= top_k <= 64 and temperature > 0");
    if (top_k > 0 && m->tp_size != 1) return lb_fail(m->c, LB_ERR_STATE, "model: sampling other than greedy is single-GPU only");
    m->temperature = temperature; m->top_k = top_k; m->sample_seed = seed;
    if (m->graph) { lb_graph_destroy(m->c, m->graph); m->graph = NULL; } /* a captured step samples the old way */
    return LB_OK;
}

LB_API int lb_model_set_chain(lb_model* m, int on) {
    if (!m) return LB_ERR_INVALID;
    m->use_chain = on ? 1 : 0;
    return LB_OK;
}

LB_API int lb_model_set_comm(lb_model* m, lb_comm* comm) {
    if (!m || !comm) return LB_ERR_INVALID;
    if (lb_comm_rank(comm) != m->tp_rank || lb_comm_size(comm) != m->tp_size)
        return lb_fail(m->c, LB_ERR_INVALID, "model: exchange buffers are for rank %d/%d, the model is shard %d/%d",
                       lb_comm_rank(comm), lb_comm_size(comm), m->tp_rank, m->tp_size);
    m->comm = comm;
    for (int slot = 0; slot < 2; slot++) { /* the exchange parameters of both slots, for all-reduce entries of the chain */
        lb_tp_params p;
        LB_TRY(lb_comm_fill(comm, &p, slot, m->cfg.hidden));
        p.x = (float*)m->X;
        if (m->tp_params[slot]) { lb_drv.MemFree(m->tp_params[slot]); m->tp_params[slot] = 0; }
        LB_TRY(lb_upload(m, &m->tp_params[slot], &p, sizeof p));
    }
    return LB_OK;
}

LB_API int lb_model_set_input(lb_model* m, int token, int pos) {
    if (!m) return LB_ERR_INVALID;
    if (token < 0 || token >= m->cfg.vocab || pos < 0 || pos >= m->cfg.max_ctx)
        return lb_fail(m->c, LB_ERR_INVALID, "model: token %d / position %d out of range", token, pos);
    /* by value, in stream order: back-to-back calls cannot overwrite each other's staging */
    LB_CU(m->c, lb_drv.MemsetD32Async(m->d_token, (unsigned)token, 1, m->c->stream));
    LB_CU(m->c, lb_drv.MemsetD32Async(m->d_pos, (unsigned)pos, 1, m->c->stream));
    m->host_pos = pos;
    return LB_OK;
}

LB_API int lb_model_read_next(lb_model* m, int* next_out) {
    if (!m || !next_out) return LB_ERR_INVALID;
    LB_CU(m->c, lb_drv.MemcpyDtoHAsync(&m->h_next[0], m->d_next, 4, m->c->stream));
    LB_CU(m->c, lb_drv.StreamSynchronize(m->c->stream));
    *next_out = m->h_next[0];
    uint32_t st = 0;
    return lb_device_status(m->c, &st);
}

LB_API int lb_model_decode(lb_model* m, int token, int pos, int* next_out) {
    if (!m || !next_out) return LB_ERR_INVALID;
    LB_CU(m->c, lb_drv.CtxSetCurrent(m->c->cu_ctx));
    LB_TRY(lb_model_set_input(m, token, pos));
    LB_TRY(issue_step(m));
    m->host_pos = pos + 1;
    return lb_model_read_next(m, next_out);
}

LB_API int lb_model_capture(lb_model* m) {
    if (!m) return LB_ERR_INVALID;
    if (m->graph) { lb_graph_destroy(m->c, m->graph); m->graph = NULL; }
    LB_CU(m->c, lb_drv.CtxSetCurrent(m->c->cu_ctx));
    LB_TRY(lb_graph_begin_capture(m->c));
    int st = issue_step(m);
    lb_graph* g = NULL;
    int st2 = lb_graph_end_capture(m->c, &g);
    if (st != LB_OK) { if (g) lb_graph_destroy(m->c, g); return st; }
    if (st2 != LB_OK) return st2;
    m->graph = g;
    m->step_kernels = lb_graph_kernel_count(g);
    return LB_OK;
}

LB_API int lb_model_replay(lb_model* m, int n_steps) {
    if (!m || n_steps < 0) return LB_ERR_INVALID;
    if (!m->graph) return lb_fail(m->c, LB_ERR_STATE, "model: replay before capture");
    /* every step appends one KV row at its position and advances the position on the device: refuse what would run past
     * the caches before anything is launched */
    if (m->host_pos + n_steps > m->cfg.max_ctx)
        return lb_fail(m->c, LB_ERR_INVALID, "model: %d steps from position %d run past the context of %d rows", n_steps, m->host_pos,
                       m->cfg.max_ctx);
    for (int i = 0; i < n_steps; i++) {
        LB_TRY(lb_graph_launch(m->c, m->graph));
        m->host_pos++;
    }
    return LB_OK;
}

/* The launcher's decode loop (src/launcher.s:552-652 generation loop, :931-1087 sample and print): run the prompt, then
 * decode until `eos` (248044 for the reference model, models/families/qwen/qwen3.5/27b/config.json:12; negative = none) or
 * max_new tokens.  out receives the generated tokens (the end-of-sequence token included when it was produced). */
LB_API int lb_model_generate(lb_model* m, const int* prompt, int n_prompt, int max_new, int eos, int* out, int* n_out) {
    if (!m || !prompt || n_prompt < 1 || max_new < 0 || !out || !n_out) return LB_ERR_INVALID;
    *n_out = 0;
    if (max_new == 0) return LB_OK;
    int tok = 0;
    LB_TRY(lb_model_prefill(m, prompt, n_prompt, 0, &tok));
    out[(*n_out)++] = tok;
    if (!m->graph) LB_TRY(lb_model_capture(m));
    while (*n_out < max_new && tok != eos) {
        if (m->host_pos >= m->cfg.max_ctx) break; /* the context is full */
        LB_TRY(lb_model_replay(m, 1)); /* token and position are already on the device */
        LB_TRY(lb_model_read_next(m, &tok));
        out[(*n_out)++] = tok;
    }
    return LB_OK;
}

LB_API void lb_model_destroy(lb_model* m) {
    if (!m) return;
    lb_ctx* c = m->c;
    if (lb_drv.loaded && c && c->cu_ctx) {
        lb_drv.CtxSetCurrent(c->cu_ctx);
        lb_drv.StreamSynchronize(c->stream);
        if (m->graph) lb_graph_destroy(c, m->graph);
        if (m->arch) m->arch->destroy(m);
        CUdeviceptr g[] = {m->embed, m->lm_head, m->final_norm, m->X, m->logits, m->d_token, m->d_pos, m->d_next, m->cand_val, m->cand_idx, m->bigram, m->d_tokens};
        for (size_t i = 0; i < sizeof g / sizeof g[0]; i++) if (g[i]) lb_drv.MemFree(g[i]);
        lb_prefill_ws_free(m);
        if (m->h_next) lb_drv.MemFreeHost(m->h_next);
    }
    free(m->L);
    free(m->impl);
    free(m);
}
