/* Continuous-batching scheduler (include/nn/serving.h, src/nn/serving.c in the C-ML tree): a
 * circular queue of submitted requests, an active batch of at most max_batch_size of them, status
 * and timing bookkeeping. As in C-ML this layer does not run the model: cml_serving_step admits
 * queued requests and moves them PREFILL -> DECODING, and whoever runs the model appends tokens
 * and calls cml_serving_finish_request.
 * cml_serving_run_lm (cml_lm.c) is such a runner for every model of the registry, cml_serving_run_llama
 * (cml_serving_llama.c) for a LLaMA. */
#include <stdlib.h>
#include <string.h>
#include <time.h>

#include "cml_internal.h"

static double wall_ms(void) {
    struct timespec ts;
    clock_gettime(CLOCK_MONOTONIC, &ts);
    return 1e3 * (double)ts.tv_sec + 1e-6 * (double)ts.tv_nsec;
}

static void request_free(CMLSequenceRequest* r) {
    if (!r) return;
    free(r->prompt_tokens);
    free(r->generated_tokens);
    free(r);
}

/* queued requests first (oldest first), then the active batch */
static CMLSequenceRequest* lookup(CMLServingContext* ctx, int request_id) {
    if (!ctx) return NULL;
    for (int i = 0; i < ctx->queue_count; i++) {
        CMLSequenceRequest* r = ctx->queue[(ctx->queue_head + i) % ctx->queue_capacity];
        if (r && r->request_id == request_id) return r;
    }
    for (int i = 0; i < ctx->batch_size; i++)
        if (ctx->active_batch[i] && ctx->active_batch[i]->request_id == request_id) return ctx->active_batch[i];
    return NULL;
}

CMLServingConfig cml_serving_default_config(void) {
    CMLServingConfig c = {.max_batch_size = 8, .max_queue_size = 256, .max_seq_len = 2048, .max_new_tokens_default = 256,
                          .temperature_default = 0.8f, .top_p_default = 0.9f};
    return c;
}

CMLServingContext* cml_serving_create(const CMLServingConfig* config) {
    if (!config) { LOG_ERROR("cml_serving_create: NULL config"); return NULL; }
    CMLServingContext* ctx = (CMLServingContext*)calloc(1, sizeof *ctx);
    if (!ctx) { LOG_ERROR("cml_serving_create: allocation failed"); return NULL; }
    ctx->config = *config;
    if (ctx->config.max_batch_size <= 0) ctx->config.max_batch_size = 8;
    if (ctx->config.max_batch_size > CML_SERVING_MAX_BATCH) ctx->config.max_batch_size = CML_SERVING_MAX_BATCH;
    if (ctx->config.max_queue_size <= 0) ctx->config.max_queue_size = 256;
    if (ctx->config.max_queue_size > CML_SERVING_MAX_QUEUE) ctx->config.max_queue_size = CML_SERVING_MAX_QUEUE;
    ctx->queue_capacity = ctx->config.max_queue_size;
    ctx->queue = (CMLSequenceRequest**)calloc((size_t)ctx->queue_capacity, sizeof *ctx->queue);
    ctx->active_batch = (CMLSequenceRequest**)calloc((size_t)ctx->config.max_batch_size, sizeof *ctx->active_batch);
    if (!ctx->queue || !ctx->active_batch) {
        LOG_ERROR("cml_serving_create: queue allocation failed");
        free(ctx->queue); free(ctx->active_batch); free(ctx);
        return NULL;
    }
    ctx->next_request_id = 1;
    LOG_INFO("Serving context created: max_batch=%d, max_queue=%d", ctx->config.max_batch_size, ctx->config.max_queue_size);
    return ctx;
}

void cml_serving_free(CMLServingContext* ctx) {
    if (!ctx) return;
    for (int i = 0; i < ctx->queue_count; i++) request_free(ctx->queue[(ctx->queue_head + i) % ctx->queue_capacity]);
    for (int i = 0; i < ctx->batch_size; i++) request_free(ctx->active_batch[i]);
    LOG_INFO("Serving context freed (total_requests=%zu, completed=%zu)", ctx->stats.total_requests, ctx->stats.completed_requests);
    free(ctx->queue);
    free(ctx->active_batch);
    free(ctx);
}

void cml_serving_set_kv_cache(CMLServingContext* ctx, CMLPagedKVCache* cache) {
    if (!ctx) return;
    ctx->kv_cache = cache;
    LOG_INFO("Paged KV cache set on serving context");
}

int cml_serving_submit(CMLServingContext* ctx, const int* prompt_tokens, int num_tokens, int max_new_tokens) {
    if (!ctx) { LOG_ERROR("cml_serving_submit: NULL context"); return -1; }
    if (!prompt_tokens || num_tokens <= 0) { LOG_ERROR("cml_serving_submit: invalid prompt (tokens=%p, n=%d)", (const void*)prompt_tokens, num_tokens); return -1; }
    if (ctx->queue_count >= ctx->queue_capacity) { LOG_WARNING("cml_serving_submit: queue full (%d/%d)", ctx->queue_count, ctx->queue_capacity); return -1; }
    CMLSequenceRequest* r = (CMLSequenceRequest*)calloc(1, sizeof *r);
    if (!r) { LOG_ERROR("cml_serving_submit: request allocation failed"); return -1; }
    r->max_new_tokens = max_new_tokens > 0 ? max_new_tokens : ctx->config.max_new_tokens_default;
    r->gen_capacity = r->max_new_tokens;
    r->prompt_tokens = (int*)malloc((size_t)num_tokens * sizeof(int));
    r->generated_tokens = (int*)calloc((size_t)(r->gen_capacity > 0 ? r->gen_capacity : 1), sizeof(int));
    if (!r->prompt_tokens || !r->generated_tokens) {
        LOG_ERROR("cml_serving_submit: token buffer allocation failed");
        request_free(r);
        return -1;
    }
    memcpy(r->prompt_tokens, prompt_tokens, (size_t)num_tokens * sizeof(int));
    r->num_prompt_tokens = num_tokens;
    r->request_id = ctx->next_request_id++;
    r->temperature = ctx->config.temperature_default;
    r->top_p = ctx->config.top_p_default;
    r->status = CML_SEQ_STATUS_QUEUED;
    r->paged_seq_id = -1;
    r->submit_time_ms = wall_ms();
    ctx->queue[ctx->queue_tail] = r;
    ctx->queue_tail = (ctx->queue_tail + 1) % ctx->queue_capacity;
    ctx->queue_count++;
    ctx->stats.total_requests++;
    return r->request_id;
}

int cml_serving_step(CMLServingContext* ctx) {
    if (!ctx) return 0;
    while (ctx->queue_count > 0 && ctx->batch_size < ctx->config.max_batch_size) {     /* oldest request first */
        CMLSequenceRequest* r = ctx->queue[ctx->queue_head];
        ctx->queue[ctx->queue_head] = NULL;
        ctx->queue_head = (ctx->queue_head + 1) % ctx->queue_capacity;
        ctx->queue_count--;
        r->status = CML_SEQ_STATUS_PREFILL;
        ctx->active_batch[ctx->batch_size++] = r;
        ctx->stats.active_sequences++;
    }
    /* the prefill compute is the runner's business: an admitted request counts as decoding */
    for (int i = 0; i < ctx->batch_size; i++) {
        CMLSequenceRequest* r = ctx->active_batch[i];
        if (r && r->status == CML_SEQ_STATUS_PREFILL) {
            r->status = CML_SEQ_STATUS_DECODING;
            r->first_token_time_ms = wall_ms();
        }
    }
    return ctx->batch_size;
}

CMLSequenceStatus cml_serving_get_status(CMLServingContext* ctx, int request_id) {
    const CMLSequenceRequest* r = lookup(ctx, request_id);
    return r ? r->status : CML_SEQ_STATUS_ERROR;
}

const int* cml_serving_get_tokens(CMLServingContext* ctx, int request_id, int* out_count) {
    if (out_count) *out_count = 0;
    const CMLSequenceRequest* r = lookup(ctx, request_id);
    if (!r) return NULL;
    if (out_count) *out_count = r->num_generated;
    return r->generated_tokens;
}

int cml_serving_finish_request(CMLServingContext* ctx, int request_id) {
    if (!ctx) return -1;
    int at = -1;
    for (int i = 0; i < ctx->batch_size && at < 0; i++)
        if (ctx->active_batch[i] && ctx->active_batch[i]->request_id == request_id) at = i;
    if (at < 0) { LOG_WARNING("cml_serving_finish_request: request %d not in active batch", request_id); return -1; }
    CMLSequenceRequest* r = ctx->active_batch[at];
    r->status = CML_SEQ_STATUS_FINISHED;
    r->finish_time_ms = wall_ms();
    CMLServingStats* s = &ctx->stats;
    s->completed_requests++;
    s->total_tokens_generated += (size_t)r->num_generated;
    if (s->active_sequences > 0) s->active_sequences--;
    s->total_time_ms += r->finish_time_ms - r->submit_time_ms;
    if (r->first_token_time_ms > 0.0) {                       /* running mean over the completed requests */
        const double n = (double)s->completed_requests;
        s->avg_time_to_first_token_ms = (s->avg_time_to_first_token_ms * (n - 1.0) + (r->first_token_time_ms - r->submit_time_ms)) / n;
    }
    if (s->total_time_ms > 0.0) s->avg_tokens_per_second = (double)s->total_tokens_generated / (s->total_time_ms / 1000.0);
    request_free(r);
    ctx->active_batch[at] = ctx->active_batch[ctx->batch_size - 1];     /* the last active request takes the hole */
    ctx->active_batch[--ctx->batch_size] = NULL;
    return 0;
}

CMLServingStats cml_serving_get_stats(const CMLServingContext* ctx) {
    CMLServingStats none;
    memset(&none, 0, sizeof none);
    return ctx ? ctx->stats : none;
}
