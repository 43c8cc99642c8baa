/* cml_serving_run_llama (no C-ML counterpart) runs the scheduler of cml_serving.c over a device-resident
 * LLaMA: every active request owns one of the model's batch slots, a newly admitted request is
 * prefilled into its slot (cml_llama_truncate + cml_llama_prefill_sequence), and all slots take one
 * greedy decode step per iteration through the batched forward, so requests of different lengths start
 * and finish independently while the weights are streamed once per step for all of them. */
#include <stdlib.h>
#include <string.h>

#include "cml_internal.h"

/* ---- a runner over a device-resident LLaMA ---------------------------------------------------------
 * Runs until the queue and the batch are empty, or for max_steps batched decode steps (0: no
 * limit). A request's slot is kept in paged_seq_id. on_finish, when given, sees every request
 * (its generated_tokens are complete) just before cml_serving_finish_request frees it. eos_token
 * < 0: requests only end at max_new_tokens or when the model's max_seq_len is reached. Returns the
 * number of decode steps taken, -1 on error. The model must have been given
 * cml_llama_set_options(model, flags, max_batch >= the context's max_batch_size) before loading. */
int cml_serving_run_llama(CMLServingContext* ctx, CMLLLaMAModel* model, int eos_token, int max_steps,
                          void (*on_finish)(const CMLSequenceRequest* request, void* user), void* user) {
    if (!ctx || !model) { LOG_ERROR("cml_serving_run_llama: NULL argument"); return -1; }
    const int B = ctx->config.max_batch_size, vocab = model->config.vocab_size, max_len = model->config.max_seq_len;
    int* slot_req = (int*)malloc((size_t)B * sizeof(int));            /* request id per model slot, 0 = free */
    int* step_tok = (int*)calloc((size_t)B, sizeof(int));
    int steps = 0, rc = 0;
    if (!slot_req || !step_tok) { free(slot_req); free(step_tok); return -1; }
    memset(slot_req, 0, (size_t)B * sizeof(int));
    for (int i = 0; i < ctx->batch_size; i++)                          /* requests admitted by an earlier call keep their slots */
        if (ctx->active_batch[i] && ctx->active_batch[i]->paged_seq_id >= 0 && ctx->active_batch[i]->paged_seq_id < B)
            slot_req[ctx->active_batch[i]->paged_seq_id] = ctx->active_batch[i]->request_id;
    CMLGenerationConfig greedy = cml_generation_default_config();
    greedy.do_sample = false;
    while (rc == 0 && (ctx->queue_count > 0 || ctx->batch_size > 0) && (max_steps <= 0 || steps < max_steps)) {
        cml_serving_step(ctx);
        /* prefill whoever has no slot yet; its first token comes from the prompt's last row */
        for (int i = 0; i < ctx->batch_size && rc == 0; i++) {
            CMLSequenceRequest* r = ctx->active_batch[i];
            if (r->paged_seq_id >= 0) continue;
            int s = 0;
            while (s < B && slot_req[s]) s++;
            if (s == B) { LOG_ERROR("cml_serving_run_llama: no free model slot"); rc = -1; break; }
            if (r->num_prompt_tokens + 1 > max_len) { r->status = CML_SEQ_STATUS_ERROR; r->paged_seq_id = s; slot_req[s] = r->request_id; continue; }
            slot_req[s] = r->request_id;
            r->paged_seq_id = s;
            if (cml_llama_truncate(model, s, 0) ||
                (r->num_prompt_tokens > 1 && cml_llama_prefill_sequence(model, s, r->prompt_tokens, r->num_prompt_tokens - 1))) { rc = -1; break; }
            r->current_pos = r->num_prompt_tokens - 1;
        }
        if (rc) break;
        /* one batched step: slot s feeds its pending token (the prompt's last one right after the prefill) */
        int live = 0;
        for (int s = 0; s < B; s++) step_tok[s] = 0;
        for (int i = 0; i < ctx->batch_size; i++) {
            CMLSequenceRequest* r = ctx->active_batch[i];
            if (r->status != CML_SEQ_STATUS_DECODING) continue;
            step_tok[r->paged_seq_id] = r->num_generated ? r->generated_tokens[r->num_generated - 1] : r->prompt_tokens[r->num_prompt_tokens - 1];
            live++;
        }
        if (live) {
            for (int s = 0; s < B; s++)                                 /* idle slots take a dummy row at position 0 */
                if (!slot_req[s] && cml_llama_truncate(model, s, 0)) rc = -1;
            Tensor* lg = rc ? NULL : cml_llama_forward_batch(model, step_tok, B);
            if (!lg) { rc = -1; break; }
            steps++;
            for (int i = 0; i < ctx->batch_size; i++) {
                CMLSequenceRequest* r = ctx->active_batch[i];
                if (r->status != CML_SEQ_STATUS_DECODING) continue;
                int row_shape[2] = {1, vocab};
                TensorConfig tc = {.dtype = DTYPE_FLOAT32, .device = DEVICE_CPU, .has_dtype = true, .has_device = true};
                Tensor* row = tensor_from_data((float*)lg->data + (size_t)r->paged_seq_id * vocab, row_shape, 2, &tc);
                const int tok = row ? cml_llama_sample_token(row, &greedy) : -1;
                tensor_free(row);
                if (tok < 0) { rc = -1; break; }
                if (r->num_generated < r->gen_capacity) r->generated_tokens[r->num_generated++] = tok;
                r->current_pos++;
            }
            tensor_free(lg);
        }
        /* retire what is done (finish_request moves the last active request into the hole) */
        for (int i = 0; i < ctx->batch_size && rc == 0;) {
            CMLSequenceRequest* r = ctx->active_batch[i];
            const int last = r->num_generated ? r->generated_tokens[r->num_generated - 1] : -1;
            const int done = r->status == CML_SEQ_STATUS_ERROR || r->num_generated >= r->max_new_tokens ||
                             (eos_token >= 0 && last == eos_token) || r->current_pos + 1 >= max_len;
            if (!done) { i++; continue; }
            if (on_finish) on_finish(r, user);
            slot_req[r->paged_seq_id] = 0;
            cml_serving_finish_request(ctx, r->request_id);
        }
    }
    free(slot_req);
    free(step_tok);
    return rc ? -1 : steps;
}
