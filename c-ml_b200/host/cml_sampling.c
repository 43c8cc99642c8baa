/* Token sampling from a row of logits and the generation defaults, shared by every model
 * (C-ML: src/nn/llama.c). */
#include <math.h>
#include <stdlib.h>

#include "cml_internal.h"

CMLGenerationConfig cml_generation_default_config(void) {
    CMLGenerationConfig c = {.temperature = 0.8f, .top_p = 0.9f, .top_k = 40, .max_new_tokens = 256, .eos_token_id = 2, .do_sample = true};
    return c;
}

void cml_generation_result_free(CMLGenerationResult* result) {
    if (!result) return;
    free(result->token_ids);
    free(result->text);
    free(result);
}

/* ---- sampling (src/nn/llama.c:614-737) ----------------------------------------------------------- */
typedef struct { float value; int index; } LogitEntry;
static int entry_cmp_desc(const void* a, const void* b) {
    const float va = ((const LogitEntry*)a)->value, vb = ((const LogitEntry*)b)->value;
    return va > vb ? -1 : (va < vb ? 1 : 0);
}

int cml_llama_sample_token(Tensor* logits, const CMLGenerationConfig* config) {
    if (!logits || !config || !logits->data) return -1;
    const float* data = (const float*)logits->data;
    int vocab;
    const float* row;
    if (logits->ndim == 2) { vocab = logits->shape[1]; row = data + (size_t)(logits->shape[0] - 1) * vocab; }
    else if (logits->ndim == 1) { vocab = logits->shape[0]; row = data; }
    else { LOG_ERROR("cml_llama_sample_token: unexpected logits ndim=%d", logits->ndim); return -1; }
    if (!config->do_sample || config->temperature <= 0.0f) {        /* greedy: first strict maximum */
        int best = 0;
        for (int i = 1; i < vocab; i++) if (row[i] > row[best]) best = i;
        return best;
    }
    LogitEntry* e = (LogitEntry*)malloc((size_t)vocab * sizeof *e);
    if (!e) return -1;
    const float inv_t = 1.0f / config->temperature;
    for (int i = 0; i < vocab; i++) { e[i].value = row[i] * inv_t; e[i].index = i; }
    qsort(e, (size_t)vocab, sizeof *e, entry_cmp_desc);
    int k = config->top_k;
    if (k <= 0 || k > vocab) k = vocab;
    const float mx = e[0].value;
    float sum = 0.f;
    for (int i = 0; i < k; i++) { e[i].value = expf(e[i].value - mx); sum += e[i].value; }
    for (int i = 0; i < k; i++) e[i].value /= sum;
    int cutoff = k;
    if (config->top_p > 0.0f && config->top_p < 1.0f) {
        float cum = 0.f;
        for (int i = 0; i < k; i++) { cum += e[i].value; if (cum >= config->top_p) { cutoff = i + 1; break; } }
    }
    if (cutoff < k) {
        float rs = 0.f;
        for (int i = 0; i < cutoff; i++) rs += e[i].value;
        if (rs > 0.f) for (int i = 0; i < cutoff; i++) e[i].value /= rs;
    }
    const float r = (float)rand() / (float)RAND_MAX;
    float acc = 0.f;
    int id = e[0].index;
    for (int i = 0; i < cutoff; i++) { acc += e[i].value; if (r <= acc) { id = e[i].index; break; } }
    free(e);
    return id;
}
