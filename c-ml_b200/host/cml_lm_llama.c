/* The "llama" class of the model registry: a GGUF file behind the interface of cml_lm.h, driven through
 * cml_llama.c. Sequences are the model's batch slots with caches of max_tokens each. A step prefills all but
 * the last token of every entry into its slot, then runs the last tokens as one batched decode step. */
#include <stdlib.h>
#include <string.h>

#include "cml_lm_internal.h"

typedef struct LlamaLM {
    CMLLLaMAModel* model;
    int slots, vocab;
    int* len;                    /* per slot: cached tokens, -1 when closed */
} LlamaLM;

static void llama_lm_free(void* p) {
    LlamaLM* m = (LlamaLM*)p;
    if (!m) return;
    cml_llama_free(m->model);
    free(m->len);
    free(m);
}

static void* llama_lm_load(const char* path, const CMLJson* config, const CMLLMOptions* options, CMLLMInfo* info) {
    CMLLLaMAConfig c;
    if (config) { LOG_ERROR("llama models are read from GGUF files"); return NULL; }
    if (options->max_sequences > 32) { LOG_ERROR("llama models serve up to 32 sequences"); return NULL; }
    if (cml_llama_config_from_gguf(path, &c)) return NULL;
    if (options->max_tokens < c.max_seq_len) c.max_seq_len = options->max_tokens;
    LlamaLM* m = (LlamaLM*)calloc(1, sizeof *m);
    if (!m) return NULL;
    m->slots = options->max_sequences;
    m->vocab = c.vocab_size;
    m->len = (int*)malloc((size_t)m->slots * sizeof(int));
    m->model = cml_llama_create(&c);
    const int flags = options->dtype == DTYPE_FLOAT32 ? CML_B200_KV_FP32 | CML_B200_ALL_LOGITS_FP32 : 0;
    if (!m->len || !m->model || cml_llama_set_options(m->model, flags, m->slots) || cml_llama_load_gguf(m->model, path)) { llama_lm_free(m); return NULL; }
    for (int i = 0; i < m->slots; i++) m->len[i] = -1;
    cml_llama_load_gguf_tokenizer(m->model, path);          /* a file without one still generates from ids */
    info->vocab = c.vocab_size;
    info->tokenizer = m->model->tokenizer;
    return m;
}

static int llama_lm_open(void* p) {
    LlamaLM* m = (LlamaLM*)p;
    for (int i = 0; i < m->slots; i++)
        if (m->len[i] < 0) {
            if (cml_llama_truncate(m->model, i, 0)) return -1;
            m->len[i] = 0;
            return i;
        }
    LOG_ERROR("llama: all %d sequences are open", m->slots);
    return -1;
}
static int llama_lm_close(void* p, int seq) { ((LlamaLM*)p)->len[seq] = -1; return 0; }
static int llama_lm_length(void* p, int seq) { return ((LlamaLM*)p)->len[seq]; }

static int llama_lm_step(void* p, const CMLLMEntry* entries, int n, float* logits) {
    LlamaLM* m = (LlamaLM*)p;
    int last[32], rows = 0;
    float* out = logits;
    memset(last, 0, sizeof last);
    for (int i = 0; i < n; i++) {
        const CMLLMEntry* e = &entries[i];
        if (e->num_want > 1 || (e->num_want == 1 && e->want[0] != e->num_tokens - 1)) { LOG_ERROR("llama: logits are given for the last token of an entry only"); return -1; }
        if (m->len[e->seq] + e->num_tokens > m->model->config.max_seq_len) { LOG_ERROR("llama: sequence %d would exceed %d tokens", e->seq, m->model->config.max_seq_len); return -1; }
    }
    for (int i = 0; i < n; i++) {
        const CMLLMEntry* e = &entries[i];
        if (e->num_tokens > 1 && cml_llama_prefill_sequence(m->model, e->seq, e->tokens, e->num_tokens - 1)) return -1;
        m->len[e->seq] += e->num_tokens - 1;
        last[e->seq] = e->tokens[e->num_tokens - 1];
        if (e->seq + 1 > rows) rows = e->seq + 1;
    }
    /* slots that take no part get a dummy row, rolled back below: closed ones at position 0, open ones where
     * they stand (a slot at the end of its cache steps back for the moment) */
    for (int s = 0; s < rows; s++)
        if (m->len[s] < 0 && cml_llama_truncate(m->model, s, 0)) return -1;
    Tensor* lg = cml_llama_forward_batch(m->model, last, rows);
    if (!lg) return -1;
    for (int i = 0; i < n; i++) m->len[entries[i].seq]++;
    int rc = 0;
    for (int s = 0; s < rows; s++)
        if (cml_llama_truncate(m->model, s, m->len[s] < 0 ? 0 : m->len[s])) rc = -1;
    for (int i = 0; i < n; i++)
        if (entries[i].num_want) {
            memcpy(out, (const float*)lg->data + (size_t)entries[i].seq * (size_t)m->vocab, (size_t)m->vocab * sizeof(float));
            out += m->vocab;
        }
    tensor_free(lg);
    return rc;
}

static const CMLLMClass kLlamaClass = {.architecture = "llama", .load = llama_lm_load, .free = llama_lm_free, .open = llama_lm_open,
                                       .close = llama_lm_close, .length = llama_lm_length, .step = llama_lm_step};

__attribute__((constructor)) static void register_llama(void) { cml_lm_register(&kLlamaClass); }
