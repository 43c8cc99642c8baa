/*
 * cml_lm.h -- language models behind one interface: a registry keyed by the architecture a model's own
 * files name, loading, sequences over a paged cache, a step function that runs any mix of prompt portions
 * and decoded tokens as one batch, generation, and the runner of the continuous-batching scheduler
 * (cml_quant_api.h). No C-ML counterpart: C-ML's forward is one LLaMA, one sequence.
 *
 * A model is either a folder with config.json ("architecture" names the class) and model.safetensors, or
 * a GGUF file (class "llama"). Built-in classes: "Rarolorn", "Situlorn", "Lenedra" and
 * "Zevilorn" (folders), "llama" (GGUF).
 *
 * Errors as in cml_quant_api.h: NULL or -1, with a line through cml_log_message.
 */
#ifndef CML_LM_H
#define CML_LM_H

#include "cml_quant_api.h"

#ifdef __cplusplus
extern "C" {
#endif

typedef struct CMLLanguageModel CMLLanguageModel;

typedef struct CMLLMOptions {
    DType dtype;                /* DTYPE_BFLOAT16: the serving form. DTYPE_FLOAT32: everything in 32-bit */
    int max_tokens;             /* tokens the cache pool holds, all sequences together */
    int max_sequences;          /* sequences open at a time */
    int max_step_rows;          /* tokens of one step; 0: max_tokens */
} CMLLMOptions;

/* One sequence's part of a step: its next tokens, and the places among them (ascending) whose logits are
 * asked for. */
typedef struct CMLLMEntry {
    int seq;
    const int* tokens;
    int num_tokens;
    const int* want;
    int num_want;
} CMLLMEntry;

CMLLMOptions cml_lm_default_options(void);      /* bfloat16, 8192 tokens, 8 sequences */
int cml_lm_known(const char* architecture);     /* 1: a class of that name is registered */
CMLLanguageModel* cml_lm_load(const char* path, const CMLLMOptions* options);
void cml_lm_free(CMLLanguageModel* lm);
const char* cml_lm_architecture(const CMLLanguageModel* lm);
int cml_lm_vocab_size(const CMLLanguageModel* lm);
CMLTokenizer* cml_lm_tokenizer(const CMLLanguageModel* lm);      /* owned by the model; NULL when it has none */

/* A sequence takes a slot now and cache blocks as it grows; closing it gives both back. */
int cml_lm_sequence_open(CMLLanguageModel* lm);                  /* id, -1: no free slot */
int cml_lm_sequence_close(CMLLanguageModel* lm, int seq);
int cml_lm_sequence_length(CMLLanguageModel* lm, int seq);
/* Blocks of the pool (cml_lm_block_size tokens each): all of them, and those not in use. */
int cml_lm_block_size(const CMLLanguageModel* lm);
int cml_lm_blocks_total(const CMLLanguageModel* lm);
int cml_lm_blocks_free(const CMLLanguageModel* lm);

/* Runs all entries as one batch. logits: host fp32 [sum of num_want][vocab], in the order of the entries
 * and of `want`; may be NULL when nothing is wanted. Nothing changes when the arguments are refused (unknown
 * token, a sequence twice, pool or step too small). The "llama" class gives logits of an entry's last token only. */
int cml_lm_step(CMLLanguageModel* lm, const CMLLMEntry* entries, int num_entries, float* logits);
/* The same, but picks the arg-max of every wanted row on the device: picked[sum of num_want]. */
int cml_lm_step_greedy(CMLLanguageModel* lm, const CMLLMEntry* entries, int num_entries, int* picked);
/* Greedy decoding that stays on the device: `steps` steps of all sequences, each step's picks the next
 * one's tokens, out_tokens [steps][num_seqs]; *elapsed_ms (optional) is the time of the loop on the device. */
int cml_lm_decode_greedy(CMLLanguageModel* lm, const int* seqs, const int* first_tokens, int num_seqs, int steps, int* out_tokens,
                         float* elapsed_ms);

/* Generates from a prompt through the scheduler: the result holds prompt + generated ids (and the decoded
 * text when the model has a tokenizer). config NULL: greedy, 256 tokens, no end token. */
CMLGenerationResult* cml_lm_generate(CMLLanguageModel* lm, const int* prompt, int num_tokens, const CMLGenerationConfig* config);
/* Runs the scheduler over a model until queue and batch are empty or max_steps (> 0) steps were taken: every
 * step is one batch of prompt portions and decoded tokens. A request waits while the pool could not hold it
 * to its end. config gives sampling (NULL: greedy) and the end token; lengths come from the requests.
 * on_finish (optional) sees each request before it is freed. Returns the number of steps, -1 on error. */
int cml_serving_run_lm(CMLServingContext* ctx, CMLLanguageModel* lm, const CMLGenerationConfig* config, int max_steps,
                       void (*on_finish)(const CMLSequenceRequest* request, void* user), void* user);

#ifdef __cplusplus
}
#endif
#endif /* CML_LM_H */
