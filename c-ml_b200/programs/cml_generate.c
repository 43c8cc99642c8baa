/* cml_generate -- generation from the command line, for every model of the registry.
 *
 *   cml_generate --model DIR|FILE.gguf [--dtype bfloat16|float32] [--max-tokens N] [--max-new N]
 *                [--temperature T --top-k K --top-p P --seed S] [--eos ID]
 *                (--tokens 1,2,3 | --prompt TEXT) ...
 *
 * Every --tokens / --prompt is one request; all of them go through the continuous-batching scheduler
 * together. --prompt needs a model with a tokenizer. Without --temperature decoding is greedy. Output: one
 * line a request, in the order given: the generated ids, and the text where there is a tokenizer. */
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include "cml_lm.h"

#define MAX_REQUESTS 64

typedef struct { int id; int* tokens; int n; } Done;
static Done g_done[MAX_REQUESTS];
static int g_num_done = 0;

static int fail(const char* what, const char* detail) {
    fprintf(stderr, "cml_generate: %s%s%s\n", what, detail ? ": " : "", detail ? detail : "");
    return 2;
}

static void on_finish(const CMLSequenceRequest* r, void* user) {
    (void)user;
    Done* d = &g_done[g_num_done++];
    d->id = r->request_id;
    d->n = r->status == CML_SEQ_STATUS_ERROR ? -1 : r->num_generated;
    d->tokens = (int*)malloc((size_t)(r->num_generated + 1) * sizeof(int));
    if (d->tokens) memcpy(d->tokens, r->generated_tokens, (size_t)r->num_generated * sizeof(int));
}

static int* parse_ids(const char* s, int* n) {
    int* ids = (int*)malloc((strlen(s) / 2 + 2) * sizeof(int));
    *n = 0;
    while (ids && *s) {
        char* end;
        const long v = strtol(s, &end, 10);
        if (end == s || (*end && *end != ',')) { free(ids); return NULL; }
        ids[(*n)++] = (int)v;
        s = *end ? end + 1 : end;
    }
    return ids;
}

int main(int argc, char** argv) {
    const char *model = NULL, *dtype = "bfloat16", *what[MAX_REQUESTS];
    int is_text[MAX_REQUESTS], ids[MAX_REQUESTS], requests = 0, max_new = 64;
    CMLLMOptions o = cml_lm_default_options();
    CMLGenerationConfig c = cml_generation_default_config();
    c.do_sample = false;
    c.eos_token_id = -1;
    for (int i = 1; i < argc; i++) {
        const char *k = argv[i], *v = i + 1 < argc ? argv[++i] : NULL;
        if (!v) return fail("an option without a value", k);
        if (!strcmp(k, "--model")) model = v;
        else if (!strcmp(k, "--dtype")) dtype = v;
        else if (!strcmp(k, "--max-tokens")) o.max_tokens = atoi(v);
        else if (!strcmp(k, "--max-new")) max_new = atoi(v);
        else if (!strcmp(k, "--temperature")) { c.temperature = (float)atof(v); c.do_sample = true; }
        else if (!strcmp(k, "--top-k")) c.top_k = atoi(v);
        else if (!strcmp(k, "--top-p")) c.top_p = (float)atof(v);
        else if (!strcmp(k, "--seed")) srand((unsigned)atoi(v));
        else if (!strcmp(k, "--eos")) c.eos_token_id = atoi(v);
        else if (!strcmp(k, "--tokens") || !strcmp(k, "--prompt")) {
            if (requests == MAX_REQUESTS) return fail("too many requests", NULL);
            is_text[requests] = k[2] == 'p';
            what[requests++] = v;
        } else return fail("unknown option", k);
    }
    if (!model || !requests || (strcmp(dtype, "bfloat16") && strcmp(dtype, "float32")))
        return fail("usage: cml_generate --model DIR|FILE.gguf [--dtype bfloat16|float32] [--max-tokens N] [--max-new N] [--temperature T] [--top-k K] "
                    "[--top-p P] [--seed S] [--eos ID] (--tokens 1,2,3 | --prompt TEXT) ...", NULL);
    o.dtype = !strcmp(dtype, "float32") ? DTYPE_FLOAT32 : DTYPE_BFLOAT16;
    o.max_sequences = requests < 8 ? requests : 8;
    CMLLanguageModel* lm = cml_lm_load(model, &o);
    if (!lm) return fail("cannot load", model);
    CMLServingConfig sc = cml_serving_default_config();
    sc.max_batch_size = o.max_sequences;
    CMLServingContext* ctx = cml_serving_create(&sc);
    if (!ctx) return fail("out of memory", NULL);
    for (int i = 0; i < requests; i++) {
        int n = 0;
        if (is_text[i] && !cml_lm_tokenizer(lm)) return fail("the model has no tokenizer; give --tokens", NULL);
        int* t = is_text[i] ? cml_tokenizer_encode(cml_lm_tokenizer(lm), what[i], &n) : parse_ids(what[i], &n);
        if (!t || n <= 0) return fail("not a prompt", what[i]);
        ids[i] = cml_serving_submit(ctx, t, n, max_new);
        free(t);
        if (ids[i] < 0) return fail("the request was refused", what[i]);
    }
    int rc = cml_serving_run_lm(ctx, lm, &c, 0, on_finish, NULL) < 0 ? fail("generation failed", NULL) : 0;
    for (int i = 0; i < requests && !rc; i++)
        for (int k = 0; k < g_num_done; k++) {
            if (g_done[k].id != ids[i]) continue;
            if (g_done[k].n < 0) { rc = fail("the request cannot be run", what[i]); break; }
            for (int t = 0; t < g_done[k].n; t++) printf("%s%d", t ? " " : "", g_done[k].tokens[t]);
            if (cml_lm_tokenizer(lm)) {
                char* text = cml_tokenizer_decode(cml_lm_tokenizer(lm), g_done[k].tokens, g_done[k].n);
                printf("\t%s", text ? text : "");
                free(text);
            }
            printf("\n");
        }
    for (int k = 0; k < g_num_done; k++) free(g_done[k].tokens);
    cml_serving_free(ctx);
    cml_lm_free(lm);
    return rc;
}
