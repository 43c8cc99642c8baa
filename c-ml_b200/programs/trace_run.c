/* trace_run -- replays a trace: given token ids go through a model step by step, logits come back.
 *
 *   trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--max-sequences N]
 *
 * Standard input holds one JSON object a line:
 *   {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
 * The entries of a line run as one batch; a request is admitted at its first entry and gives its slot and
 * cache blocks back when it is named in "end". Where something is wanted the logits go to OUT/<step>.f32
 * (little-endian fp32, [wanted][vocab], in the order of the entries and of "want"); "done <step>" follows on
 * standard output. The cache pool is made for N tokens. Exit code 0 at the end of the input, 2 on an error. */
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include "cml_json.h"
#include "cml_lm.h"

typedef struct { char id[64]; int seq; } Request;

static int fail(const char* what, const char* detail) {
    fprintf(stderr, "trace_run: %s%s%s\n", what, detail ? ": " : "", detail ? detail : "");
    return 2;
}

static int int_list(const CMLJson* a, int** out, int* n) {
    *out = NULL;
    *n = 0;
    if (!a) return 0;
    if (a->type != CML_JSON_ARRAY) return -1;
    *out = (int*)malloc((size_t)(a->count + 1) * sizeof(int));
    if (!*out) return -1;
    for (const CMLJson* c = a->child; c; c = c->next) {
        if (c->type != CML_JSON_NUMBER || c->number != (double)(int)c->number) return -1;
        (*out)[(*n)++] = (int)c->number;
    }
    return 0;
}

static int write_logits(const char* dir, int step, const float* v, size_t n) {
    char path[4096];
    snprintf(path, sizeof path, "%s/%d.f32", dir, step);
    FILE* f = fopen(path, "wb");
    if (!f) return -1;
    const int ok = fwrite(v, sizeof(float), n, f) == n;
    return fclose(f) == 0 && ok ? 0 : -1;
}

static Request* request_of(Request* r, int n, const char* id) {
    for (int i = 0; i < n; i++)
        if (r[i].seq >= 0 && !strcmp(r[i].id, id)) return &r[i];
    return NULL;
}

static int run_line(CMLLanguageModel* lm, const char* out_dir, Request* req, int slots, const CMLJson* line) {
    const CMLJson *entries = cml_json_get(line, "entries"), *end = cml_json_get(line, "end");
    int step;
    if (cml_json_int(line, "step", &step) || !entries || entries->type != CML_JSON_ARRAY) return fail("a line without step or entries", NULL);
    const int n = entries->count;
    CMLLMEntry* e = (CMLLMEntry*)calloc((size_t)n + 1, sizeof *e);
    int **tokens = (int**)calloc((size_t)n + 1, sizeof *tokens), **want = (int**)calloc((size_t)n + 1, sizeof *want), i = 0, wanted = 0, rc = 0;
    float* logits = NULL;
    if (!e || !tokens || !want) rc = fail("out of memory", NULL);
    for (const CMLJson* c = entries->child; c && !rc; c = c->next, i++) {
        const char* id = cml_json_string(c, "id");
        if (!id || strlen(id) >= sizeof req->id || int_list(cml_json_get(c, "tokens"), &tokens[i], &e[i].num_tokens) ||
            int_list(cml_json_get(c, "want"), &want[i], &e[i].num_want)) { rc = fail("a malformed entry", id); break; }
        Request* r = request_of(req, slots, id);
        if (!r) {
            for (int k = 0; k < slots && !r; k++) if (req[k].seq < 0) r = &req[k];
            if (!r || (r->seq = cml_lm_sequence_open(lm)) < 0) { rc = fail("no free slot for request", id); break; }
            strcpy(r->id, id);
        }
        e[i].seq = r->seq;
        e[i].tokens = tokens[i];
        e[i].want = want[i];
        wanted += e[i].num_want;
    }
    const size_t values = (size_t)wanted * (size_t)cml_lm_vocab_size(lm);
    if (!rc && !(logits = (float*)malloc((values + 1) * sizeof(float)))) rc = fail("out of memory", NULL);
    if (!rc && n && cml_lm_step(lm, e, n, logits)) rc = fail("the step failed", NULL);
    if (!rc && wanted && write_logits(out_dir, step, logits, values)) rc = fail("cannot write logits to", out_dir);
    for (const CMLJson* c = end && end->type == CML_JSON_ARRAY ? end->child : NULL; c && !rc; c = c->next) {
        Request* r = c->string ? request_of(req, slots, c->string) : NULL;
        if (!r || cml_lm_sequence_close(lm, r->seq)) { rc = fail("an unknown request ends", c->string); break; }
        r->seq = -1;
    }
    if (!rc) {
        printf("done %d\n", step);
        fflush(stdout);
    }
    for (int k = 0; k < n; k++) { if (tokens) free(tokens[k]); if (want) free(want[k]); }
    free(tokens); free(want); free(e); free(logits);
    return rc;
}

int main(int argc, char** argv) {
    const char *model = NULL, *dtype = "bfloat16", *out = NULL;
    CMLLMOptions o = cml_lm_default_options();
    o.max_sequences = 4;
    for (int i = 1; i < argc; i++) {
        const char* v = i + 1 < argc ? argv[i + 1] : NULL;
        if (!v) return fail("an option without a value", argv[i]);
        if (!strcmp(argv[i], "--model")) model = v;
        else if (!strcmp(argv[i], "--dtype")) dtype = v;
        else if (!strcmp(argv[i], "--out")) out = v;
        else if (!strcmp(argv[i], "--max-tokens")) o.max_tokens = atoi(v);
        else if (!strcmp(argv[i], "--max-sequences")) o.max_sequences = atoi(v);
        else return fail("unknown option", argv[i]);
        i++;
    }
    if (!model || !out || (strcmp(dtype, "bfloat16") && strcmp(dtype, "float32")))
        return fail("usage: trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--max-sequences N]", NULL);
    o.dtype = !strcmp(dtype, "float32") ? DTYPE_FLOAT32 : DTYPE_BFLOAT16;
    CMLLanguageModel* lm = cml_lm_load(model, &o);
    Request* req = (Request*)malloc((size_t)(o.max_sequences > 0 ? o.max_sequences : 1) * sizeof *req);
    if (!lm || !req) return fail("cannot load", model);
    for (int i = 0; i < o.max_sequences; i++) req[i].seq = -1;
    char* text = NULL;
    size_t cap = 0;
    ssize_t len;
    int rc = 0;
    while (!rc && (len = getline(&text, &cap, stdin)) > 0) {
        if (strspn(text, " \t\r\n") == (size_t)len) continue;
        CMLJson* line = cml_json_parse(text, (size_t)len);
        rc = line ? run_line(lm, out, req, o.max_sequences, line) : fail("a line that is not JSON", NULL);
        cml_json_free(line);
    }
    free(text);
    free(req);
    cml_lm_free(lm);
    return rc;
}
