/* Language models behind one interface: the class registry, loading, sequences and their blocks, the
 * batch of a step, captured decode steps, and the scheduler's runner. See cml_lm.h.
 *
 * One pool of blocks serves all sequences; a block's id addresses the same slot range of every layer's
 * device pools. A step uploads one packed array of row descriptions (tokens, positions, slots, wanted rows,
 * prompt tiles) and the block table entries that changed, then enqueues the model's layers. Steps of single
 * tokens alone are captured as CUDA graphs, keyed by their shape: every pointer the kernels get is fixed,
 * what changes lives in the packed array. */
#include <pthread.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>
#include <sys/stat.h>
#include <time.h>

#include "cml_lm_internal.h"

#define BLOCK 16
#define TILE_ROWS 64
#define SMALL_ROWS 64              /* steps up to this many rows share one compact upload layout, and may be captured */
#define HEAD_ROWS 256              /* rows of logits per pass of the vocabulary projection */
#define MAX_CLASSES 16
#define MAX_GRAPHS 32

#define DEV(call) do { if (CML_DEV_FAIL((call), __func__)) return -1; } while (0)

typedef struct { int rows, want, greedy, keys; void* graph; unsigned stamp; } StepGraph;

struct CMLLanguageModel {
    const CMLLMClass* cls;
    void* model;
    CMLLMInfo info;
    CMLLMOptions opt;
    /* classes over the paged pool */
    CMLPagedKVCache* cache;
    void* stream;
    int table_ld;
    int *h_meta, *d_meta;          /* packed rows of a step; the host side is page-locked */
    size_t meta_cap;
    int *h_table, *d_table;        /* block table, host mirror page-locked */
    float* d_logits;
    int *d_picked, *h_picked;
    int *d_hist, *d_step;
    size_t hist_cap;
    StepGraph graphs[MAX_GRAPHS];
    unsigned clock;
    unsigned char* in_step;        /* per sequence: already in the entries being checked */
    CMLLMPortion* portions;        /* of the step being run, one per sequence at most */
};

/* ---- registry ------------------------------------------------------------------------------------ */
static const CMLLMClass* g_classes[MAX_CLASSES];
static int g_num_classes = 0;

void cml_lm_register(const CMLLMClass* cls) {
    if (g_num_classes < MAX_CLASSES) g_classes[g_num_classes++] = cls;
}
static const CMLLMClass* find_class(const char* architecture) {
    for (int i = 0; architecture && i < g_num_classes; i++)
        if (!strcmp(g_classes[i]->architecture, architecture)) return g_classes[i];
    return NULL;
}
int cml_lm_known(const char* architecture) { return find_class(architecture) != NULL; }

/* ---- load / free ----------------------------------------------------------------------------------- */
CMLLMOptions cml_lm_default_options(void) {
    CMLLMOptions o = {.dtype = DTYPE_BFLOAT16, .max_tokens = 8192, .max_sequences = 8, .max_step_rows = 0};
    return o;
}

static int make_buffers(CMLLanguageModel* lm) {
    const int blocks = (lm->opt.max_tokens + BLOCK - 1) / BLOCK;
    const size_t R = (size_t)lm->opt.max_step_rows;
    lm->cache = cml_paged_kv_cache_create_device(blocks, lm->opt.max_sequences, BLOCK);
    if (!lm->cache) return -1;
    /* blocks that every window has passed go back to the pool, so a sequence may outgrow it */
    lm->table_ld = lm->info.window > 0 ? 4 * blocks : blocks;
    lm->meta_cap = 4 * (R > SMALL_ROWS ? R : SMALL_ROWS) + 4 * (R / 2 + R / TILE_ROWS + SMALL_ROWS + 2 * (size_t)lm->opt.max_sequences);
    const size_t table = (size_t)lm->opt.max_sequences * (size_t)lm->table_ld * sizeof(int);
    DEV(cmlb200_stream_create(&lm->stream));
    DEV(cmlb200_host_alloc_pinned((void**)&lm->h_meta, lm->meta_cap * sizeof(int)));
    DEV(cmlb200_malloc((void**)&lm->d_meta, lm->meta_cap * sizeof(int)));
    DEV(cmlb200_host_alloc_pinned((void**)&lm->h_table, table));
    DEV(cmlb200_malloc((void**)&lm->d_table, table));
    memset(lm->h_table, 0, table);
    DEV(cmlb200_memset(lm->d_table, 0, table, lm->stream));
    DEV(cmlb200_malloc((void**)&lm->d_logits, (size_t)HEAD_ROWS * (size_t)lm->info.vocab * sizeof(float)));
    DEV(cmlb200_malloc((void**)&lm->d_picked, HEAD_ROWS * sizeof(int)));
    DEV(cmlb200_host_alloc_pinned((void**)&lm->h_picked, HEAD_ROWS * sizeof(int)));
    DEV(cmlb200_malloc((void**)&lm->d_step, sizeof(int)));
    return lm->cls->make_pools(lm->model, blocks, BLOCK, lm->opt.max_sequences, lm->table_ld);
}

CMLLanguageModel* cml_lm_load(const char* path, const CMLLMOptions* options) {
    static const char* who = "cml_lm_load";
    if (!path) { LOG_ERROR("%s: NULL path", who); return NULL; }
    CMLLMOptions o = options ? *options : cml_lm_default_options();
    if (o.dtype != DTYPE_BFLOAT16 && o.dtype != DTYPE_FLOAT32) { LOG_ERROR("%s: dtype must be bfloat16 or float32", who); return NULL; }
    if (o.max_tokens <= 0 || o.max_sequences <= 0 || o.max_tokens > (1 << 28)) { LOG_ERROR("%s: max_tokens %d, max_sequences %d", who, o.max_tokens, o.max_sequences); return NULL; }
    if (o.max_step_rows <= 0) o.max_step_rows = o.max_tokens;
    struct stat sb;
    char arch[128] = "";
    CMLJson* config = NULL;
    if (stat(path, &sb)) { LOG_ERROR("%s: no such model: %s", who, path); return NULL; }
    if (S_ISDIR(sb.st_mode)) {
        char file[4096];
        snprintf(file, sizeof file, "%s/config.json", path);
        config = cml_json_parse_file(file);
        const char* a = cml_json_string(config, "architecture");
        if (!a) { LOG_ERROR("%s: %s is missing, malformed or names no architecture", who, file); cml_json_free(config); return NULL; }
        snprintf(arch, sizeof arch, "%s", a);
    } else {
        snprintf(arch, sizeof arch, "llama");              /* the reader of other files than folders is GGUF's */
    }
    const CMLLMClass* cls = find_class(arch);
    if (!cls) { LOG_ERROR("%s: architecture '%s' is not known", who, arch); cml_json_free(config); return NULL; }
    CMLLanguageModel* lm = (CMLLanguageModel*)calloc(1, sizeof *lm);
    if (lm) {
        lm->cls = cls;
        lm->opt = o;
        lm->in_step = (unsigned char*)calloc((size_t)o.max_sequences, 1);
        lm->portions = (CMLLMPortion*)calloc((size_t)o.max_sequences, sizeof *lm->portions);
        lm->model = cls->load(path, config, &o, &lm->info);
    }
    cml_json_free(config);
    if (!lm || !lm->in_step || !lm->portions || !lm->model || (cls->make_pools && make_buffers(lm))) {
        LOG_ERROR("%s: %s could not be loaded", who, path);
        cml_lm_free(lm);
        return NULL;
    }
    return lm;
}

void cml_lm_free(CMLLanguageModel* lm) {
    if (!lm) return;
    for (int i = 0; i < MAX_GRAPHS; i++) if (lm->graphs[i].graph) cmlb200_graph_destroy(lm->graphs[i].graph);
    if (lm->model) lm->cls->free(lm->model);
    cml_paged_kv_cache_free(lm->cache);
    void* dev[] = {lm->d_meta, lm->d_table, lm->d_logits, lm->d_picked, lm->d_hist, lm->d_step};
    for (size_t i = 0; i < sizeof dev / sizeof dev[0]; i++) cmlb200_free(dev[i]);
    cmlb200_host_free_pinned(lm->h_meta);
    cmlb200_host_free_pinned(lm->h_table);
    cmlb200_host_free_pinned(lm->h_picked);
    if (lm->stream) cmlb200_stream_destroy(lm->stream);
    free(lm->in_step);
    free(lm->portions);
    free(lm);
}

const char* cml_lm_architecture(const CMLLanguageModel* lm) { return lm ? lm->cls->architecture : NULL; }
int cml_lm_vocab_size(const CMLLanguageModel* lm) { return lm ? lm->info.vocab : -1; }
CMLTokenizer* cml_lm_tokenizer(const CMLLanguageModel* lm) { return lm ? lm->info.tokenizer : NULL; }
int cml_lm_block_size(const CMLLanguageModel* lm) { return lm && lm->cache ? lm->cache->block_size : 0; }
int cml_lm_blocks_total(const CMLLanguageModel* lm) { return lm && lm->cache ? lm->cache->num_blocks : 0; }
int cml_lm_blocks_free(const CMLLanguageModel* lm) { return lm && lm->cache ? lm->cache->free_count : 0; }

/* ---- sequences --------------------------------------------------------------------------------------- */
int cml_lm_sequence_open(CMLLanguageModel* lm) {
    if (!lm) { LOG_ERROR("cml_lm_sequence_open: NULL model"); return -1; }
    return lm->cache ? cml_paged_cache_init_sequence(lm->cache) : lm->cls->open(lm->model);
}

static int seq_is_open(CMLLanguageModel* lm, int seq) {
    if (!lm || seq < 0 || seq >= lm->opt.max_sequences) return 0;
    return lm->cache ? lm->cache->sequences[seq].block_ids != NULL : lm->cls->length(lm->model, seq) >= 0;
}

int cml_lm_sequence_close(CMLLanguageModel* lm, int seq) {
    if (!seq_is_open(lm, seq)) { LOG_ERROR("cml_lm_sequence_close: sequence %d is not open", seq); return -1; }
    if (!lm->cache) return lm->cls->close(lm->model, seq);
    cml_paged_cache_free_sequence(lm->cache, seq);
    return 0;
}

int cml_lm_sequence_length(CMLLanguageModel* lm, int seq) {
    if (!seq_is_open(lm, seq)) return -1;
    return lm->cache ? lm->cache->sequences[seq].seq_len : lm->cls->length(lm->model, seq);
}

/* Takes the blocks of n further tokens and uploads the new part of the sequence's block table. */
static int grow_sequence(CMLLanguageModel* lm, int seq, int n) {
    CMLBlockTable* bt = &lm->cache->sequences[seq];
    const int had = bt->num_blocks;
    if (cml_paged_cache_extend(lm->cache, seq, n)) return -1;
    if (bt->num_blocks > had) {
        const size_t at = (size_t)seq * (size_t)lm->table_ld + (size_t)had, bytes = (size_t)(bt->num_blocks - had) * sizeof(int);
        memcpy(lm->h_table + at, bt->block_ids + had, bytes);
        DEV(cmlb200_memcpy_h2d(lm->d_table + at, lm->h_table + at, bytes, lm->stream));
    }
    return 0;
}

/* Blocks that every layer's window has passed go back to the pool, those of first tokens that stay in sight aside. */
static void release_passed(CMLLanguageModel* lm, int seq) {
    if (lm->info.window > 0) cml_paged_cache_release_between(lm->cache, seq, lm->info.keep_first, lm->cache->sequences[seq].seq_len - lm->info.window + 1);
}

/* ---- steps ------------------------------------------------------------------------------------------- */
/* Everything that can be wrong with a step, before anything changes. Returns the number of rows, -1. */
static int check_step(CMLLanguageModel* lm, const CMLLMEntry* entries, int n, int* want, const char* who) {
    if (!lm || !entries || n <= 0) { LOG_ERROR("%s: invalid arguments", who); return -1; }
    long rows = 0, blocks = 0;
    int bad = 0;
    *want = 0;
    memset(lm->in_step, 0, (size_t)lm->opt.max_sequences);
    for (int i = 0; i < n && !bad; i++) {
        const CMLLMEntry* e = &entries[i];
        bad = 1;
        if (!seq_is_open(lm, e->seq)) { LOG_ERROR("%s: sequence %d is not open", who, e->seq); break; }
        if (lm->in_step[e->seq]) { LOG_ERROR("%s: sequence %d twice in one step", who, e->seq); break; }
        lm->in_step[e->seq] = 1;
        if (!e->tokens || e->num_tokens <= 0 || e->num_want < 0 || (e->num_want && !e->want)) { LOG_ERROR("%s: entry %d is malformed", who, i); break; }
        int k = 0;
        while (k < e->num_tokens && e->tokens[k] >= 0 && e->tokens[k] < lm->info.vocab) k++;
        if (k < e->num_tokens) { LOG_ERROR("%s: token %d is outside the vocabulary of %d", who, e->tokens[k], lm->info.vocab); break; }
        k = 0;
        while (k < e->num_want && e->want[k] >= 0 && e->want[k] < e->num_tokens) k++;
        if (k < e->num_want) { LOG_ERROR("%s: place %d wanted of %d tokens", who, e->want[k], e->num_tokens); break; }
        if (lm->cache) {
            const int len = lm->cache->sequences[e->seq].seq_len;
            if ((long)len + e->num_tokens > (long)lm->table_ld * BLOCK) { LOG_ERROR("%s: sequence %d would grow beyond %ld tokens", who, e->seq, (long)lm->table_ld * BLOCK); break; }
            blocks += cml_paged_cache_blocks_for(lm->cache, e->seq, e->num_tokens);
        }
        rows += e->num_tokens;
        *want += e->num_want;
        bad = 0;
    }
    if (bad) return -1;
    if (rows > lm->opt.max_step_rows) { LOG_ERROR("%s: %ld tokens in a step of at most %d", who, rows, lm->opt.max_step_rows); return -1; }
    if (lm->cache && blocks > lm->cache->free_count) { LOG_ERROR("%s: %ld blocks needed, %d free", who, blocks, lm->cache->free_count); return -1; }
    return (int)rows;
}

static int round_keys(int keys) {
    int r = 128;
    while (r < keys) r *= 2;
    return r;
}

/* Fills the packed row array from the entries (whose sequences have grown already) and uploads it. */
static int upload_rows(CMLLanguageModel* lm, const CMLLMEntry* entries, int n, int rows, CMLLMBatch* b, const int** d_want) {
    const int stride = rows <= SMALL_ROWS ? SMALL_ROWS : (lm->opt.max_step_rows + 3) & ~3;
    int *tok = lm->h_meta, *pos = tok + stride, *slot = pos + stride, *want = slot + stride, *runs = want + stride;
    int *tiles = runs + 4 * lm->opt.max_sequences, num_runs = 0;
    int one = 0, one_keys = 0, w = 0, t = 0, short_rows = 0, short_tiles = 0, short_keys = 0, portions = 0;
    for (int i = 0; i < n; i++) {
        const int k = entries[i].num_tokens;
        one += k == 1;
        if (k > 1 && k <= TILE_ROWS) { short_rows += k; short_tiles++; }
    }
    /* next row and, for portions, next tile of each of the three kinds */
    int at_one = 0, at_short = one, at_long = one + short_rows, tile_short = 0;
    t = short_tiles;
    for (int i = 0; i < n; i++) {
        const CMLLMEntry* e = &entries[i];
        const int len = e->num_tokens, first = lm->cache->sequences[e->seq].seq_len - len;
        int* at = len == 1 ? &at_one : (len <= TILE_ROWS ? &at_short : &at_long);
        int* tile = len <= TILE_ROWS ? &tile_short : &t;
        const int r0 = *at;
        *at += len;
        for (int k = 0; k < len; k++) {
            tok[r0 + k] = e->tokens[k];
            pos[r0 + k] = first + k;
            slot[r0 + k] = e->seq;
        }
        for (int k = 0; k < e->num_want; k++) want[w++] = r0 + e->want[k];
        if (len == 1) { if (first > one_keys) one_keys = first; continue; }
        num_runs++;
        if (len <= TILE_ROWS && first + len > short_keys) short_keys = first + len;
        if (len > TILE_ROWS) { CMLLMPortion p = {r0, len, e->seq, first, t}; lm->portions[portions++] = p; }
        for (int k = 0; k < len; k += TILE_ROWS, ++*tile) {
            tiles[4 * *tile] = r0 + k;
            tiles[4 * *tile + 1] = len - k < TILE_ROWS ? len - k : TILE_ROWS;
            tiles[4 * *tile + 2] = e->seq;
            tiles[4 * *tile + 3] = first + k;
        }
    }
    for (int i = 0, at = 0; i < 2; i++)                    /* portions of one tile, then the longer ones, as their rows lie */
        for (int k = 0; k < n; k++) {
            const CMLLMEntry* e = &entries[k];
            if (e->num_tokens == 1 || (e->num_tokens > TILE_ROWS) != i) continue;
            const int r[4] = {one + at, e->num_tokens, e->seq, lm->cache->sequences[e->seq].seq_len - e->num_tokens};
            memcpy(runs, r, sizeof r);
            runs += 4;
            at += e->num_tokens;
        }
    DEV(cmlb200_memcpy_h2d(lm->d_meta, lm->h_meta, (4 * (size_t)stride + 4 * (size_t)lm->opt.max_sequences + 4 * (size_t)t) * sizeof(int), lm->stream));
    memset(b, 0, sizeof *b);
    b->rows = rows;
    b->one_rows = one;
    b->tiles = t;
    b->short_rows = short_rows;
    b->short_tiles = short_tiles;
    b->short_keys = short_keys;
    b->portions = lm->portions;
    b->num_portions = portions;
    b->max_keys = round_keys(one_keys);
    b->d_tokens = lm->d_meta;
    b->d_pos = lm->d_meta + stride;
    b->d_slot = lm->d_meta + 2 * stride;
    *d_want = lm->d_meta + 3 * stride;
    b->d_runs = lm->d_meta + 4 * stride;
    b->num_runs = num_runs;
    b->d_tiles = b->d_runs + 4 * lm->opt.max_sequences;
    b->d_table = lm->d_table;
    b->table_ld = lm->table_ld;
    return 0;
}

/* The launches of a step whose wanted rows fit one pass of the vocabulary projection. */
static int enqueue_step(CMLLanguageModel* lm, const CMLLMBatch* b, const int* d_want, int want, int greedy) {
    if (lm->cls->forward(lm->model, b, lm->stream)) return -1;
    if (!want) return 0;
    if (lm->cls->head(lm->model, d_want, want, lm->d_logits, lm->stream)) return -1;
    if (greedy) DEV(cmlb200_argmax(lm->d_logits, want, lm->info.vocab, lm->d_picked, lm->stream));
    return 0;
}

/* A captured step of that shape, or NULL. The first use of a shape runs eagerly (launchers set themselves
 * up), the second captures. */
static int run_captured(CMLLanguageModel* lm, const CMLLMBatch* b, const int* d_want, int want, int greedy) {
    StepGraph *g = NULL, *oldest = &lm->graphs[0];
    for (int i = 0; i < MAX_GRAPHS; i++) {
        StepGraph* c = &lm->graphs[i];
        if (c->stamp && c->rows == b->rows && c->want == want && c->greedy == greedy && c->keys == b->max_keys) g = c;
        if (c->stamp < oldest->stamp) oldest = c;
    }
    lm->clock++;
    if (!g) {
        if (oldest->graph) cmlb200_graph_destroy(oldest->graph);
        StepGraph fresh = {b->rows, want, greedy, b->max_keys, NULL, lm->clock};
        *oldest = fresh;
        return enqueue_step(lm, b, d_want, want, greedy);
    }
    g->stamp = lm->clock;
    if (!g->graph) {
        DEV(cmlb200_graph_begin(lm->stream));
        const int rc = enqueue_step(lm, b, d_want, want, greedy);
        void* made = NULL;
        if (CML_DEV_FAIL(cmlb200_graph_end(lm->stream, &made), "cml_lm_step") || rc) { if (made) cmlb200_graph_destroy(made); return -1; }
        g->graph = made;
    }
    DEV(cmlb200_graph_launch(g->graph, lm->stream));
    return 0;
}

static int run_step(CMLLanguageModel* lm, const CMLLMEntry* entries, int n, float* logits, int* picked, const char* who) {
    int want = 0;
    const int rows = check_step(lm, entries, n, &want, who), greedy = picked != NULL;
    if (rows < 0) return -1;
    if (want && !logits && !picked) { LOG_ERROR("%s: no room for the wanted logits", who); return -1; }
    for (int i = 0; i < n; i++) if (grow_sequence(lm, entries[i].seq, entries[i].num_tokens)) return -1;
    CMLLMBatch b;
    const int* d_want;
    if (upload_rows(lm, entries, n, rows, &b, &d_want)) return -1;
    const size_t V = (size_t)lm->info.vocab;
    const int first = want < HEAD_ROWS ? want : HEAD_ROWS;
    if ((b.one_rows == rows && rows <= SMALL_ROWS) ? run_captured(lm, &b, d_want, first, greedy) : enqueue_step(lm, &b, d_want, first, greedy)) return -1;
    for (int at = 0; at < want; at += HEAD_ROWS) {
        const int k = want - at < HEAD_ROWS ? want - at : HEAD_ROWS;
        if (at) {
            if (lm->cls->head(lm->model, d_want + at, k, lm->d_logits, lm->stream)) return -1;
            if (greedy) DEV(cmlb200_argmax(lm->d_logits, k, lm->info.vocab, lm->d_picked, lm->stream));
        }
        if (greedy) {
            DEV(cmlb200_memcpy_d2h(lm->h_picked, lm->d_picked, (size_t)k * sizeof(int), lm->stream));
            DEV(cmlb200_stream_sync(lm->stream));
            memcpy(picked + at, lm->h_picked, (size_t)k * sizeof(int));
        } else {
            DEV(cmlb200_memcpy_d2h(logits + (size_t)at * V, lm->d_logits, (size_t)k * V * sizeof(float), lm->stream));
        }
    }
    DEV(cmlb200_stream_sync(lm->stream));
    if (lm->cls->check && lm->cls->check(lm->model, &b)) { LOG_ERROR("%s: a bounded device-side wait expired", who); return -1; }
    for (int i = 0; i < n; i++) release_passed(lm, entries[i].seq);
    return 0;
}

int cml_lm_step(CMLLanguageModel* lm, const CMLLMEntry* entries, int num_entries, float* logits) {
    static const char* who = "cml_lm_step";
    int want;
    if (lm && !lm->cache) return check_step(lm, entries, num_entries, &want, who) < 0 ? -1 : lm->cls->step(lm->model, entries, num_entries, logits);
    return run_step(lm, entries, num_entries, logits, NULL, who);
}

static int argmax_row(const float* row, int n) {
    int best = 0;
    for (int i = 1; i < n; i++) if (row[i] > row[best]) best = i;
    return best;
}

int cml_lm_step_greedy(CMLLanguageModel* lm, const CMLLMEntry* entries, int num_entries, int* picked) {
    static const char* who = "cml_lm_step_greedy";
    if (!picked) { LOG_ERROR("%s: invalid arguments", who); return -1; }
    if (!lm || lm->cache) return run_step(lm, entries, num_entries, NULL, picked, who);
    int want = 0;
    if (check_step(lm, entries, num_entries, &want, who) < 0) return -1;
    float* lg = (float*)malloc((size_t)(want ? want : 1) * (size_t)lm->info.vocab * sizeof(float));
    const int rc = lg ? lm->cls->step(lm->model, entries, num_entries, lg) : -1;
    for (int i = 0; i < want && !rc; i++) picked[i] = argmax_row(lg + (size_t)i * (size_t)lm->info.vocab, lm->info.vocab);
    free(lg);
    return rc;
}

int cml_lm_decode_greedy(CMLLanguageModel* lm, const int* seqs, const int* first_tokens, int num_seqs, int steps, int* out_tokens, float* elapsed_ms) {
    static const char* who = "cml_lm_decode_greedy";
    if (!lm || !lm->cache || !seqs || !first_tokens || !out_tokens || num_seqs <= 0 || num_seqs > SMALL_ROWS || num_seqs > lm->opt.max_sequences || steps <= 0) {
        LOG_ERROR("%s: invalid arguments", who);
        return -1;
    }
    CMLLMEntry e[SMALL_ROWS];
    const int zero = 0;
    int want, max_len = 0;
    long blocks = 0;
    for (int i = 0; i < num_seqs; i++) { CMLLMEntry x = {seqs[i], &first_tokens[i], 1, &zero, 1}; e[i] = x; }
    if (check_step(lm, e, num_seqs, &want, who) < 0) return -1;
    for (int i = 0; i < num_seqs; i++) {
        blocks += cml_paged_cache_blocks_for(lm->cache, seqs[i], steps);
        if ((long)lm->cache->sequences[seqs[i]].seq_len + steps > (long)lm->table_ld * BLOCK) { LOG_ERROR("%s: sequence %d would grow beyond its block table", who, seqs[i]); return -1; }
        if (lm->cache->sequences[seqs[i]].seq_len + steps > max_len) max_len = lm->cache->sequences[seqs[i]].seq_len + steps;
    }
    if (blocks > lm->cache->free_count) { LOG_ERROR("%s: %ld blocks needed, %d free", who, blocks, lm->cache->free_count); return -1; }
    const size_t hist = (size_t)steps * (size_t)num_seqs * sizeof(int);
    if (hist > lm->hist_cap) {
        cmlb200_free(lm->d_hist);
        lm->d_hist = NULL;
        lm->hist_cap = 0;
        DEV(cmlb200_malloc((void**)&lm->d_hist, hist));
        lm->hist_cap = hist;
    }
    CMLLMBatch b;
    const int* d_want;
    for (int i = 0; i < num_seqs; i++) if (grow_sequence(lm, seqs[i], 1)) return -1;
    if (upload_rows(lm, e, num_seqs, num_seqs, &b, &d_want)) return -1;
    for (int i = 0; i < num_seqs; i++) if (steps > 1 && grow_sequence(lm, seqs[i], steps - 1)) return -1;
    b.max_keys = round_keys(max_len);
    DEV(cmlb200_memset(lm->d_step, 0, sizeof(int), lm->stream));
    int *d_tokens = lm->d_meta, *d_pos = lm->d_meta + SMALL_ROWS;
    void *e0 = NULL, *e1 = NULL, *graph = NULL;
    int rc = -1;
    if (CML_DEV_FAIL(cmlb200_event_create(&e0), who) || CML_DEV_FAIL(cmlb200_event_create(&e1), who)) goto done;
#define STEP_ONCE() (enqueue_step(lm, &b, d_want, num_seqs, 1) || \
                     CML_DEV_FAIL(cmlb200_advance_tokens(lm->d_picked, num_seqs, d_tokens, d_pos, lm->d_hist, lm->d_step, lm->stream), who))
    int s = 0;
    if (steps > 2) {                                       /* first step eager, the rest one captured step replayed */
        if (STEP_ONCE()) goto done;
        s = 1;
        if (CML_DEV_FAIL(cmlb200_stream_sync(lm->stream), who) || CML_DEV_FAIL(cmlb200_graph_begin(lm->stream), who)) goto done;
        const int bad = STEP_ONCE();
        if (CML_DEV_FAIL(cmlb200_graph_end(lm->stream, &graph), who) || bad) goto done;
    }
    if (CML_DEV_FAIL(cmlb200_event_record(e0, lm->stream), who)) goto done;
    const int timed = steps - s;
    for (; s < steps; s++)
        if (graph ? CML_DEV_FAIL(cmlb200_graph_launch(graph, lm->stream), who) : STEP_ONCE()) goto done;
#undef STEP_ONCE
    float ms = 0.f;
    if (CML_DEV_FAIL(cmlb200_event_record(e1, lm->stream), who) || CML_DEV_FAIL(cmlb200_event_elapsed_ms(e0, e1, &ms), who) ||
        CML_DEV_FAIL(cmlb200_memcpy_d2h(out_tokens, lm->d_hist, hist, lm->stream), who) || CML_DEV_FAIL(cmlb200_stream_sync(lm->stream), who))
        goto done;
    if (elapsed_ms) *elapsed_ms = ms * (float)steps / (float)timed;
    for (int i = 0; i < num_seqs; i++) release_passed(lm, seqs[i]);
    rc = lm->cls->check && lm->cls->check(lm->model, &b) ? -1 : 0;
done:
    if (graph) cmlb200_graph_destroy(graph);
    if (e0) cmlb200_event_destroy(e0);
    if (e1) cmlb200_event_destroy(e1);
    return rc;
}

/* ---- scheduler --------------------------------------------------------------------------------------- */
/* The most blocks a request holds at any time: all of its tokens, or, where every layer has a window, the
 * largest portion of its prompt and the tokens still in reach of it. */
static int blocks_of(const CMLLanguageModel* lm, const CMLSequenceRequest* r) {
    if (!lm->cache) return 0;
    const int bs = lm->cache->block_size;
    long tokens = (long)r->num_prompt_tokens + r->max_new_tokens;
    if (lm->info.window > 0) {
        const long portion = r->num_prompt_tokens < lm->opt.max_step_rows ? r->num_prompt_tokens : lm->opt.max_step_rows;
        const long reach = lm->info.window + portion + bs + (lm->info.keep_first ? lm->info.keep_first + bs : 0);
        if (reach < tokens) tokens = reach;
    }
    return (int)((tokens + bs - 1) / bs);
}

static int pick_token(CMLLanguageModel* lm, float* row, const CMLGenerationConfig* config) {
    int shape[2] = {1, lm->info.vocab};
    TensorConfig tc = {.dtype = DTYPE_FLOAT32, .device = DEVICE_CPU, .has_dtype = true, .has_device = true};
    Tensor* t = tensor_from_data(row, shape, 2, &tc);
    const int tok = t ? cml_llama_sample_token(t, config) : -1;
    tensor_free(t);
    return tok;
}

int cml_serving_run_lm(CMLServingContext* ctx, CMLLanguageModel* lm, const CMLGenerationConfig* config, int max_steps,
                       void (*on_finish)(const CMLSequenceRequest* request, void* user), void* user) {
    static const char* who = "cml_serving_run_lm";
    if (!ctx || !lm) { LOG_ERROR("%s: NULL argument", who); return -1; }
    const int B = ctx->config.max_batch_size, V = lm->info.vocab, sampled = config && config->do_sample && config->temperature > 0.f;
    const int eos = config ? config->eos_token_id : -1;
    CMLLMEntry* e = (CMLLMEntry*)calloc((size_t)B, sizeof *e);
    CMLSequenceRequest** who_is = (CMLSequenceRequest**)calloc((size_t)B, sizeof *who_is);
    int *last = (int*)calloc((size_t)B, sizeof(int)), *picked = (int*)calloc((size_t)B, sizeof(int));
    float* logits = sampled ? (float*)malloc((size_t)B * (size_t)V * sizeof(float)) : NULL;
    int steps = 0, rc = e && who_is && last && picked && (logits || !sampled) ? 0 : -1;
    while (rc == 0 && (ctx->queue_count > 0 || ctx->batch_size > 0) && (max_steps <= 0 || steps < max_steps)) {
        cml_serving_step(ctx);
        long committed = 0;
        for (int i = 0; i < ctx->batch_size; i++)
            if (ctx->active_batch[i]->paged_seq_id >= 0) committed += blocks_of(lm, ctx->active_batch[i]);
        /* admission in order of arrival: a request starts when the pool can hold it to its end */
        for (int i = 0; i < ctx->batch_size; i++) {
            CMLSequenceRequest* r = ctx->active_batch[i];
            if (r->paged_seq_id >= 0 || r->status == CML_SEQ_STATUS_ERROR) continue;
            int bad = 0;
            for (int k = 0; k < r->num_prompt_tokens; k++) bad |= r->prompt_tokens[k] < 0 || r->prompt_tokens[k] >= V;
            const int need = blocks_of(lm, r);
            const long length = (long)r->num_prompt_tokens + r->max_new_tokens, most = lm->cache ? (long)lm->table_ld * BLOCK : lm->opt.max_tokens;
            if (bad || length > most || (lm->cache && need > lm->cache->num_blocks)) { r->status = CML_SEQ_STATUS_ERROR; continue; }
            if (lm->cache && committed + need > lm->cache->num_blocks) break;
            const int open = lm->cache ? lm->cache->num_sequences : 0;
            if (lm->cache && open >= lm->opt.max_sequences) break;
            const int seq = cml_lm_sequence_open(lm);
            if (seq < 0) { if (!i) rc = -1; break; }
            r->paged_seq_id = seq;
            r->current_pos = 0;
            committed += need;
        }
        if (rc) break;
        /* one batch: the next token of whoever decodes, then prompt portions as far as the step has room */
        int n = 0, room = lm->opt.max_step_rows;
        for (int pass = 0; pass < 2; pass++) {
            for (int i = 0; i < ctx->batch_size; i++) {
                CMLSequenceRequest* r = ctx->active_batch[i];
                if (r->paged_seq_id < 0 || r->status != CML_SEQ_STATUS_DECODING || room <= 0) continue;
                const int prompt_left = r->num_prompt_tokens - r->current_pos;
                if ((prompt_left <= 0) != (pass == 0)) continue;
                CMLLMEntry x = {r->paged_seq_id, NULL, 1, &last[n], 1};
                if (pass == 0) x.tokens = &r->generated_tokens[r->num_generated - 1];
                else {
                    x.tokens = r->prompt_tokens + r->current_pos;
                    x.num_tokens = prompt_left < room ? prompt_left : room;
                    if (x.num_tokens < prompt_left) x.num_want = 0;
                }
                last[n] = x.num_tokens - 1;
                room -= x.num_tokens;
                who_is[n] = r;
                e[n++] = x;
            }
        }
        if (n) {
            rc = sampled ? cml_lm_step(lm, e, n, logits) : cml_lm_step_greedy(lm, e, n, picked);
            if (rc) break;
            steps++;
            for (int k = 0, w = 0; k < n; k++) {
                CMLSequenceRequest* r = who_is[k];
                r->current_pos += e[k].num_tokens;
                if (!e[k].num_want) continue;
                const int tok = sampled ? pick_token(lm, logits + (size_t)w * (size_t)V, config) : picked[w];
                w++;
                if (tok < 0) { rc = -1; break; }
                if (r->num_generated < r->gen_capacity) r->generated_tokens[r->num_generated++] = tok;
            }
        }
        int retired = 0;
        for (int i = 0; i < ctx->batch_size && rc == 0;) {
            CMLSequenceRequest* r = ctx->active_batch[i];
            const int done = r->status == CML_SEQ_STATUS_ERROR || (r->paged_seq_id >= 0 && r->num_generated > 0 &&
                             (r->num_generated >= r->max_new_tokens || (eos >= 0 && r->generated_tokens[r->num_generated - 1] == eos)));
            if (!done) { i++; continue; }
            if (on_finish) on_finish(r, user);
            if (r->paged_seq_id >= 0) cml_lm_sequence_close(lm, r->paged_seq_id);
            cml_serving_finish_request(ctx, r->request_id);
            retired++;
        }
        if (!n && !retired && rc == 0) { LOG_ERROR("%s: no request can be run (are sequences open outside the scheduler?)", who); rc = -1; }
    }
    free(e); free(who_is); free(last); free(picked); free(logits);
    return rc ? -1 : steps;
}

/* ---- generation -------------------------------------------------------------------------------------- */
typedef struct { CMLGenerationResult* res; int ok; } Finished;
static void take_result(const CMLSequenceRequest* r, void* user) {
    Finished* f = (Finished*)user;
    if (r->status == CML_SEQ_STATUS_ERROR) return;
    memcpy(f->res->token_ids + f->res->num_tokens, r->generated_tokens, (size_t)r->num_generated * sizeof(int));
    f->res->num_tokens += r->num_generated;
    f->ok = 1;
}

CMLGenerationResult* cml_lm_generate(CMLLanguageModel* lm, const int* prompt, int num_tokens, const CMLGenerationConfig* config) {
    if (!lm || !prompt || num_tokens <= 0) { LOG_ERROR("cml_lm_generate: invalid arguments"); return NULL; }
    CMLGenerationConfig c = cml_generation_default_config();
    c.do_sample = false;
    c.eos_token_id = -1;
    if (config) c = *config;
    if (c.max_new_tokens <= 0) c.max_new_tokens = 256;
    CMLServingConfig sc = cml_serving_default_config();
    sc.max_batch_size = 1;
    sc.max_queue_size = 1;
    CMLServingContext* ctx = cml_serving_create(&sc);
    CMLGenerationResult* res = (CMLGenerationResult*)calloc(1, sizeof *res);
    Finished f = {res, 0};
    struct timespec t0, t1;
    clock_gettime(CLOCK_MONOTONIC, &t0);
    if (ctx && res && (res->token_ids = (int*)malloc((size_t)(num_tokens + c.max_new_tokens) * sizeof(int)))) {
        memcpy(res->token_ids, prompt, (size_t)num_tokens * sizeof(int));
        res->num_tokens = num_tokens;
        if (cml_serving_submit(ctx, prompt, num_tokens, c.max_new_tokens) < 0 || cml_serving_run_lm(ctx, lm, &c, 0, take_result, &f) < 0) f.ok = 0;
    }
    clock_gettime(CLOCK_MONOTONIC, &t1);
    cml_serving_free(ctx);
    if (!f.ok) { cml_generation_result_free(res); return NULL; }
    const double ms = (double)(t1.tv_sec - t0.tv_sec) * 1e3 + (double)(t1.tv_nsec - t0.tv_nsec) / 1e6;
    res->total_time_ms = (float)ms;
    if (ms > 0.0) res->tokens_per_second = (float)((res->num_tokens - num_tokens) * 1e3 / ms);
    if (lm->info.tokenizer) res->text = cml_tokenizer_decode(lm->info.tokenizer, res->token_ids, res->num_tokens);
    return res;
}
