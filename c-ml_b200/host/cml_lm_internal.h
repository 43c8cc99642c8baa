/* What a model class provides to the core in cml_lm.c. */
#ifndef CML_LM_INTERNAL_H
#define CML_LM_INTERNAL_H

#include "cml_internal.h"
#include "cml_json.h"
#include "cml_lm.h"

/* One entry's rows that make more than one tile. */
typedef struct CMLLMPortion {
    int row, rows, slot, pos;       /* first row and its position */
    int tile;                       /* its first tile */
} CMLLMPortion;

/* A step as the kernels see it. Rows 0 .. one_rows - 1 are single tokens, at most one per sequence; the
 * rows behind them are prompt portions, cut into tiles of up to 64 rows: first those of one tile (short_rows rows,
 * a tile each), then the longer ones. */
typedef struct CMLLMBatch {
    int rows, one_rows, tiles;
    int short_rows, short_tiles, short_keys;         /* short_keys: most keys of such a tile, its own included */
    const CMLLMPortion* portions;   /* host: the longer ones */
    int num_portions;
    int max_keys;                   /* no single-token row has more cached keys than this */
    const int *d_tokens, *d_pos, *d_slot;
    const int* d_tiles;             /* {first row, rows, slot, position of the first row} each */
    const int* d_runs;              /* whole portions, the same way, in the order of their rows */
    int num_runs;
    const int* d_table;             /* [slots][table_ld] block ids */
    int table_ld;
} CMLLMBatch;

typedef struct CMLLMInfo {
    int vocab;
    int window;                     /* no layer looks further back than this many tokens (itself included); 0: no bound */
    int keep_first;                 /* except at a sequence's first tokens, up to this many */
    CMLTokenizer* tokenizer;
} CMLLMInfo;

typedef struct CMLLMClass {
    const char* architecture;
    /* path as given to cml_lm_load; config: the parsed config.json, NULL for a GGUF file */
    void* (*load)(const char* path, const CMLJson* config, const CMLLMOptions* options, CMLLMInfo* info);
    void (*free)(void* model);
    /* Classes over the paged pool: pools of `blocks` blocks, for `slots` sequences whose block tables have `table_ld` entries; the layers of a step (enqueued on the stream);
     * final norm and vocabulary projection of rows d_rows[0 .. n-1] of that step into d_logits [n][vocab]. */
    int (*make_pools)(void* model, int blocks, int block_size, int slots, int table_ld);
    int (*forward)(void* model, const CMLLMBatch* batch, void* stream);
    int (*head)(void* model, const int* d_rows, int n, float* d_logits, void* stream);
    int (*check)(void* model, const CMLLMBatch* batch);      /* after the stream drained: -1 when a bounded wait expired */
    /* Classes with caches of their own instead (make_pools == NULL) */
    int (*open)(void* model);
    int (*close)(void* model, int seq);
    int (*length)(void* model, int seq);
    int (*step)(void* model, const CMLLMEntry* entries, int num_entries, float* logits);
} CMLLMClass;

/* Classes register themselves before main (a program links those it wants). */
void cml_lm_register(const CMLLMClass* cls);

#endif
