/* Grouped heads whose projections are convolved over time and whose scores are capped and mixed across heads: configuration,
 * weights, state, and the launches of a step.
 *
 *   mixer     conv (taps), softcap, beside what grouped heads have
 *   tensors   q.conv, k.conv, v.conv [channels, taps], talk [heads, heads]
 *
 * The scores of a step's rows pass through memory on their way into the softmax. Their buffer is made once, of bounded size, and
 * rows or tiles go through it a few at a time where it does not hold all of them. The latest projections of a sequence lie
 * in a ring per slot; tokens at a sequence's start do not look at it, so nothing is cleared when slots change hands. */
#include <stdlib.h>

#include "cml_lm_layered.h"

#define SCORES_BYTES ((size_t)192 << 20)
#define TILE 64

int cml_talk_read(const CMLJson* mixer, Layer* l, int index) {
    const GroupedForm* form = &l->kind->grouped;
    cmlb200_attn* a = &l->attn;
    double cap = 0.0;
    if (form->conv && (cml_json_int(mixer, "conv", &a->taps) || a->taps <= 0 || a->taps > 64)) { LOG_ERROR("layer %d: conv is missing or not 1 .. 64", index); return -1; }
    if (!form->talk) return 0;
    if (!cml_json_double(mixer, "softcap", &cap) && cap <= 0.0) { LOG_ERROR("layer %d: softcap", index); return -1; }
    if (a->heads > cmlb200_talk_scores_heads()) { LOG_ERROR("layer %d: %d heads that mix their scores, %d at most", index, a->heads, cmlb200_talk_scores_heads()); return -1; }
    a->cap = (float)cap;
    return 0;
}

int cml_talk_load(const CMLSafetensors* st, const char* prefix, Layer* l) {
    const GroupedForm* form = &l->kind->grouped;
    const cmlb200_attn* a = &l->attn;
    static const char* const taps[3] = {"q.conv", "k.conv", "v.conv"};
    const int channels[3] = {a->heads * a->dim, a->kv_heads * a->dim, a->kv_heads * a->vdim};
    if (form->conv && lml_load_taps(st, prefix, taps, channels, 3, a->taps, &l->w.conv)) return -1;
    if (!form->talk) return 0;
    CMLSafetensor t;
    if (lml_find(st, prefix, "talk", a->heads, a->heads, &t)) return -1;
    const size_t n = (size_t)a->heads * (size_t)a->heads;
    float* v = (float*)malloc(n * sizeof(float));
    if (!v) return -1;
    for (size_t i = 0; i < n; i++) v[i] = lml_element(&t, i);
    const int rc = lml_upload((void**)&l->w.talk, v, n * sizeof(float));
    free(v);
    return rc;
}

int cml_talk_make_state(Layer* l, const LayerWeights* w, int slots) {
    cmlb200_attn* a = &l->attn;
    a->conv = w->conv;
    a->talk = w->talk;
    const size_t channels = (size_t)(a->heads + a->kv_heads) * (size_t)a->dim + (size_t)a->kv_heads * (size_t)a->vdim;
    return a->taps ? lml_zeroed((void**)&a->ring, (size_t)slots * (size_t)a->taps * channels * sizeof(float)) : 0;
}

/* Row stride of a layer's scores: the keys that a tile of rows may see together, its first row's rounded down to 16. */
static int scores_ld(const Layered* m, const cmlb200_attn* a) {
    const long reach = a->window > 0 && (long)a->window + TILE + 15 < m->scores_keys ? (long)a->window + TILE + 15 : m->scores_keys;
    return lml_round_up((int)reach, 64);
}

/* Room for at least one tile, or one row per slot, of every layer; for all tiles of a step if that is not too much. */
int cml_talk_make_scores(Layered* m, int slots, int table_ld, int block_size) {
    size_t least = 0, all = 0, q = 0;
    m->scores_keys = table_ld * block_size;
    for (int i = 0; i < m->num_layers; i++) {
        const Layer* l = &m->layers[i];
        if (l->kind->form == MIXER_LATENT || (!l->kind->grouped.talk && !l->kind->grouped.conv)) continue;
        const size_t row = (size_t)l->attn.heads * (size_t)scores_ld(m, &l->attn);
        const size_t some = row * (size_t)(m->f32 ? slots : lml_most(slots, TILE)), every = row * (size_t)(m->f32 ? m->max_rows : (m->max_rows / TILE + slots) * TILE);
        if (some > least) least = some;
        if (every > all) all = every;
        if ((size_t)l->attn.heads * (size_t)l->attn.dim_ld > q) q = (size_t)l->attn.heads * (size_t)l->attn.dim_ld;
    }
    if (!q) return 0;
    const size_t most = SCORES_BYTES / sizeof(float);
    m->scores_room = all < most ? (all > least ? all : least) : (least > most ? least : most);
    return lml_zeroed((void**)&m->scores, m->scores_room * sizeof(float)) || lml_zeroed(&m->q_rows_out, (size_t)m->max_rows * q * (m->f32 ? 4 : 2)) ? -1 : 0;
}

int cml_talk_run(const Layered* m, const cmlb200_attn* layer, const CMLLMBatch* b, void* st) {
    cmlb200_attn a = *layer;
    const int ld = scores_ld(m, &a);
    const size_t row = (size_t)a.heads * (size_t)ld, q_row = (size_t)a.heads * (size_t)a.dim_ld;
    DEV(cmlb200_rotate_append(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, 0, b->rows, b->one_rows, m->q_rows_out, st));
    if (b->num_runs && a.taps > 1) DEV(cmlb200_ring_rows(&a, m->qkvg, m->ld_qkvg, b->d_runs, b->num_runs, st));
    a.scores = m->scores;
    a.scores_ld = ld;
    if (m->f32) {
        const int at_once = (int)(m->scores_room / row < 65535 ? m->scores_room / row : 65535);
        for (int r = 0; r < b->rows; r += at_once) {
            const int n = b->rows - r < at_once ? b->rows - r : at_once;
            DEV(cmlb200_talk_scores_rows(&a, (const float*)m->q_rows_out + (size_t)r * q_row, b->d_pos + r, b->d_slot + r, n, ld, m->scores, ld, st));
            DEV(cmlb200_attention_rows_f32(&a, m->qkvg + (size_t)r * (size_t)m->ld_qkvg, m->ld_qkvg, b->d_pos + r, b->d_slot + r, n,
                                           (float*)m->att + (size_t)r * (size_t)m->ld_att, m->ld_att, st));
        }
        return 0;
    }
    const int tiles = (int)(m->scores_room / (row * TILE) < 65535 ? m->scores_room / (row * TILE) : 65535);
    for (int t = 0; t < b->tiles; t += tiles) {
        const int n = b->tiles - t < tiles ? b->tiles - t : tiles;
        DEV(cmlb200_talk_scores_tiles(&a, (const uint16_t*)m->q_rows_out, b->d_tiles + 4 * t, n, ld, m->scores, ld, st));
        DEV(cmlb200_attention_tiles(&a, m->qkvg, m->ld_qkvg, b->d_tiles + 4 * t, n, (uint16_t*)m->att, m->ld_att, st));
    }
    if (b->one_rows) {
        const int keys = b->max_keys + 1 < ld ? b->max_keys + 1 : ld;
        DEV(cmlb200_talk_scores_rows(&a, m->q_rows_out, b->d_pos, b->d_slot, b->one_rows, keys, m->scores, ld, st));
        DEV(cmlb200_attention_one(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, b->one_rows, keys, (uint16_t*)m->att, m->ld_att, st));
    }
    return 0;
}
