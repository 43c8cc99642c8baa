/* The gated delta rule among the layered models' mixers: configuration, weights, state and the launches of a step.
 *
 *   mixer     heads, kv_heads, dim, vdim, conv (taps of the convolutions over time)
 *   tensors   q, k, v (each with .conv [channels, taps]), b (step sizes), a1 / a2, dt_bias and A_log (decays), g1 / g2
 *             (gate), norm, and o, which the layer stacks beside the other mixer's
 *
 * q, k, v, b, a1 and g1 are rows of the layer's one projection. a2 and g2 make decays and gates of every head's channels
 * from a few columns. State and ring belong to a sequence's slot; what a slot held before is not looked at by a sequence
 * that starts in it, so nothing is cleared when a sequence is opened or closed. */
#include <math.h>
#include <stdlib.h>
#include <string.h>

#include "cml_lm_layered.h"

static int channels_of(const cmlb200_delta* a) { return 2 * a->kv_heads * a->dim + a->heads * a->vdim; }

int cml_delta_read(const CMLJson* mixer, Layer* l, int index, int col) {
    cmlb200_delta* a = &l->delta;
    if (cml_json_int(mixer, "heads", &a->heads) || cml_json_int(mixer, "kv_heads", &a->kv_heads) || cml_json_int(mixer, "dim", &a->dim) ||
        cml_json_int(mixer, "vdim", &a->vdim) || cml_json_int(mixer, "conv", &a->taps) || a->heads <= 0 || a->heads > 8192 || a->kv_heads <= 0 ||
        a->heads % a->kv_heads || a->dim <= 0 || a->dim > 256 || a->vdim <= 0 || a->vdim > 256 || a->taps <= 0 || a->taps > 64) {
        LOG_ERROR("layer %d: heads, kv_heads, dim, vdim (up to 256) or conv (up to 64) of the delta rule are missing or do not fit", index);
        return -1;
    }
    a->vdim_ld = lml_round_up(a->vdim, 4);
    a->col = col;
    return 0;
}

int cml_delta_ranks(const CMLSafetensors* st, const char* prefix, Layer* l, int width) {
    CMLSafetensor t;
    if (lml_find(st, prefix, "mix.right.a1", -1, width, &t)) return -1;
    l->a_rank = (int)t.shape[0];
    if (lml_find(st, prefix, "mix.right.g1", -1, width, &t)) return -1;
    l->g_rank = (int)t.shape[0];
    return 0;
}

static int load_rates(const CMLSafetensors* st, const char* prefix, int heads, float** dst) {
    CMLSafetensor t;
    if (lml_find(st, prefix, "mix.right.A_log", heads, 0, &t)) return -1;
    float* v = (float*)malloc((size_t)heads * sizeof(float));
    if (!v) return -1;
    for (int h = 0; h < heads; h++) v[h] = expf(lml_element(&t, (size_t)h));
    const int rc = lml_upload((void**)dst, v, (size_t)heads * sizeof(float));
    free(v);
    return rc;
}

int cml_delta_load(Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l) {
    const cmlb200_delta* a = &l->delta;
    LayerWeights* w = &l->w;
    const char *a2[1] = {"mix.right.a2"}, *g2[1] = {"mix.right.g2"};
    static const char* const taps[3] = {"mix.right.q.conv", "mix.right.k.conv", "mix.right.v.conv"};
    const int decays[1] = {a->heads * a->dim}, gates[1] = {a->heads * a->vdim}, channels[3] = {a->kv_heads * a->dim, a->kv_heads * a->dim, a->heads * a->vdim};
    return lml_load_taps(st, prefix, taps, channels, 3, a->taps, &w->conv) || load_rates(st, prefix, a->heads, &w->rate) ||
           lml_load_vector(st, prefix, "mix.right.dt_bias", decays[0], 0.f, &w->dt_bias) || lml_load_vector(st, prefix, "mix.right.norm", a->vdim, 0.f, &w->o_norm) ||
           lml_load_matrix(m, st, prefix, a2, decays, 1, l->a_rank, 0, &w->wa) || lml_load_matrix(m, st, prefix, g2, gates, 1, l->g_rank, 0, &w->wg) ? -1 : 0;
}

int cml_delta_activations(Layered* m, int rows) {
    int dec = 0, gate = 0, low = 0;
    long work = 0;
    for (int i = 0; i < m->num_layers; i++) {
        const Layer *l = &m->layers[i], *s = &m->layers[l->source];
        if (l->kind->form != MIXER_PARALLEL || l->kind->beside != BESIDE_DELTA) continue;
        dec = lml_most(dec, l->delta.heads * l->delta.dim);
        gate = lml_most(gate, l->delta.heads * l->delta.vdim);
        low = lml_most(low, lml_round_up(s->a_rank, 64) + lml_round_up(s->g_rank, 64));
        const long floats = cmlb200_delta_work_floats(&l->delta, rows, m->max_sequences);
        if (floats > work) work = floats;
    }
    if (!dec) return 0;
    m->ld_dec = lml_round_up(dec, 16);
    m->ld_gate = lml_round_up(gate, 16);
    m->ld_low = low;
    const size_t R = (size_t)rows;
    return lml_zeroed((void**)&m->dec, R * (size_t)m->ld_dec * 4) || lml_zeroed((void**)&m->gate, R * (size_t)m->ld_gate * 4) ||
           lml_zeroed((void**)&m->delta_work, (size_t)work * 4) || (!m->f32 && lml_zeroed(&m->low, R * (size_t)m->ld_low * 2)) ? -1 : 0;
}

int cml_delta_make_state(Layered* m, Layer* l, const LayerWeights* w, int slots) {
    cmlb200_delta* a = &l->delta;
    a->conv = w->conv;
    a->rate = w->rate;
    a->dt_bias = w->dt_bias;
    a->norm = w->o_norm;
    a->eps = m->eps;
    return lml_zeroed((void**)&a->state, (size_t)slots * (size_t)a->heads * (size_t)a->dim * (size_t)a->vdim_ld * 4) ||
           lml_zeroed((void**)&a->ring, (size_t)slots * (size_t)a->taps * (size_t)channels_of(a) * 4) ? -1 : 0;
}

/* Inputs of the decays and gate logits: second factors on the columns of the first ones, which lie side by side. */
static int second_factors(const Layered* m, const Layer* s, const LayerWeights* w, int col, int rows, void* st) {
    const int g = lml_round_up(s->a_rank, 64);
    if (m->f32)
        return lml_product(m, &w->wa, m->qkvg + col, m->ld_qkvg, rows, m->dec, m->ld_dec, st) ||
               lml_product(m, &w->wg, m->qkvg + col + s->a_rank, m->ld_qkvg, rows, m->gate, m->ld_gate, st) ? -1 : 0;
    uint16_t* low = (uint16_t*)m->low;
    DEV(cmlb200_pack_columns(m->qkvg, m->ld_qkvg, col, s->a_rank, s->g_rank, g, rows, low, m->ld_low, st));
    return lml_product(m, &w->wa, low, m->ld_low, rows, m->dec, m->ld_dec, st) || lml_product(m, &w->wg, low + g, m->ld_low, rows, m->gate, m->ld_gate, st) ? -1 : 0;
}

int cml_delta_run(const Layered* m, const Layer* l, const LayerWeights* w, const CMLLMBatch* b, int col, void* st) {
    const cmlb200_delta* a = &l->delta;
    const Layer* s = &m->layers[l->source];
    const int low = a->col + channels_of(a) + a->heads, type = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    uint8_t* out = (uint8_t*)m->att + (size_t)col * (m->f32 ? 4 : 2);
    if (second_factors(m, s, w, low, b->rows, st)) return -1;
    if (b->rows > b->one_rows)
        DEV(cmlb200_delta_rows(a, m->qkvg, m->ld_qkvg, m->dec, m->ld_dec, m->gate, m->ld_gate, b->d_pos, b->d_slot, b->one_rows, b->rows - b->one_rows, b->d_runs,
                               b->num_runs, m->delta_work, out, type, m->ld_att, st));
    if (b->one_rows)
        DEV(cmlb200_delta_one(a, m->qkvg, m->ld_qkvg, m->dec, m->ld_dec, m->gate, m->ld_gate, b->d_pos, b->d_slot, b->one_rows, out, type, m->ld_att, st));
    return 0;
}
