/* The minimal gated recurrence among the layered models' mixers: configuration, state and the launches of a step.
 *
 *   mixer     width
 *   tensors   z and x (each with a bias .b), g, which are rows of the layer's one projection, and o, a product of its own
 *
 * A state is `width` floats per sequence slot. What a slot held before is not looked at by a sequence that starts in it, so
 * nothing is cleared when a sequence is opened or closed. */
#include "cml_lm_layered.h"

int cml_gru_read(const CMLJson* mixer, Layer* l, int index) {
    cmlb200_gru* a = &l->gru;
    if (cml_json_int(mixer, "width", &a->width) || a->width <= 0 || a->width > (1 << 20)) { LOG_ERROR("layer %d: width of the recurrence is missing or does not fit", index); return -1; }
    return 0;
}

int cml_gru_make_state(Layer* l, int slots) { return lml_zeroed((void**)&l->gru.state, (size_t)slots * (size_t)l->gru.width * sizeof(float)); }

int cml_gru_run(const Layered* m, const Layer* l, const CMLLMBatch* b, int col, void* st) {
    const int type = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    uint8_t* out = (uint8_t*)m->att + (size_t)col * (m->f32 ? 4 : 2);
    if (b->num_runs) DEV(cmlb200_gru_rows(&l->gru, m->qkvg, m->ld_qkvg, b->d_runs, b->num_runs, out, type, m->ld_att, st));
    if (b->one_rows) DEV(cmlb200_gru_one(&l->gru, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, b->one_rows, out, type, m->ld_att, st));
    return 0;
}
