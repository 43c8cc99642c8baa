/* Decoder-only models described layer by layer in config.json and stored as safetensors. A design is a row
 * of switches (LayeredDesign); sizes, windows, scales and the order of layers come from the file.
 *
 *   config.json     architecture, vocab, width, norm.eps, layers: [{type, mixer, mlp, weights_of?}]; designs with streams also
 *                   streams, embedding.scale and logit_softcap; designs with loops also loop {start, stop, times}
 *   mixer           grouped heads: heads, kv_heads, dim, vdim, scale, mask {size, keep_first}, q_temp {coef, every}, rot {base, dims,
 *                   scaling {factor}, or {factor, low, high, original}}, and what cml_lm_talk.c says
 *                   latents: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask.size, rot {base, dims, scaling {factor,
 *                   original, fast, slow}}, kv_from (the layer whose cache this one reads)
 *                   parallel: left (grouped heads), right (gated delta rule, cml_lm_delta.c, with left_scale and right_scale; or
 *                   minimal gated recurrence, cml_lm_gru.c)
 *   mlp             {kind: "dense", ff}, {kind: "moe", expert {ff, limit}, router {experts, top, identity, groups {count, keep},
 *                   scale}, shared {ff}} or null
 *   weights_of      index of the layer whose tensors this one uses; its cache is its own
 *   tensors         embed, final.norm, head, l<i>.norm1 / norm1b / norm2 / norm2b (as the design has them),
 *                   l<i>.mix.q / k / v / g / o / q.norm / k.norm / sink and biases .b, the same under mix.left and mix.right, or
 *                   q (or dq / dq.norm / uq) / dkv / dkv.norm / uk / uv / sink / g / o, l<i>.mlp.gate / up / down, up / down / act, or
 *                   router, correction, e<j>.gate / up / down and shared.gate / up / down, l<i>.hc1 / hc2 .in / out / mix, l<i>.rg1 /
 *                   rg2 and biases; linear weights [out, in]
 *
 * On the device all of a layer's projections of its input are one matrix, and the feed-forward's gate and up rows one
 * matrix interleaved in groups of 16 (the epilogues of both products pair them). Two mixers side by side leave their
 * outputs, scaled, in neighbouring columns, which one output matrix takes, unless their outputs are normed one by one. Between two
 * sublayers runs one kernel: norm of the finished sublayer's output, residual add, norm for the next one; with streams, the
 * join into all of them, what the next sublayer reads, and its norm. Where both sublayers read the same row, the gates' and
 * the router's rows belong to the layer's one projection too, and one kernel joins both. A layer that runs several times
 * has an entry for every pass, with a cache of its own and the first pass's weights. The residual, norms,
 * scores and weights are fp32; in the bfloat16 form matrix operands are bf16 and cached keys, values and latents
 * fp16. Up to 32 rows a step streams its weights through the decode product, above that tcgen05 tiles.
 *
 * A latent layer attends in one of two ways. Single tokens and portions of one tile bring their queries to the latents
 * (Wuk^T q) and what they weighted back to values (Wuv o). Longer portions expand the latents in their reach into
 * per-head keys and values in a scratch cache and run the attention of grouped heads over that. */
#include <math.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include "cml_lm_layered.h"

#define MAX_LAYERS 4096
#define EXPAND_KEYS 65536          /* keys the scratch cache of long portions holds at most (CMLB200_EXPAND_KEYS: another number) */

static const LayeredDesign kDesigns[] = {
    {.architecture = "Rarolorn",
     .mixers = {{.type = "attention", .form = MIXER_GROUPED, .grouped = {.norm = NORM_WIDE, .sink = SINK_ONE, .linear_bias = 1, .head_gate = 1}}},
     .position_base = 10000.0, .input_norms = 1, .output_norms = {"norm1b", "norm2b"}, .dense = FF_GATED, .act = CMLB200_ACT_GELU_TANH},
    {.architecture = "Situlorn",
     .mixers = {{.type = "latent_attention", .form = MIXER_LATENT}, {.type = "latent_attention_2", .form = MIXER_LATENT, .gate = GATE_WIDE}},
     .output_norms = {"norm1", "norm2"}, .dense = FF_POLY_NORM, .act = CMLB200_ACT_CLAMPED, .experts = EXPERTS_PLAIN},
    {.architecture = "Lenedra",
     .mixers = {{.type = "attention", .form = MIXER_GROUPED,
                 .grouped = {.norm = NORM_HEAD, .linear_bias = 1, .in_bias = 1, .out_bias = 1, .keys_as_values = 1}},
                {.type = "parallel", .form = MIXER_PARALLEL, .beside = BESIDE_DELTA, .grouped = {.sink = SINK_LEARNED, .chunked = 1, .in_bias = 1}}},
     .input_norms = 1, .norm_offset = 1.f, .streams = 1, .dense = FF_GATED, .act = CMLB200_ACT_SILU, .experts = EXPERTS_GROUPED},
    {.architecture = "Zevilorn",
     .mixers = {{.type = "attention", .form = MIXER_GROUPED,
                 .grouped = {.sink = SINK_ONE, .in_bias = 1, .out_bias = 1, .rotate = ROTATE_BANDS, .conv = 1, .talk = 1}},
                {.type = "latent_attention", .form = MIXER_LATENT, .gate = GATE_HEAD, .q_latent = 1, .sink = SINK_LEARNED},
                {.type = "parallel", .form = MIXER_PARALLEL, .beside = BESIDE_GRU, .grouped = {.head_gate = 1, .rotate = ROTATE_LINEAR}}},
     .input_norms = 1, .side_by_side = 1, .loops = 1, .act = CMLB200_ACT_GELU_ERF, .experts = EXPERTS_SIGMOID},
};

/* ---- configuration ---------------------------------------------------------------------------------- */
static int is_object(const CMLJson* j) { return j && j->type == CML_JSON_OBJECT; }

static int grouped_columns(const cmlb200_attn* a) { return a->heads * a->dim + a->kv_heads * (a->dim + (a->keys_as_values ? 0 : a->vdim)); }

/* Rotated dimensions and what scales their frequencies: the constants' names in `keys` (the first is a factor). */
static int read_rotation(const CMLJson* mixer, Layer* l, const char* const* keys, int count, int* dims, int index) {
    const CMLJson *rot = cml_json_get(mixer, "rot"), *scaling = cml_json_get(rot, "scaling");
    if (cml_json_double(rot, "base", &l->rot_base) || cml_json_int(rot, "dims", dims) || *dims <= 0 || *dims % 2 || l->rot_base <= 0.0 || l->rot_base == 1.0) {
        LOG_ERROR("layer %d: rot.base or rot.dims is missing or does not fit", index);
        return -1;
    }
    for (int k = 0; is_object(scaling) && k < count; k++)
        if (cml_json_double(scaling, keys[k], &l->rot_scaling[k]) || l->rot_scaling[k] <= 0.0) { LOG_ERROR("layer %d: rot.scaling.%s", index, keys[k]); return -1; }
    return 0;
}

static int read_grouped(const CMLJson* mixer, Layer* l, int index) {
    const GroupedForm* form = &l->kind->grouped;
    const CMLJson *mask = cml_json_get(mixer, "mask"), *temp = cml_json_get(mixer, "q_temp");
    cmlb200_attn* a = &l->attn;
    double scale = 0.0, coef = 0.0, every = 0.0;
    if (cml_json_int(mixer, "heads", &a->heads) || cml_json_int(mixer, "kv_heads", &a->kv_heads) || cml_json_int(mixer, "dim", &a->dim) ||
        cml_json_int(mixer, "vdim", &a->vdim) || cml_json_double(mixer, "scale", &scale) || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads ||
        a->dim <= 0 || a->vdim <= 0 || a->heads > 65535 || a->dim > 256 || a->vdim > 256) {
        LOG_ERROR("layer %d: heads, kv_heads, dim, vdim (up to 256) or scale are missing or do not fit", index);
        return -1;
    }
    int* size = form->chunked ? &a->chunk : &a->window;
    if (is_object(mask) && (cml_json_int(mask, "size", size) || *size <= 0)) { LOG_ERROR("layer %d: mask.size", index); return -1; }
    if (!cml_json_int(mask, "keep_first", &a->keep) && a->keep < 0) { LOG_ERROR("layer %d: mask.keep_first", index); return -1; }
    if (form->keys_as_values && a->dim != a->vdim) { LOG_ERROR("layer %d: values are keys, but vdim %d is not dim %d", index, a->vdim, a->dim); return -1; }
    if (is_object(temp) && (cml_json_double(temp, "coef", &coef) || cml_json_double(temp, "every", &every) || every <= 0.0)) { LOG_ERROR("layer %d: q_temp", index); return -1; }
    a->scale = (float)scale;
    a->temp_coef = (float)coef;
    a->temp_every = (float)every;
    a->dim_ld = lml_round_up(a->dim, 16);
    a->vdim_ld = lml_round_up(a->vdim, 16);
    a->sink = form->sink != SINK_NONE;
    a->keys_as_values = form->keys_as_values;
    a->head_norm = form->norm == NORM_HEAD;
    a->gate_col = form->head_gate ? grouped_columns(a) : -1;
    if (form->rotate != ROTATE_NONE) {
        static const char* const keys[4] = {"factor", "original", "low", "high"};
        if (read_rotation(mixer, l, keys, form->rotate == ROTATE_BANDS ? 4 : 1, &a->rot_dims, index)) return -1;
        if (a->rot_dims > a->dim || (l->rot_scaling[3] > 0.0 && l->rot_scaling[3] <= l->rot_scaling[2])) { LOG_ERROR("layer %d: rot.dims or rot.scaling.high", index); return -1; }
    }
    return form->conv || form->talk ? cml_talk_read(mixer, l, index) : 0;
}

static int read_latent(const CMLJson* mixer, Layer* l, int index) {
    const CMLJson* mask = cml_json_get(mixer, "mask");
    static const char* const keys[4] = {"factor", "original", "fast", "slow"};
    cmlb200_latent* a = &l->lat;
    double scale = 0.0;
    int dims = 0;
    if (cml_json_int(mixer, "heads", &a->heads) || cml_json_int(mixer, "dim", &a->dim) || cml_json_int(mixer, "rot_dim", &a->rot_dim) ||
        cml_json_int(mixer, "vdim", &a->vdim) || cml_json_int(mixer, "kv_rank", &a->rank) || cml_json_double(mixer, "scale", &scale) || a->heads <= 0 ||
        a->heads > 8192 || a->dim <= 0 || a->rot_dim <= 0 || a->rot_dim % 2 || a->dim > 256 || a->rot_dim > 256 || a->dim + a->rot_dim > 384 || a->vdim <= 0 || a->vdim > 256 ||
        a->rank <= 0 || a->rank > 512) {
        LOG_ERROR("layer %d: heads, dim, rot_dim, vdim (up to 256), kv_rank (up to 512) or scale are missing or do not fit", index);
        return -1;
    }
    if (is_object(mask) && (cml_json_int(mask, "size", &a->window) || a->window <= 0)) { LOG_ERROR("layer %d: mask.size", index); return -1; }
    if (read_rotation(mixer, l, keys, 4, &dims, index)) return -1;
    if (dims != a->rot_dim) { LOG_ERROR("layer %d: rot.dims is not rot_dim", index); return -1; }
    if (l->kind->q_latent && (cml_json_int(mixer, "q_rank", &l->q_rank) || l->q_rank <= 0)) { LOG_ERROR("layer %d: q_rank", index); return -1; }
    const CMLJson* from = cml_json_get(mixer, "kv_from");
    if (from && from->type != CML_JSON_NULL && cml_json_int(mixer, "kv_from", &l->kv_from)) { LOG_ERROR("layer %d: kv_from", index); return -1; }
    /* queries out of a latent of their own land in front of the projection, which then begins with that latent */
    l->proj_col = l->kind->q_latent ? lml_round_up(a->heads * (a->dim + a->rot_dim), 16) : 0;
    const int q = l->kind->q_latent ? l->proj_col + l->q_rank : a->heads * (a->dim + a->rot_dim), kv = a->rank + a->rot_dim;
    a->scale = (float)scale;
    a->ld = lml_round_up(kv, 16);
    a->ld_rank = lml_round_up(a->rank, 64);
    a->kv_col = l->kv_from == index ? q : -1;
    a->gate_col = l->kind->gate != GATE_NONE ? q + (l->kv_from == index ? kv : 0) : -1;
    a->gate_heads = l->kind->gate == GATE_HEAD;
    return 0;
}

static int read_parallel(const CMLJson* mixer, Layer* l, int index) {
    if (l->kind->beside == BESIDE_GRU)
        return read_grouped(cml_json_get(mixer, "left"), l, index) || cml_gru_read(cml_json_get(mixer, "right"), l, index) ? -1 : 0;
    double left = 0.0, right = 0.0;
    if (cml_json_double(mixer, "left_scale", &left) || cml_json_double(mixer, "right_scale", &right) || left == 0.0 || right == 0.0) {
        LOG_ERROR("layer %d: left_scale or right_scale is missing or 0", index);
        return -1;
    }
    if (read_grouped(cml_json_get(mixer, "left"), l, index) || cml_delta_read(cml_json_get(mixer, "right"), l, index, grouped_columns(&l->attn))) return -1;
    l->attn.out_scale = (float)left;
    l->delta.out_scale = (float)right;
    return 0;
}

static int read_feed_forward(const CMLJson* mlp, Layer* l, int index, const LayeredDesign* design) {
    const char* kind = cml_json_string(mlp, "kind");
    if (kind && !strcmp(kind, "dense") && !design->side_by_side && !cml_json_int(mlp, "ff", &l->ff) && l->ff > 0) return 0;
    const CMLJson *expert = cml_json_get(mlp, "expert"), *router = cml_json_get(mlp, "router"), *groups = cml_json_get(router, "groups");
    const CMLJson* shared = cml_json_get(mlp, "shared");
    double limit = 0.0, scale = 1.0;
    if (design->experts == EXPERTS_NONE || !kind || strcmp(kind, "moe") || cml_json_int(expert, "ff", &l->ff) || l->ff <= 0 ||
        (design->act == CMLB200_ACT_CLAMPED && cml_json_double(expert, "limit", &limit)) || cml_json_int(router, "experts", &l->experts) ||
        cml_json_int(router, "top", &l->top) || l->experts <= 0 || l->experts > 1024 || l->top <= 0) {
        LOG_ERROR("layer %d: feed-forward of kind '%s' is not known or incomplete", index, kind ? kind : "(none)");
        return -1;
    }
    l->limit = (float)limit;
    if (design->experts >= EXPERTS_GROUPED) {
        if (design->experts == EXPERTS_GROUPED) {
            cml_json_int(router, "identity", &l->identity);
            cml_json_double(router, "scale", &scale);
        }
        l->router_scale = (float)scale;
        const int all = l->experts + l->identity;
        if (l->identity < 0 || l->identity > 1024 || (is_object(groups) && (cml_json_int(groups, "count", &l->groups) || cml_json_int(groups, "keep", &l->keep) || l->groups <= 0 ||
            all % l->groups || l->keep <= 0 || l->keep > l->groups || (long)l->keep * (all / l->groups) < l->top)) ||
            (design->experts == EXPERTS_GROUPED && is_object(shared) && (cml_json_int(shared, "ff", &l->shared_ff) || l->shared_ff <= 0))) {
            LOG_ERROR("layer %d: router.identity, router.groups or shared.ff does not fit", index);
            return -1;
        }
    }
    if (l->top > l->experts + l->identity) { LOG_ERROR("layer %d: %d of %d experts", index, l->top, l->experts + l->identity); return -1; }
    return 0;
}

/* Columns of a side-by-side layer's projection behind its mixer's own: the sublayers' gates (which the join reads four columns at a
 * time), the gates of heads, the router's logits. */
static void place_gates(Layer* l, int width) {
    const int latent = l->kind->form == MIXER_LATENT;
    int col = !latent ? grouped_columns(&l->attn) : (l->lat.kv_col >= 0 ? l->lat.kv_col + l->lat.rank + l->lat.rot_dim : l->proj_col + l->q_rank);
    if (l->kind->form == MIXER_PARALLEL) {
        l->gru.col = col;
        col += 3 * l->gru.width;
    }
    l->gate_cols = col;
    col += (l->ff ? 2 : 1) * width;
    int* heads = latent ? &l->lat.gate_col : &l->attn.gate_col;
    if (*heads >= 0) {
        *heads = col;
        col += latent ? l->lat.heads : l->attn.heads;
    }
    l->router_col = col;
}

static int read_layer(const CMLJson* j, Layer* l, int index, int width, const LayeredDesign* design) {
    const CMLJson *mixer = cml_json_get(j, "mixer"), *mlp = cml_json_get(j, "mlp");
    const char* type = cml_json_string(j, "type");
    for (size_t k = 0; k < sizeof design->mixers / sizeof design->mixers[0]; k++)
        if (type && design->mixers[k].type && !strcmp(type, design->mixers[k].type)) l->kind = &design->mixers[k];
    if (!l->kind) { LOG_ERROR("layer %d: mixer type '%s' is not known to %s", index, type ? type : "(none)", design->architecture); return -1; }
    l->index = l->kv_from = index;
    if (l->kind->form == MIXER_LATENT ? read_latent(mixer, l, index) : (l->kind->form == MIXER_PARALLEL ? read_parallel(mixer, l, index) : read_grouped(mixer, l, index)))
        return -1;
    if (is_object(mlp) && read_feed_forward(mlp, l, index, design)) return -1;
    if (design->side_by_side) place_gates(l, width);
    l->source = index;
    int of;
    if (!cml_json_int(j, "weights_of", &of)) l->source = of;
    return 0;
}

/* No token sees further back than this, kept first tokens aside; 0: no bound. */
static int window_of(const Layer* l) {
    if (l->kind->form == MIXER_LATENT) return l->lat.window;
    return l->kind->grouped.chunked ? l->attn.chunk : l->attn.window;
}

static int same_shape(const Layer* a, const Layer* b) {
    if (a->kind != b->kind || a->ff != b->ff || a->experts != b->experts || a->identity != b->identity || a->shared_ff != b->shared_ff) return 0;
    if (a->q_rank != b->q_rank || a->gru.width != b->gru.width || a->attn.taps != b->attn.taps) return 0;
    if (a->kind->form == MIXER_PARALLEL && (a->delta.heads != b->delta.heads || a->delta.kv_heads != b->delta.kv_heads || a->delta.dim != b->delta.dim ||
                                            a->delta.vdim != b->delta.vdim || a->delta.taps != b->delta.taps))
        return 0;
    if (a->kind->form == MIXER_LATENT)
        return a->lat.heads == b->lat.heads && a->lat.dim == b->lat.dim && a->lat.rot_dim == b->lat.rot_dim && a->lat.vdim == b->lat.vdim &&
               a->lat.rank == b->lat.rank && (a->lat.kv_col < 0) == (b->lat.kv_col < 0);
    return a->attn.heads == b->attn.heads && a->attn.kv_heads == b->attn.kv_heads && a->attn.dim == b->attn.dim && a->attn.vdim == b->attn.vdim;
}

/* A layer that reads another one's cache: an earlier one, which fills its own, with the same latents and rotation. */
static int check_kv_from(const Layered* m, int i) {
    const Layer* l = &m->layers[i];
    if (l->kind->form != MIXER_LATENT || l->kv_from == i) return 0;
    const Layer* f = l->kv_from >= 0 && l->kv_from < i ? &m->layers[l->kv_from] : NULL;
    if (f && f->kind->form == MIXER_LATENT && f->kv_from == l->kv_from && f->lat.rank == l->lat.rank && f->lat.rot_dim == l->lat.rot_dim && f->rot_base == l->rot_base &&
        !memcmp(f->rot_scaling, l->rot_scaling, sizeof l->rot_scaling))
        return 0;
    LOG_ERROR("layer %d: kv_from does not name an earlier layer with the same latents", i);
    return -1;
}

static int read_config(const CMLJson* c, Layered* m) {
    double eps;
    const CMLJson* layers = cml_json_get(c, "layers");
    if (cml_json_int(c, "vocab", &m->vocab) || cml_json_int(c, "width", &m->width) || m->vocab <= 0 || m->width <= 0 ||
        cml_json_double(cml_json_get(c, "norm"), "eps", &eps) || !layers || layers->type != CML_JSON_ARRAY || layers->count < 1 || layers->count > MAX_LAYERS) {
        LOG_ERROR("config.json: vocab, width, norm.eps or layers are missing or do not fit");
        return -1;
    }
    m->eps = (float)eps;
    if (m->design->streams) {
        double scale = 1.0, cap = 0.0;
        if (cml_json_int(c, "streams", &m->streams) || m->streams < 1 || m->streams > 8) { LOG_ERROR("config.json: streams is missing or not 1 .. 8"); return -1; }
        cml_json_double(cml_json_get(c, "embedding"), "scale", &scale);
        cml_json_double(c, "logit_softcap", &cap);
        m->embed_scale = (float)scale;
        m->cap = (float)cap;
    }
    int start = 0, stop = 0, times = 1;
    const CMLJson* loop = m->design->loops ? cml_json_get(c, "loop") : NULL;
    if (is_object(loop) && (cml_json_int(loop, "start", &start) || cml_json_int(loop, "stop", &stop) || cml_json_int(loop, "times", &times) || start < 0 || stop < start ||
                            stop > layers->count || times < 1 || (long)times * (stop - start) > MAX_LAYERS)) {
        LOG_ERROR("config.json: loop does not fit %d layers", layers->count);
        return -1;
    }
    const int span = stop - start, more = (times - 1) * span;
    m->num_layers = layers->count + more;
    m->layers = (Layer*)calloc((size_t)m->num_layers, sizeof(Layer));
    if (!m->layers) return -1;
    int i = 0;
    for (const CMLJson* j = layers->child; j; j = j->next, i++) {
        Layer* l = &m->layers[i < stop ? i : i + more];
        if (read_layer(j, l, i, m->width, m->design)) return -1;
        /* from the places in config.json to the first passes over them */
        if (l->source >= stop) l->source += more;
        if (l->kv_from >= stop) l->kv_from += more;
    }
    for (i = stop; i < stop + more; i++) {                 /* further passes */
        m->layers[i] = m->layers[i - span];
        m->layers[i].again = m->layers[i].index == start;
        m->layers[i].source = start + (i - start) % span;
        if (m->layers[i].kv_from == i - span) m->layers[i].kv_from = i;
    }
    for (i = 0; i < m->num_layers; i++) {                  /* follow chains of weights_of to the layer that has tensors */
        int s = m->layers[i].source, hops = 0;
        while (s >= 0 && s < m->num_layers && m->layers[s].source != s && hops++ < m->num_layers) s = m->layers[s].source;
        if (s < 0 || s >= m->num_layers || hops > m->num_layers || !same_shape(&m->layers[i], &m->layers[s])) { LOG_ERROR("layer %d: weights_of does not lead to a layer of its shape", i); return -1; }
        m->layers[i].source = s;
        if (check_kv_from(m, i)) return -1;
    }
    return 0;
}

/* ---- weights ------------------------------------------------------------------------------------------ */
static float bits_f32(uint32_t u) {
    float f;
    memcpy(&f, &u, sizeof f);
    return f;
}
float lml_element(const CMLSafetensor* t, size_t i) {
    uint16_t h;
    float f;
    if (t->dtype == DTYPE_FLOAT32) { memcpy(&f, (const uint8_t*)t->data + 4 * i, 4); return f; }
    memcpy(&h, (const uint8_t*)t->data + 2 * i, 2);
    return t->dtype == DTYPE_FLOAT16 ? cml_f16_to_f32(h) : bits_f32((uint32_t)h << 16);
}
static uint16_t to_bf16(float f) {
    uint32_t u;
    memcpy(&u, &f, sizeof u);
    if ((u & 0x7FFFFFFFu) > 0x7F800000u) return (uint16_t)((u >> 16) | 64);
    return (uint16_t)((u + 0x7FFFu + ((u >> 16) & 1)) >> 16);
}

int lml_find(const CMLSafetensors* st, const char* prefix, const char* name, int rows, int cols, CMLSafetensor* t) {
    char full[160];
    snprintf(full, sizeof full, "%s%s", prefix, name);
    if (cml_safetensors_find(st, full, t)) { LOG_ERROR("tensor '%s' is missing", full); return -1; }
    if (t->dtype == DTYPE_INT32 || t->ndim != (cols ? 2 : 1) || (rows < 0 ? t->shape[0] < 1 || t->shape[0] > 65536 : t->shape[0] != rows) || (cols && t->shape[1] != cols)) {
        LOG_ERROR("tensor '%s' has another shape or type than config.json says ([%d, %d] expected)", full, rows, cols);
        return -1;
    }
    return 0;
}

int lml_upload(void** dst, const void* src, size_t bytes) {
    if (CML_DEV_FAIL(cmlb200_malloc(dst, bytes), "upload") || CML_DEV_FAIL(cmlb200_memcpy_h2d(*dst, src, bytes, NULL), "upload") ||
        CML_DEV_FAIL(cmlb200_stream_sync(NULL), "upload"))
        return -1;
    return 0;
}

/* Frequencies of the rotated pairs of grouped heads: all divided by a factor, or by where 2 pi / f lies between two shares of
 * `original`: short wavelengths stay, long ones are stretched by the factor, a ramp in original / wavelength lies between. */
static double grouped_frequency(const Layer* l, double f) {
    const double *s = l->rot_scaling, turns = s[1] * f / 6.283185307179586476925;
    if (s[0] <= 0.0) return f;
    if (l->kind->grouped.rotate == ROTATE_LINEAR) return f / s[0];
    const double keep = fmin(fmax((turns - s[2]) / (s[3] - s[2]), 0.0), 1.0);
    return keep < 1.0 ? (1.0 - keep) * f / s[0] + keep * f : f;
}

/* Frequencies of the rotated pairs, for latents with the factor on sine and cosine. With scaling, the pairs of a latent layer
 * that turn fewer than `slow` times within `original` positions are slowed down by the factor, those that turn more than
 * `fast` times are not, and a ramp over the pairs lies between. */
static int make_rotation(Layer* l) {
    const int latent = l->kind->form == MIXER_LATENT, dims = latent ? l->lat.rot_dim : l->attn.rot_dims;
    if (!dims) return 0;
    const double n = dims, *s = l->rot_scaling;
    float* f = (float*)malloc((size_t)(dims / 2) * sizeof(float));
    if (!f) return -1;
    double lo = 0.0, hi = 0.0;
    if (latent && s[0] > 0.0) {
        const double two_pi = 6.283185307179586476925;
        lo = fmax(floor(n * log(s[1] / (two_pi * s[2])) / (2.0 * log(l->rot_base))), 0.0);
        hi = fmin(ceil(n * log(s[1] / (two_pi * s[3])) / (2.0 * log(l->rot_base))), n - 1.0);
    }
    for (int i = 0; i < dims / 2; i++) {
        const double plain = pow(l->rot_base, -2.0 * i / n);
        const double ramp = latent && s[0] > 0.0 ? fmin(fmax((i - lo) / fmax(hi - lo, 0.001), 0.0), 1.0) : 0.0;
        f[i] = (float)(latent ? (ramp > 0.0 ? plain / s[0] * ramp + plain * (1.0 - ramp) : plain) : grouped_frequency(l, plain));
    }
    const int rc = lml_upload((void**)&l->freq, f, (size_t)(dims / 2) * sizeof(float));
    free(f);
    l->attn.freq = l->lat.freq = l->freq;
    l->lat.rot_mul = latent && s[0] > 0.0 ? (float)(0.1 * log(s[0]) + 1.0) : 1.0f;
    return rc;
}

int lml_load_vector(const CMLSafetensors* st, const char* prefix, const char* name, int n, float offset, float** dst) {
    CMLSafetensor t;
    if (lml_find(st, prefix, name, n, 0, &t)) return -1;
    float* v = (float*)malloc((size_t)n * sizeof(float));
    if (!v) return -1;
    for (int i = 0; i < n; i++) v[i] = lml_element(&t, (size_t)i) + offset;
    const int rc = lml_upload((void**)dst, v, (size_t)n * sizeof(float));
    free(v);
    return rc;
}

int lml_load_taps(const CMLSafetensors* st, const char* prefix, const char* const* names, const int* channels, int parts, int taps, float** dst) {
    int all = 0, at = 0, rc = 0;
    for (int p = 0; p < parts; p++) all += channels[p];
    float* v = (float*)malloc((size_t)all * (size_t)taps * sizeof(float));
    if (!v) return -1;
    for (int p = 0; p < parts && !rc; at += channels[p++]) {
        CMLSafetensor t;
        rc = lml_find(st, prefix, names[p], channels[p], taps, &t);
        for (int c = 0; c < channels[p] && !rc; c++)
            for (int k = 0; k < taps; k++) v[(size_t)k * (size_t)all + (size_t)(at + c)] = lml_element(&t, (size_t)c * (size_t)taps + (size_t)k);
    }
    rc = rc || lml_upload((void**)dst, v, (size_t)all * (size_t)taps * sizeof(float));
    free(v);
    return rc ? -1 : 0;
}

static void put_row(const Layered* m, uint8_t* dst, const CMLSafetensor* t, int row, int cols) {
    const size_t at = (size_t)row * (size_t)cols;
    if (!m->f32 && t->dtype == DTYPE_BFLOAT16) memcpy(dst, (const uint8_t*)t->data + 2 * at, (size_t)cols * 2);
    else if (m->f32) for (int c = 0; c < cols; c++) ((float*)(void*)dst)[c] = lml_element(t, at + (size_t)c);
    else for (int c = 0; c < cols; c++) ((uint16_t*)(void*)dst)[c] = to_bf16(lml_element(t, at + (size_t)c));
}

int lml_load_matrix(const Layered* m, const CMLSafetensors* st, const char* prefix, const char* const* names, const int* rows, int parts, int cols,
                       int interleave, cmlb200_dense* out) {
    int total = 0;
    CMLSafetensor t[MAX_PARTS];
    for (int p = 0; p < parts; p++) {
        if (lml_find(st, prefix, names[p], rows[p], cols, &t[p])) return -1;
        total += interleave ? lml_round_up(rows[p], 16) : rows[p];
    }
    const size_t es = m->f32 ? 4 : 2, ld = (size_t)lml_round_up(cols, 64), bytes = (size_t)lml_round_up(total, 16) * ld * es;
    uint8_t* host = (uint8_t*)calloc(bytes, 1);
    if (!host) { LOG_ERROR("out of memory for '%s%s'", prefix, names[0]); return -1; }
    int at = 0;
    for (int p = 0; p < parts; p++) {
        for (int r = 0; r < rows[p]; r++) {
            const int to = interleave ? (r / 16) * 16 * parts + p * 16 + r % 16 : at + r;
            put_row(m, host + (size_t)to * ld * es, &t[p], r, cols);
        }
        at += rows[p];
    }
    out->dtype = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    out->rows = total;
    out->cols = cols;
    out->ld = (int)ld;
    const int rc = lml_upload(&out->w, host, bytes);
    free(host);
    return rc;
}

static int alloc_matrix(const Layered* m, int rows, int cols, cmlb200_dense* out, uint8_t** host) {
    out->dtype = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    out->rows = rows;
    out->cols = cols;
    out->ld = lml_round_up(cols, 64);
    *host = (uint8_t*)calloc((size_t)lml_round_up(rows, 16) * (size_t)out->ld, m->f32 ? 4 : 2);
    if (!*host) LOG_ERROR("out of memory for a [%d, %d] weight", rows, cols);
    return *host ? 0 : -1;
}
static int upload_matrix(const Layered* m, cmlb200_dense* w, uint8_t* host) {
    const int rc = lml_upload(&w->w, host, (size_t)lml_round_up(w->rows, 16) * (size_t)w->ld * (m->f32 ? 4 : 2));
    free(host);
    return rc;
}

/* The experts' gate and up rows (interleaved as in load_matrix), or their up rows alone, and their down rows, one expert behind
 * the other. */
static int load_experts(Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l) {
    LayerWeights* w = &l->w;
    const int gated = m->design->experts != EXPERTS_SIGMOID, gu = (gated ? 2 : 1) * lml_round_up(l->ff, 16), down = lml_round_up(m->width, 16);
    const size_t es = m->f32 ? 4 : 2;
    const char* router[1] = {"mlp.router"};
    uint8_t *hg, *hd;
    const int outputs = l->experts + l->identity;
    if ((!m->design->side_by_side && lml_load_matrix(m, st, prefix, router, &outputs, 1, m->width, 0, &w->router)) || alloc_matrix(m, l->experts * gu, m->width, &w->experts_gu, &hg)) return -1;
    if (alloc_matrix(m, l->experts * down, l->ff, &w->experts_down, &hd)) { free(hg); return -1; }
    int rc = 0;
    for (int e = 0; e < l->experts && !rc; e++) {
        char name[3][48];
        CMLSafetensor t[3];
        snprintf(name[0], sizeof name[0], "mlp.e%d.gate", e);
        snprintf(name[1], sizeof name[1], "mlp.e%d.up", e);
        snprintf(name[2], sizeof name[2], "mlp.e%d.down", e);
        rc = (gated && lml_find(st, prefix, name[0], l->ff, m->width, &t[0])) || lml_find(st, prefix, name[1], l->ff, m->width, &t[1]) || lml_find(st, prefix, name[2], m->width, l->ff, &t[2]);
        for (int p = gated ? 0 : 1; p < 2 && !rc; p++)
            for (int r = 0; r < l->ff; r++) {
                const size_t at = gated ? (size_t)(r / 16) * 32 + (size_t)(p * 16 + r % 16) : (size_t)r;
                put_row(m, hg + ((size_t)e * gu + at) * (size_t)w->experts_gu.ld * es, &t[p], r, m->width);
            }
        for (int r = 0; r < m->width && !rc; r++) put_row(m, hd + ((size_t)e * down + (size_t)r) * (size_t)w->experts_down.ld * es, &t[2], r, l->ff);
    }
    if (rc) { free(hg); free(hd); return -1; }
    rc = upload_matrix(m, &w->experts_gu, hg);
    if (upload_matrix(m, &w->experts_down, hd) || rc) return -1;
    if (m->design->experts != EXPERTS_GROUPED) return 0;
    const char *gate_up[2] = {"mlp.shared.gate", "mlp.shared.up"}, *shared_down[1] = {"mlp.shared.down"};
    const int rows[2] = {l->shared_ff, l->shared_ff};
    return lml_load_vector(st, prefix, "mlp.correction", outputs, 0.f, &w->correction) ||
           (l->shared_ff && (lml_load_matrix(m, st, prefix, gate_up, rows, 2, m->width, 1, &w->shared_gu) ||
                             lml_load_matrix(m, st, prefix, shared_down, &m->width, 1, l->shared_ff, 0, &w->shared_down))) ? -1 : 0;
}

/* Wuk and Wuv in the forms of the two ways a latent layer attends, or of the 32-bit one. */
static int load_latent_heads(const Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l) {
    const cmlb200_latent* a = &l->lat;
    LayerWeights* w = &l->w;
    CMLSafetensor uk, uv;
    const int H = a->heads, D = a->dim, V = a->vdim, R = a->rank;
    if (lml_find(st, prefix, "mix.uk", H * D, R, &uk) || lml_find(st, prefix, "mix.uv", H * V, R, &uv)) return -1;
    const int rp = m->f32 ? R : lml_round_up(R, 16), dp = m->f32 ? D : lml_round_up(D, 64);
    const size_t es = m->f32 ? 4 : 2, bytes = (size_t)H * (size_t)rp * (size_t)dp * es;
    uint8_t* t = (uint8_t*)calloc(bytes, 1);
    if (!t) { LOG_ERROR("out of memory for '%smix.uk'", prefix); return -1; }
    for (int h = 0; h < H; h++)
        for (int d = 0; d < D; d++)
            for (int r = 0; r < R; r++) {
                const size_t to = ((size_t)h * (size_t)rp + (size_t)r) * (size_t)dp + (size_t)d;
                const float v = lml_element(&uk, (size_t)(h * D + d) * (size_t)R + (size_t)r);
                if (m->f32) ((float*)(void*)t)[to] = v;
                else ((uint16_t*)(void*)t)[to] = to_bf16(v);
            }
    int rc = lml_upload(&w->wukt, t, bytes);
    free(t);
    if (rc) return -1;
    if (m->f32) {
        float* v = (float*)malloc((size_t)H * (size_t)V * (size_t)R * sizeof(float));
        if (!v) return -1;
        for (int r = 0; r < H * V; r++) put_row(m, (uint8_t*)(v + (size_t)r * (size_t)R), &uv, r, R);
        rc = lml_upload(&w->wukv.w, v, (size_t)H * (size_t)V * (size_t)R * sizeof(float));
        free(v);
        return rc;
    }
    const int vp = lml_round_up(V, 16);
    uint8_t* host;
    if (alloc_matrix(m, H * (D + vp), R, &w->wukv, &host)) return -1;
    const size_t row = (size_t)w->wukv.ld * es;
    for (int r = 0; r < H * D; r++) put_row(m, host + (size_t)r * row, &uk, r, R);
    for (int r = 0; r < H * V; r++) put_row(m, host + (size_t)(H * D + r / V * vp + r % V) * row, &uv, r, R);
    return upload_matrix(m, &w->wukv, host);
}

static const uint16_t* value_rows(const Layer* l, const LayerWeights* w) {
    return (const uint16_t*)w->wukv.w + (size_t)(l->lat.heads * l->lat.dim) * (size_t)w->wukv.ld;
}

/* A bias of the stacked projections: the tensors' where they have one (bit p of with_bias), else zero. */
static int load_bias(const CMLSafetensors* st, const char* prefix, const char* const* names, const int* rows, int parts, unsigned with_bias, cmlb200_dense* w) {
    if (!with_bias) return 0;
    float* v = (float*)calloc((size_t)w->rows, sizeof(float));
    int rc = v ? 0 : -1;
    for (int p = 0, at = 0; p < parts && !rc; at += rows[p++]) {
        char name[64];
        CMLSafetensor t;
        if (!(with_bias >> p & 1)) continue;
        snprintf(name, sizeof name, "%s.b", names[p]);
        rc = lml_find(st, prefix, name, rows[p], 0, &t);
        for (int i = 0; i < rows[p] && !rc; i++) v[at + i] = lml_element(&t, (size_t)i);
    }
    rc = rc || lml_upload((void**)&w->bias, v, (size_t)w->rows * sizeof(float));
    free(v);
    return rc ? -1 : 0;
}

/* Tensors whose rows make one matrix, with their names' room. */
typedef struct Parts {
    char names[MAX_PARTS][32];
    const char* list[MAX_PARTS];
    int rows[MAX_PARTS], count, total;
    unsigned with_bias;
} Parts;

static void add_part(Parts* p, const char* where, const char* name, int rows, int bias) {
    snprintf(p->names[p->count], sizeof p->names[p->count], "%s%s", where, name);
    p->list[p->count] = p->names[p->count];
    p->with_bias |= (unsigned)(bias != 0) << p->count;
    p->rows[p->count++] = rows;
    p->total += rows;
}

/* The rest of a layer's projection, and the matrix: gates of sublayers side by side and the router read the same row. */
static int load_projection(const Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l, Parts* p) {
    const int latent = l->kind->form == MIXER_LATENT;
    if (m->design->side_by_side) {                         /* in the order of place_gates */
        add_part(p, "", "rg1", m->width, 1);
        if (l->ff) add_part(p, "", "rg2", m->width, 1);
        if ((latent ? l->lat.gate_col : l->attn.gate_col) >= 0) add_part(p, l->kind->form == MIXER_PARALLEL ? "mix.left." : "mix.", "g", latent ? l->lat.heads : l->attn.heads, 0);
        if (l->ff) add_part(p, "mlp.", "router", l->experts, 0);
    }
    return lml_load_matrix(m, st, prefix, p->list, p->rows, p->count, m->width, 0, &l->w.wqkvg) || load_bias(st, prefix, p->list, p->rows, p->count, p->with_bias, &l->w.wqkvg) ? -1 : 0;
}

/* Output matrices of two mixers side by side: [width, left | right]. */
static int load_outputs(const Layered* m, const CMLSafetensors* st, const char* prefix, int left, int right, cmlb200_dense* out) {
    CMLSafetensor l, r;
    uint8_t* host;
    if (lml_find(st, prefix, "mix.left.o", m->width, left, &l) || lml_find(st, prefix, "mix.right.o", m->width, right, &r) ||
        alloc_matrix(m, m->width, left + right, out, &host))
        return -1;
    const size_t es = m->f32 ? 4 : 2;
    for (int i = 0; i < m->width; i++) {
        uint8_t* row = host + (size_t)i * (size_t)out->ld * es;
        put_row(m, row, &l, i, left);
        put_row(m, row + (size_t)left * es, &r, i, right);
    }
    return upload_matrix(m, out, host);
}

/* Grouped heads, alone or with a recurrence beside them. */
static int load_grouped(Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l) {
    const GroupedForm* form = &l->kind->grouped;
    const cmlb200_attn* a = &l->attn;
    const cmlb200_delta* d = &l->delta;
    LayerWeights* w = &l->w;
    const int both = l->kind->form == MIXER_PARALLEL, delta = both && l->kind->beside == BESIDE_DELTA, gru = both && !delta;
    const char* at = both ? "mix.left." : "mix.";
    char group[64];
    Parts p = {.count = 0};
    add_part(&p, at, "q", a->heads * a->dim, form->in_bias);
    add_part(&p, at, "k", a->kv_heads * a->dim, form->in_bias);
    if (!form->keys_as_values) add_part(&p, at, "v", a->kv_heads * a->vdim, form->in_bias);
    if (form->head_gate && !m->design->side_by_side) add_part(&p, at, "g", a->heads, 0);
    if (delta) {
        if (cml_delta_ranks(st, prefix, l, m->width)) return -1;
        add_part(&p, "mix.right.", "q", d->kv_heads * d->dim, 0);
        add_part(&p, "mix.right.", "k", d->kv_heads * d->dim, 0);
        add_part(&p, "mix.right.", "v", d->heads * d->vdim, 0);
        add_part(&p, "mix.right.", "b", d->heads, 0);
        add_part(&p, "mix.right.", "a1", l->a_rank, 0);
        add_part(&p, "mix.right.", "g1", l->g_rank, 0);
    }
    if (gru) {
        add_part(&p, "mix.right.", "z", l->gru.width, 1);
        add_part(&p, "mix.right.", "x", l->gru.width, 1);
        add_part(&p, "mix.right.", "g", l->gru.width, 0);
    }
    snprintf(group, sizeof group, "%s%s", prefix, at);
    const int norm_q = form->norm == NORM_HEAD ? a->dim : p.rows[0], norm_k = form->norm == NORM_HEAD ? a->dim : p.rows[1];
    const char *out[1] = {"o"}, *right[1] = {"mix.right.o"};
    if ((form->norm != NORM_NONE && (lml_load_vector(st, group, "q.norm", norm_q, 0.f, &w->q_norm) || lml_load_vector(st, group, "k.norm", norm_k, 0.f, &w->k_norm))) ||
        (form->sink == SINK_LEARNED && lml_load_vector(st, group, "sink", a->heads, 0.f, &w->sinks)) || load_projection(m, st, prefix, l, &p) ||
        (delta ? load_outputs(m, st, prefix, a->heads * a->vdim, d->heads * d->vdim, &w->wo)
               : lml_load_matrix(m, st, group, out, &m->width, 1, a->heads * a->vdim, 0, &w->wo)) ||
        (form->out_bias && load_bias(st, group, out, &m->width, 1, 1, &w->wo)) || (delta && cml_delta_load(m, st, prefix, l)) ||
        (gru && (lml_load_matrix(m, st, prefix, right, &m->width, 1, l->gru.width, 0, &w->wo2) || lml_load_vector(st, prefix, "mix.left.out", m->width, 0.f, &w->left_out) ||
                 lml_load_vector(st, prefix, "mix.right.out", m->width, 0.f, &w->right_out))) ||
        ((form->conv || form->talk) && cml_talk_load(st, group, l)))
        return -1;
    if (!form->linear_bias) return 0;
    float* s = (float*)malloc((size_t)a->heads * sizeof(float));
    if (!s) return -1;
    for (int h = 0; h < a->heads; h++) s[h] = (float)exp2(-8.0 * (h + 1) / a->heads);
    const int rc = lml_upload((void**)&w->slopes, s, (size_t)a->heads * sizeof(float));
    free(s);
    return rc;
}

static int load_mixer(Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l) {
    LayerWeights* w = &l->w;
    const char* out[1] = {"mix.o"};
    const int out_rows[1] = {m->width};
    if (l->kind->form == MIXER_LATENT) {
        const cmlb200_latent* a = &l->lat;
        const int q[1] = {a->heads * (a->dim + a->rot_dim)};
        const char* uq[1] = {"mix.uq"};
        Parts p = {.count = 0};
        if (l->kind->q_latent) add_part(&p, "mix.", "dq", l->q_rank, 0);
        else add_part(&p, "mix.", "q", q[0], 0);
        if (a->kv_col >= 0) add_part(&p, "mix.", "dkv", a->rank + a->rot_dim, 0);
        if (a->gate_col >= 0 && !m->design->side_by_side) add_part(&p, "mix.", "g", a->heads * (a->gate_heads ? 1 : a->vdim), 0);
        if (l->kind->q_latent && (lml_load_vector(st, prefix, "mix.dq.norm", l->q_rank, 0.f, &w->dq_norm) || lml_load_matrix(m, st, prefix, uq, q, 1, l->q_rank, 0, &w->wuq)))
            return -1;
        return (a->kv_col >= 0 && lml_load_vector(st, prefix, "mix.dkv.norm", a->rank, 0.f, &w->c_norm)) || load_projection(m, st, prefix, l, &p) ||
               (l->kind->sink == SINK_LEARNED && lml_load_vector(st, prefix, "mix.sink", a->heads, 0.f, &w->sinks)) || load_latent_heads(m, st, prefix, l) ||
               lml_load_matrix(m, st, prefix, out, out_rows, 1, a->heads * a->vdim, 0, &w->wo) ? -1 : 0;
    }
    return load_grouped(m, st, prefix, l);
}

static int load_sublayer(const Layered* m, const CMLSafetensors* st, const char* prefix, int which, LayerWeights* w) {
    const LayeredDesign* d = m->design;
    Sublayer* s = &w->sub[which];
    char name[4][16];
    snprintf(name[0], sizeof name[0], "norm%d", which + 1);
    snprintf(name[1], sizeof name[1], "hc%d.in", which + 1);
    snprintf(name[2], sizeof name[2], "hc%d.out", which + 1);
    snprintf(name[3], sizeof name[3], "hc%d.mix", which + 1);
    if ((d->input_norms && lml_load_vector(st, prefix, name[0], m->width, d->norm_offset, &s->norm)) ||
        (d->output_norms[which] && lml_load_vector(st, prefix, d->output_norms[which], m->width, d->norm_offset, &s->post)))
        return -1;
    if (!m->streams) return 0;
    CMLSafetensor t;
    if (lml_load_vector(st, prefix, name[1], m->streams, 0.f, &s->in) || lml_load_vector(st, prefix, name[2], m->streams, 0.f, &s->out) ||
        lml_find(st, prefix, name[3], m->streams, m->streams, &t))
        return -1;
    float mix[64];
    for (int i = 0; i < m->streams * m->streams; i++) mix[i] = lml_element(&t, (size_t)i);
    return lml_upload((void**)&s->mix, mix, (size_t)(m->streams * m->streams) * sizeof(float));
}

static int load_layer(Layered* m, const CMLSafetensors* st, int run) {
    Layer* l = &m->layers[run];
    LayerWeights* w = &l->w;
    const LayeredDesign* d = m->design;
    char prefix[32];
    snprintf(prefix, sizeof prefix, "l%d.", l->index);
    const char *gu[2] = {"mlp.gate", "mlp.up"}, *up[1] = {"mlp.up"}, *down[1] = {"mlp.down"};
    const int ff_rows[2] = {l->ff, l->ff};
    if (load_sublayer(m, st, prefix, 0, w) || load_mixer(m, st, prefix, l)) return -1;
    if (!l->ff) return 0;
    if (!d->side_by_side && load_sublayer(m, st, prefix, 1, w)) return -1;
    if (l->experts) return load_experts(m, st, prefix, l);
    if (d->dense == FF_POLY_NORM ? lml_load_matrix(m, st, prefix, up, ff_rows, 1, m->width, 0, &w->wgu) || lml_load_vector(st, prefix, "mlp.act", 4, 0.f, &w->coef)
                                 : lml_load_matrix(m, st, prefix, gu, ff_rows, 2, m->width, 1, &w->wgu))
        return -1;
    return lml_load_matrix(m, st, prefix, down, &m->width, 1, l->ff, 0, &w->wd);
}

static int load_shared(Layered* m, const CMLSafetensors* st) {
    CMLSafetensor t;
    const char* head[1] = {"head"};
    const int head_rows[1] = {m->vocab};
    if (lml_find(st, "", "embed", m->vocab, m->width, &t)) return -1;
    const size_t row = (size_t)m->width * (m->f32 ? 4 : 2);
    uint8_t* e = (uint8_t*)malloc((size_t)m->vocab * row);
    float* fr = (float*)malloc((size_t)(m->width / 2 + 1) * sizeof(float));
    int rc = e && fr ? 0 : -1;
    for (int i = 0; i < m->vocab && !rc; i++) put_row(m, e + (size_t)i * row, &t, i, m->width);
    rc = rc || lml_upload(&m->embed, e, (size_t)m->vocab * row);
    if (!rc && m->design->position_base > 0.0) {
        for (int i = 0; i <= m->width / 2; i++) fr[i] = (float)pow(m->design->position_base, -2.0 * i / m->width);
        rc = lml_upload((void**)&m->freq, fr, (size_t)(m->width / 2 + 1) * sizeof(float));
    }
    free(e);
    free(fr);
    rc = rc || lml_load_vector(st, "", "final.norm", m->width, m->design->norm_offset, &m->final_norm) || lml_load_matrix(m, st, "", head, head_rows, 1, m->width, 0, &m->head);
    m->head.cap = m->cap;
    return rc ? -1 : 0;
}

/* ---- activations and caches --------------------------------------------------------------------------- */
int lml_zeroed(void** dst, size_t bytes) {
    DEV(cmlb200_malloc(dst, bytes));
    DEV(cmlb200_memset(*dst, 0, bytes, NULL));
    return 0;
}

/* Where a second mixer with an output product of its own leaves its operand: a product reads whole groups of 64 columns. */
static int beside_col(const Layer* l) { return lml_round_up(l->attn.heads * l->attn.vdim, 64); }

/* Operand buffers have strides that are multiples of 64 and start out zero: the decode product reads up
 * to the padded width, where its weights are zero. */
static int make_activations(Layered* m, int rows) {
    int q = 0, att = 0, ff = 0, z = 0, latent_q = 0, latent_o = 0, cq = 0, two = 0, experts = 0, identity = 0, outputs = 0, top = 0, shared = 0;
    long positions = 0, tiles = 0;
    for (int i = 0; i < m->num_layers; i++) {
        const Layer* l = &m->layers[i];
        q = lml_most(q, l->proj_col + m->layers[l->source].w.wqkvg.rows);
        cq = lml_most(cq, l->q_rank);
        ff = lml_most(ff, l->ff);
        if (l->kind->form == MIXER_LATENT) {
            const cmlb200_latent* a = &l->lat;
            att = lml_most(att, a->heads * a->vdim);
            latent_q = lml_most(latent_q, a->heads * (m->f32 ? a->rank + a->rot_dim : a->ld));
            latent_o = lml_most(latent_o, a->heads * (m->f32 ? a->rank : a->ld_rank));
        } else if (l->kind->form == MIXER_PARALLEL && l->kind->beside == BESIDE_GRU) {
            att = lml_most(att, beside_col(l) + l->gru.width);
            two = 1;
        } else {
            att = lml_most(att, l->attn.heads * l->attn.vdim + (l->kind->form == MIXER_PARALLEL ? l->delta.heads * l->delta.vdim : 0));
        }
        if (l->experts) {
            const long p = cmlb200_moe_positions(rows, l->top, l->experts, EXPERT_ROWS);
            if (p > positions) positions = p;
            if (p / EXPERT_ROWS + l->experts + 1 > tiles) tiles = p / EXPERT_ROWS + l->experts + 1;
            experts = lml_most(experts, l->experts);
            identity = lml_most(identity, l->identity);
            outputs = lml_most(outputs, l->experts + l->identity);
            shared = lml_most(shared, l->shared_ff);
            top = lml_most(top, l->top);
        } else if (l->ff) {
            z = lml_most(z, m->design->dense == FF_POLY_NORM ? l->ff : (m->f32 ? 2 * lml_round_up(l->ff, 16) : 0));
        }
        if (l->experts && m->f32) z = lml_most(z, 2 * lml_round_up(lml_most(l->ff, l->shared_ff), 16));
    }
    ff = lml_most(ff, shared);
    m->max_rows = rows;
    m->ld_h = lml_round_up(m->width, 64);
    m->ld_qkvg = lml_round_up(q, 16);
    m->ld_att = lml_round_up(att, 64);
    m->ld_y = lml_round_up(m->width, 16);
    m->ld_f = lml_round_up(ff ? ff : 1, 64);
    m->ld_gu = lml_round_up(z, 16);
    m->ld_router = lml_round_up(outputs, 16);
    const size_t R = (size_t)rows, P = (size_t)(positions > rows ? positions : rows), es = m->f32 ? 4 : 2;
    const size_t head = R > 256 ? R : 256;                 /* the head normalises up to 256 rows at once into h */
    if (lml_zeroed((void**)&m->x, R * (size_t)m->width * (size_t)lml_most(m->streams, 1) * 4) || lml_zeroed(&m->h, head * (size_t)m->ld_h * es) || lml_zeroed((void**)&m->qkvg, R * (size_t)m->ld_qkvg * 4) ||
        lml_zeroed(&m->att, R * (size_t)m->ld_att * es) || lml_zeroed((void**)&m->y, P * (size_t)m->ld_y * 4) || lml_zeroed(&m->f, P * (size_t)m->ld_f * es) ||
        (z && lml_zeroed((void**)&m->gu, (m->f32 ? P : R) * (size_t)m->ld_gu * 4)))
        return -1;
    if (latent_q) {
        const long q_rows = (long)m->max_sequences * 64;
        m->q_rows = q_rows < rows ? (int)q_rows : rows;
        if (lml_zeroed(&m->q, (size_t)m->q_rows * (size_t)latent_q * es) || lml_zeroed(&m->o, (size_t)m->q_rows * (size_t)latent_o * es)) return -1;
    }
    if (experts) {
        cmlb200_moe* p = &m->plan;
        const size_t pairs = R * (size_t)top * 4, pos = P * 4, per = (size_t)experts * 4;
        if (lml_zeroed((void**)&m->router, R * (size_t)m->ld_router * 4) || (!m->f32 && lml_zeroed(&m->xp, P * (size_t)m->ld_h * es)) || lml_zeroed((void**)&p->ids, pairs) ||
            lml_zeroed((void**)&p->weight, pairs) || lml_zeroed((void**)&p->pos, pairs) || lml_zeroed((void**)&p->src, pos) || lml_zeroed((void**)&p->expert, pos) ||
            lml_zeroed((void**)&p->start, per) || lml_zeroed((void**)&p->count, per) || lml_zeroed((void**)&p->active, per) || lml_zeroed((void**)&p->num_active, 4) ||
            lml_zeroed((void**)&p->tiles, (size_t)tiles * 16) || lml_zeroed((void**)&p->num_tiles, 4) || (identity && lml_zeroed((void**)&p->self, R * 4)) ||
            (shared && lml_zeroed((void**)&m->y_shared, R * (size_t)m->ld_y * 4)))
            return -1;
    }
    if (cq) {
        m->ld_cq = lml_round_up(cq, 64);
        if (lml_zeroed(&m->cq, R * (size_t)m->ld_cq * es)) return -1;
    }
    if (m->design->side_by_side && (lml_zeroed((void**)&m->y_mix, R * (size_t)m->ld_y * 4) || (two && lml_zeroed((void**)&m->y_mix2, R * (size_t)m->ld_y * 4)))) return -1;
    if (cml_delta_activations(m, rows)) return -1;
    return CML_DEV_FAIL(cmlb200_stream_sync(NULL), "make_activations") ? -1 : 0;
}

/* The scratch cache of long portions: keys and values per head for as many tokens as a step may expand at a time. */
static int make_expansion(Layered* m, int blocks, int block_size, int slots, int table_ld) {
    int k = 0, v = 0, c = 0;
    for (int i = 0; i < m->num_layers; i++) {
        const cmlb200_latent* a = &m->layers[i].lat;
        if (m->layers[i].kind->form != MIXER_LATENT) continue;
        k = lml_most(k, a->heads * lml_round_up(a->dim + a->rot_dim, 16));
        v = lml_most(v, a->heads * lml_round_up(a->vdim, 16));
        c = lml_most(c, a->ld_rank);
    }
    if (!k || m->f32) return 0;
    m->slots = slots;
    m->table_ld = table_ld;
    const char* env = getenv("CMLB200_EXPAND_KEYS");
    int keys = env && atoi(env) > 0 && atoi(env) < (1 << 28) ? lml_round_up(atoi(env), block_size) : EXPAND_KEYS;
    if ((long)blocks * block_size < keys) keys = blocks * block_size;
    m->expand_keys = keys;
    const size_t n = (size_t)m->expand_keys;
    return lml_zeroed(&m->expand_k, n * (size_t)k * 2) || lml_zeroed(&m->expand_v, n * (size_t)v * 2) || lml_zeroed(&m->expand_c, n * (size_t)c * 2) ||
           lml_zeroed((void**)&m->expand_table, (size_t)slots * (size_t)table_ld * sizeof(int)) ? -1 : 0;
}

static int layered_make_pools(void* model, int blocks, int block_size, int slots, int table_ld) {
    Layered* m = (Layered*)model;
    const size_t es = m->f32 ? 4 : 2, tokens = (size_t)blocks * (size_t)block_size;
    for (int i = 0; i < m->num_layers; i++) {
        Layer* l = &m->layers[i];
        const LayerWeights* w = &m->layers[l->source].w;
        if (l->kind->form == MIXER_LATENT) {
            cmlb200_latent* a = &l->lat;
            a->cache_dtype = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_F16;
            a->block_size = block_size;
            a->pool_blocks = blocks;
            a->c_norm = w->c_norm;
            a->sinks = w->sinks;
            a->eps = m->eps;
            if (l->kv_from != i) a->pool = m->layers[l->kv_from].lat.pool;
            else if (lml_zeroed(&a->pool, tokens * (size_t)a->ld * es)) return -1;
            continue;
        }
        cmlb200_attn* a = &l->attn;
        const size_t heads = tokens * (size_t)a->kv_heads;
        a->cache_dtype = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_F16;
        a->block_size = block_size;
        a->q_norm = w->q_norm;
        a->k_norm = w->k_norm;
        a->eps = m->eps;
        a->slopes = w->slopes;
        a->sinks = w->sinks;
        if (l->kind->form == MIXER_PARALLEL && (l->kind->beside == BESIDE_GRU ? cml_gru_make_state(l, slots) : cml_delta_make_state(m, l, w, slots))) return -1;
        if ((l->kind->grouped.conv || l->kind->grouped.talk) && cml_talk_make_state(l, w, slots)) return -1;
        if (lml_zeroed(&a->k_pool, heads * (size_t)a->dim_ld * es) || lml_zeroed(&a->v_pool, heads * (size_t)a->vdim_ld * es)) return -1;
    }
    if (make_expansion(m, blocks, block_size, slots, table_ld) || cml_talk_make_scores(m, slots, table_ld, block_size)) return -1;
    DEV(cmlb200_stream_sync(NULL));
    return 0;
}

/* ---- a step ------------------------------------------------------------------------------------------- */
int lml_product(const Layered* m, const cmlb200_dense* w, const void* x, int ldx, int rows, float* y, int ldy, void* st) {
    if (m->f32) DEV(cmlb200_linear_dense_f32(w, (const float*)x, ldx, rows, y, ldy, st));
    else if (rows <= SKINNY_ROWS) DEV(cmlb200_gemv_dense(w, (const uint16_t*)x, ldx, rows, y, ldy, st));
    else DEV(cmlb200_gemm_dense(w, (const uint16_t*)x, ldx, rows, y, ldy, st));
    return 0;
}

/* y = Wd (act(gate) * up) of the rows in h */
static int gated_product(const Layered* m, const cmlb200_dense* gu, const cmlb200_dense* down, int ff, int rows, float* y, void* st) {
    const int act = m->design->act;
    if (m->f32) {
        DEV(cmlb200_linear_dense_f32(gu, (const float*)m->h, m->ld_h, rows, m->gu, m->ld_gu, st));
        DEV(cmlb200_glu_rows_f32(m->gu, m->ld_gu, rows, ff, act, (float*)m->f, m->ld_f, st));
    } else if (rows <= SKINNY_ROWS) {
        DEV(cmlb200_gemv_dense_glu(gu, (const uint16_t*)m->h, m->ld_h, rows, ff, act, (uint16_t*)m->f, m->ld_f, st));
    } else {
        DEV(cmlb200_gemm_dense_glu(gu, (const uint16_t*)m->h, m->ld_h, rows, ff, act, (uint16_t*)m->f, m->ld_f, st));
    }
    return lml_product(m, down, m->f, m->ld_f, rows, y, m->ld_y, st);
}

/* Router, plan, the chosen experts' products (and a shared expert's); y then holds a row per (row, expert) pair. */
static int expert_layer(const Layered* m, const Layer* l, const LayerWeights* w, int rows, cmlb200_moe* plan, void* st) {
    const int act = m->design->act;
    *plan = m->plan;
    plan->experts = l->experts;
    plan->top = l->top;
    if (m->design->experts == EXPERTS_GROUPED) {
        plan->identity = l->identity;
        plan->groups = l->groups;
        plan->keep = l->keep;
        plan->correction = w->correction;
        plan->normalize = 1;
        plan->scale = l->router_scale;
        if (l->shared_ff && gated_product(m, &w->shared_gu, &w->shared_down, l->shared_ff, rows, m->y_shared, st)) return -1;
    }
    const int side = m->design->side_by_side, ld_router = side ? m->ld_qkvg : m->ld_router;
    const float* router = side ? m->qkvg + l->router_col : m->router;
    if (!side && lml_product(m, &w->router, m->h, m->ld_h, rows, m->router, m->ld_router, st)) return -1;
    if (m->design->experts == EXPERTS_SIGMOID) {
        plan->sigmoid = 1;
        plan->group_best = 2;
        plan->groups = l->groups;
        plan->keep = l->keep;
    }
    DEV(cmlb200_moe_route(plan, router, ld_router, rows, m->f32 || rows <= SKINNY_ROWS ? 1 : EXPERT_ROWS, st));
    if (m->design->experts == EXPERTS_SIGMOID) {           /* no gate */
        if (m->f32) {
            DEV(cmlb200_moe_linear_f32(plan, &w->experts_gu, (const float*)m->h, m->ld_h, 1, rows, l->ff, m->gu, m->ld_gu, st));
            DEV(cmlb200_act_rows_f32(m->gu, m->ld_gu, rows * l->top, l->ff, act, (float*)m->f, m->ld_f, st));
            DEV(cmlb200_moe_linear_f32(plan, &w->experts_down, (const float*)m->f, m->ld_f, 0, rows, m->width, m->y, m->ld_y, st));
        } else if (rows <= SKINNY_ROWS) {
            DEV(cmlb200_moe_gemv_act(plan, &w->experts_gu, (const uint16_t*)m->h, m->ld_h, 1, rows, l->ff, act, (uint16_t*)m->f, m->ld_f, st));
            DEV(cmlb200_moe_gemv(plan, &w->experts_down, (const uint16_t*)m->f, m->ld_f, 0, rows, m->width, m->y, m->ld_y, st));
        } else {
            DEV(cmlb200_moe_gather(plan, (const uint16_t*)m->h, m->ld_h, rows, m->width, (uint16_t*)m->xp, m->ld_h, st));
            DEV(cmlb200_moe_gemm_act(plan, &w->experts_gu, (const uint16_t*)m->xp, m->ld_h, rows, l->ff, act, (uint16_t*)m->f, m->ld_f, st));
            DEV(cmlb200_moe_gemm(plan, &w->experts_down, (const uint16_t*)m->f, m->ld_f, rows, m->width, m->y, m->ld_y, st));
        }
        return 0;
    }
    if (m->f32) {
        DEV(cmlb200_moe_linear_f32(plan, &w->experts_gu, (const float*)m->h, m->ld_h, 1, rows, 2 * lml_round_up(l->ff, 16), m->gu, m->ld_gu, st));
        DEV(cmlb200_moe_glu_rows_f32(m->gu, m->ld_gu, rows * l->top, l->ff, act, l->limit, (float*)m->f, m->ld_f, st));
        DEV(cmlb200_moe_linear_f32(plan, &w->experts_down, (const float*)m->f, m->ld_f, 0, rows, m->width, m->y, m->ld_y, st));
    } else if (rows <= SKINNY_ROWS) {
        DEV(cmlb200_moe_gemv_glu(plan, &w->experts_gu, (const uint16_t*)m->h, m->ld_h, 1, rows, l->ff, act, l->limit, (uint16_t*)m->f, m->ld_f, st));
        DEV(cmlb200_moe_gemv(plan, &w->experts_down, (const uint16_t*)m->f, m->ld_f, 0, rows, m->width, m->y, m->ld_y, st));
    } else {
        DEV(cmlb200_moe_gather(plan, (const uint16_t*)m->h, m->ld_h, rows, m->width, (uint16_t*)m->xp, m->ld_h, st));
        DEV(cmlb200_moe_gemm_glu(plan, &w->experts_gu, (const uint16_t*)m->xp, m->ld_h, rows, l->ff, act, l->limit, (uint16_t*)m->f, m->ld_f, st));
        DEV(cmlb200_moe_gemm(plan, &w->experts_down, (const uint16_t*)m->f, m->ld_f, rows, m->width, m->y, m->ld_y, st));
    }
    return 0;
}

static int feed_forward(const Layered* m, const Layer* l, const LayerWeights* w, int rows, void* st) {
    if (m->design->dense != FF_POLY_NORM) return gated_product(m, &w->wgu, &w->wd, l->ff, rows, m->y, st);
    if (lml_product(m, &w->wgu, m->h, m->ld_h, rows, m->gu, m->ld_gu, st)) return -1;
    DEV(cmlb200_poly_norm(m->gu, m->ld_gu, rows, l->ff, w->coef, m->eps, m->f, m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16, m->ld_f, st));
    return lml_product(m, &w->wd, m->f, m->ld_f, rows, m->y, m->ld_y, st);
}

/* Rows first .. first + rows - 1 against the latents themselves: queries through Wuk^T, weighted latents through Wuv.
 * one: that many single tokens, then `tiles` tiles from the batch's tile `tile` on, with up to tile_keys keys. */
static int attend_latents(const Layered* m, const cmlb200_latent* a, const Layer* l, const LayerWeights* w, const CMLLMBatch* b, int first, int rows, int one,
                          int tile, int tiles, int tile_keys, void* st) {
    const float* proj = m->qkvg + (size_t)first * (size_t)m->ld_qkvg;
    uint16_t *q = (uint16_t*)m->q, *o = (uint16_t*)m->o;
    DEV(cmlb200_latent_query(a, (const uint16_t*)w->wukt, proj, m->ld_qkvg, b->d_pos + first, b->d_slot + first, rows, q, st));
    if (one) DEV(cmlb200_attention_latent(a, q, rows, b->d_pos + first, b->d_slot + first, one, b->max_keys, NULL, 0, o, st));
    if (tiles) DEV(cmlb200_attention_latent(a, q, rows, NULL, NULL, first, tile_keys, b->d_tiles + 4 * tile, tiles, o, st));
    DEV(cmlb200_latent_output(a, value_rows(l, w), o, proj, m->ld_qkvg, rows, (uint16_t*)m->att + (size_t)first * (size_t)m->ld_att, m->ld_att, st));
    return 0;
}

/* Portions of more than one tile: as many at a time as the scratch cache takes. One whose keys it can not take at all
 * goes over the latents, a few tiles at a time. */
static int attend_expanded(const Layered* m, const cmlb200_latent* a, const Layer* l, const LayerWeights* w, const CMLLMBatch* b, void* st) {
    cmlb200_attn s;
    memset(&s, 0, sizeof s);
    s.heads = s.kv_heads = a->heads;
    s.dim = a->dim + a->rot_dim;
    s.vdim = a->vdim;
    s.dim_ld = lml_round_up(s.dim, 16);
    s.vdim_ld = lml_round_up(s.vdim, 16);
    s.scale = a->scale;
    s.window = a->window;
    s.gate_col = a->gate_col;
    s.gate_wide = a->gate_col >= 0 && !a->gate_heads;
    s.sink = a->sinks != NULL;
    s.sinks = a->sinks;
    s.cache_dtype = CMLB200_DT_F16;
    s.k_pool = m->expand_k;
    s.v_pool = m->expand_v;
    s.block_size = a->block_size;
    s.block_table = m->expand_table;
    s.table_ld = m->table_ld;
    if (b->table_ld != m->table_ld) return -1;
    int i = 0;
    while (i < b->num_portions) {
        int list[16][4], n = 0, keys = 0, rows = 0, tiles = 0;
        const CMLLMPortion* p0 = &b->portions[i];
        for (; i + n < b->num_portions && n < 16; n++) {
            const CMLLMPortion* p = &b->portions[i + n];
            const int lo = (a->window > 0 && a->window <= p->pos ? p->pos - a->window + 1 : 0) / a->block_size * a->block_size, k = p->pos + p->rows - lo;
            if (keys + k > m->expand_keys) break;
            list[n][0] = p->slot;
            list[n][1] = lo;
            list[n][2] = k;
            list[n][3] = keys;
            keys += lml_round_up(k, a->block_size);
            rows += p->rows;
            tiles += (p->rows + 63) / 64;
        }
        if (n) {
            DEV(cmlb200_latent_append(a, m->qkvg + (size_t)p0->row * (size_t)m->ld_qkvg, m->ld_qkvg, b->d_pos + p0->row, b->d_slot + p0->row, rows, st));
            DEV(cmlb200_latent_gather(a, (const int(*)[4])list, n, (uint16_t*)m->expand_c, &s, st));
            DEV(cmlb200_latent_expand(a, &w->wukv, (const uint16_t*)m->expand_c, keys < m->expand_keys ? keys : m->expand_keys, &s, st));
            DEV(cmlb200_attention_tiles(&s, m->qkvg, m->ld_qkvg, b->d_tiles + 4 * p0->tile, tiles, (uint16_t*)m->att, m->ld_att, st));
            i += n;
            continue;
        }
        const int at_once = m->q_rows / 64 * 64;
        for (int r = 0; r < p0->rows; r += at_once) {
            const int k = p0->rows - r < at_once ? p0->rows - r : at_once;
            if (attend_latents(m, a, l, w, b, p0->row + r, k, 0, p0->tile + r / 64, (k + 63) / 64, p0->pos + p0->rows, st)) return -1;
        }
        i++;
    }
    return 0;
}

static int attend_latent(const Layered* m, const Layer* l, const LayerWeights* w, const CMLLMBatch* b, void* st) {
    cmlb200_latent a = l->lat;
    a.block_table = b->d_table;
    a.table_ld = b->table_ld;
    if (m->f32) {                                          /* the latents as one head of keys and values, fp32 */
        cmlb200_attn s;
        memset(&s, 0, sizeof s);
        s.heads = a.heads;
        s.kv_heads = 1;
        s.dim = a.rank + a.rot_dim;
        s.vdim = a.rank;
        s.dim_ld = s.vdim_ld = a.ld;
        s.scale = a.scale;
        s.window = a.window;
        s.gate_col = -1;
        s.sink = a.sinks != NULL;
        s.sinks = a.sinks;
        s.cache_dtype = CMLB200_DT_F32;
        s.k_pool = s.v_pool = a.pool;
        s.block_size = a.block_size;
        s.block_table = a.block_table;
        s.table_ld = a.table_ld;
        for (int r = 0; r < b->rows; r += m->q_rows) {
            const int n = b->rows - r < m->q_rows ? b->rows - r : m->q_rows;
            const float* proj = m->qkvg + (size_t)r * (size_t)m->ld_qkvg;
            DEV(cmlb200_latent_query_f32(&a, (const float*)w->wukt, proj, m->ld_qkvg, b->d_pos + r, b->d_slot + r, n, (float*)m->q, st));
            DEV(cmlb200_attention_rows_f32(&s, (const float*)m->q, a.heads * s.dim, b->d_pos + r, b->d_slot + r, n, (float*)m->o, a.heads * a.rank, st));
            DEV(cmlb200_latent_output_f32(&a, (const float*)w->wukv.w, (const float*)m->o, proj, m->ld_qkvg, n, (float*)m->att + (size_t)r * (size_t)m->ld_att, m->ld_att, st));
        }
        return 0;
    }
    const int near = b->one_rows + b->short_rows;
    if (near && attend_latents(m, &a, l, w, b, 0, near, b->one_rows, 0, b->short_tiles, b->short_keys, st)) return -1;
    return b->num_portions ? attend_expanded(m, &a, l, w, b, st) : 0;
}

static int attend(const Layered* m, const Layer* l, const LayerWeights* w, const CMLLMBatch* b, void* st) {
    if (l->kind->form == MIXER_PARALLEL &&
        (l->kind->beside == BESIDE_GRU ? cml_gru_run(m, l, b, beside_col(l), st) : cml_delta_run(m, l, w, b, l->attn.heads * l->attn.vdim, st)))
        return -1;
    if (l->kind->form == MIXER_LATENT) return attend_latent(m, l, w, b, st);
    cmlb200_attn a = l->attn;
    a.block_table = b->d_table;
    a.table_ld = b->table_ld;
    if (l->kind->grouped.conv || l->kind->grouped.talk) return cml_talk_run(m, &a, b, st);
    if (m->f32) {
        if (a.freq) DEV(cmlb200_rotate_append(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, 0, b->rows, 0, NULL, st));
        else DEV(cmlb200_qk_norm_append(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, b->rows, st));
        DEV(cmlb200_attention_rows_f32(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, b->rows, (float*)m->att, m->ld_att, st));
        return 0;
    }
    const int one = b->one_rows, more = b->rows - one;
    if (more) {
        if (a.freq) DEV(cmlb200_rotate_append(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, one, more, one, NULL, st));
        else DEV(cmlb200_qk_norm_append(&a, m->qkvg + (size_t)one * m->ld_qkvg, m->ld_qkvg, b->d_pos + one, b->d_slot + one, more, st));
        DEV(cmlb200_attention_tiles(&a, m->qkvg, m->ld_qkvg, b->d_tiles, b->tiles, (uint16_t*)m->att, m->ld_att, st));
    }
    if (one) DEV(cmlb200_attention_one(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, one, b->max_keys, (uint16_t*)m->att, m->ld_att, st));
    return 0;
}

/* A sublayer's output joins the residual; `next`: the sublayer that reads it then (NULL: none). parts: y holds a row per pair of that
 * plan. done NULL: the embedding is all there is. */
static int join(const Layered* m, const Sublayer* done, const Sublayer* next, const cmlb200_moe* parts, const float* add, int rows, void* st) {
    const int out = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    const float* y = done ? m->y : NULL;
    const float *post = done ? done->post : NULL, *norm = next ? next->norm : NULL;
    if (m->streams) {
        const cmlb200_streams hc = {m->streams, done ? done->mix : NULL, done ? done->out : NULL, next ? next->in : NULL};
        const cmlb200_join j = {parts, m->h, add, m->ld_y};
        DEV(cmlb200_stream_join(&hc, m->x, y, m->ld_y, done ? &j : NULL, norm, m->eps, rows, m->width, NULL, m->h, out, m->ld_h, st));
    } else if (m->design->input_norms) {
        DEV(cmlb200_residual_norm(m->x, y, m->ld_y, post, norm, m->eps, rows, m->width, NULL, m->h, out, m->ld_h, st));
    } else {
        DEV(cmlb200_residual_add(m->x, y, m->ld_y, parts, post, m->eps, rows, m->width, m->h, out, m->ld_h, st));
    }
    return 0;
}

/* A layer whose sublayers read the same row: h holds its norm, and is the next layer's behind it. */
static int forward_side_by_side(const Layered* m, int run, const CMLLMBatch* b, void* st) {
    const Layer *l = &m->layers[run], *next = run + 1 < m->num_layers ? &m->layers[run + 1] : NULL;
    const LayerWeights* w = &m->layers[l->source].w;
    const int rows = b->rows, type = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    cmlb200_moe plan;
    cmlb200_gated_join j;
    memset(&j, 0, sizeof j);
    if (lml_product(m, &w->wqkvg, m->h, m->ld_h, rows, m->qkvg + l->proj_col, m->ld_qkvg, st)) return -1;
    if (w->wuq.w) {
        DEV(cmlb200_norm_columns(m->qkvg, m->ld_qkvg, l->proj_col, l->q_rank, w->dq_norm, m->eps, rows, m->cq, type, m->ld_cq, st));
        if (lml_product(m, &w->wuq, m->cq, m->ld_cq, rows, m->qkvg, m->ld_qkvg, st)) return -1;
    }
    if (attend(m, l, w, b, st) || lml_product(m, &w->wo, m->att, m->ld_att, rows, m->y_mix, m->ld_y, st)) return -1;
    if (w->wo2.w) {
        const void* operand = (const uint8_t*)m->att + (size_t)beside_col(l) * (m->f32 ? 4 : 2);
        if (lml_product(m, &w->wo2, operand, m->ld_att, rows, m->y_mix2, m->ld_y, st)) return -1;
        j.b = m->y_mix2;
        j.a_norm = w->left_out;
        j.b_norm = w->right_out;
    }
    j.a = m->y_mix;
    j.ldm = j.ldf = m->ld_y;
    j.ga = m->qkvg + l->gate_cols;
    j.ldg = m->ld_qkvg;
    if (l->ff) {
        if (expert_layer(m, l, w, rows, &plan, st)) return -1;
        j.f = m->y;
        j.gf = j.ga + m->width;
        j.parts = &plan;
    }
    if (next && next->again) {
        j.table = m->embed;
        j.table_dtype = type;
        j.vocab = m->vocab;
        j.tokens = b->d_tokens;
    }
    DEV(cmlb200_gated_join_rows(&j, m->x, next ? m->layers[next->source].w.sub[0].norm : NULL, m->eps, rows, m->width, m->h, type, m->ld_h, st));
    return 0;
}

static int layered_forward(void* model, const CMLLMBatch* b, void* st) {
    const Layered* m = (const Layered*)model;
    const int rows = b->rows, out = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    if (rows > m->max_rows) { LOG_ERROR("layered_forward: %d rows of %d", rows, m->max_rows); return -1; }
    if (m->streams) DEV(cmlb200_embed_streams(m->embed, out, b->d_tokens, m->embed_scale, m->streams, rows, m->width, m->vocab, m->x, st));
    else DEV(cmlb200_embed_rows(m->embed, out, b->d_tokens, b->d_pos, m->freq, rows, m->width, m->vocab, m->x, st));
    if (join(m, NULL, &m->layers[m->layers[0].source].w.sub[0], NULL, NULL, rows, st)) return -1;
    for (int i = 0; i < m->num_layers; i++) {
        const Layer* l = &m->layers[i];
        const LayerWeights* w = &m->layers[l->source].w;
        const Sublayer* next = i + 1 < m->num_layers ? &m->layers[m->layers[i + 1].source].w.sub[0] : NULL;
        cmlb200_moe plan;
        if (m->design->side_by_side) {
            if (forward_side_by_side(m, i, b, st)) return -1;
            continue;
        }
        if (lml_product(m, &w->wqkvg, m->h, m->ld_h, rows, m->qkvg, m->ld_qkvg, st) || attend(m, l, w, b, st) ||
            lml_product(m, &w->wo, m->att, m->ld_att, rows, m->y, m->ld_y, st) || join(m, &w->sub[0], l->ff ? &w->sub[1] : next, NULL, NULL, rows, st))
            return -1;
        if (!l->ff) continue;
        if (l->experts ? expert_layer(m, l, w, rows, &plan, st) : feed_forward(m, l, w, rows, st)) return -1;
        if (join(m, &w->sub[1], next, l->experts ? &plan : NULL, l->shared_ff ? m->y_shared : NULL, rows, st)) return -1;
    }
    return 0;
}

static int layered_head(void* model, const int* d_rows, int n, float* d_logits, void* st) {
    const Layered* m = (const Layered*)model;
    const int out = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    if (m->streams) {
        const cmlb200_streams sum = {m->streams, NULL, NULL, NULL};
        DEV(cmlb200_stream_join(&sum, m->x, NULL, 0, NULL, m->final_norm, m->eps, n, m->width, d_rows, m->h, out, m->ld_h, st));
    } else {
        DEV(cmlb200_residual_norm(m->x, NULL, 0, NULL, m->final_norm, m->eps, n, m->width, d_rows, m->h, out, m->ld_h, st));
    }
    return lml_product(m, &m->head, m->h, m->ld_h, n, d_logits, m->vocab, st);
}

static int layered_check(void* model, const CMLLMBatch* b) {
    const Layered* m = (const Layered*)model;
    int status = 0;
    if (m->f32) return 0;
    if (m->q) DEV(cmlb200_attention_latent_status(&status, 1));
    if (status) return -1;
    if (b->rows <= SKINNY_ROWS) return 0;
    DEV(cmlb200_gemm_dense_status(&status, 1));
    return status ? -1 : 0;
}

/* ---- class --------------------------------------------------------------------------------------------- */
static void layered_free(void* model) {
    Layered* m = (Layered*)model;
    if (!m) return;
    for (int i = 0; m->layers && i < m->num_layers; i++) {
        Layer* l = &m->layers[i];
        LayerWeights* w = &l->w;
        const Sublayer *a = &w->sub[0], *b = &w->sub[1];
        void* bufs[] = {w->wqkvg.w, w->wo.w, w->wgu.w, w->wd.w, a->norm, a->post, a->in, a->out, a->mix, b->norm, b->post, b->in, b->out, b->mix, w->q_norm, w->k_norm,
                        w->slopes, w->sinks, w->c_norm, w->coef, (void*)w->wqkvg.bias, (void*)w->wo.bias, w->wukt, w->wukv.w, w->router.w, w->experts_gu.w,
                        w->experts_down.w, w->shared_gu.w, w->shared_down.w, w->correction, w->conv, w->rate, w->dt_bias, w->o_norm, w->wa.w, w->wg.w, w->wuq.w, w->wo2.w, w->dq_norm, w->talk, w->left_out, w->right_out, l->attn.ring, l->gru.state, l->freq,
                        l->attn.k_pool, l->attn.v_pool, l->delta.state, l->delta.ring, l->kv_from == i ? l->lat.pool : NULL};
        for (size_t k = 0; k < sizeof bufs / sizeof bufs[0]; k++) cmlb200_free(bufs[k]);
    }
    const cmlb200_moe* p = &m->plan;
    void* bufs[] = {m->embed, m->freq, m->final_norm, m->head.w, m->x, m->qkvg, m->y, m->gu, m->h, m->att, m->f, m->q, m->o, m->expand_table, m->expand_k,
                    m->expand_v, m->expand_c, m->xp, m->router, p->ids, p->weight, p->pos, p->src, p->expert, p->start, p->count, p->active, p->num_active,
                    p->tiles, p->num_tiles, p->self, m->y_shared, m->dec, m->gate, m->low, m->delta_work, m->y_mix, m->y_mix2, m->cq, m->q_rows_out, m->scores};
    for (size_t k = 0; k < sizeof bufs / sizeof bufs[0]; k++) cmlb200_free(bufs[k]);
    free(m->layers);
    free(m);
}

static void* layered_load(const char* path, const CMLJson* config, const CMLLMOptions* options, CMLLMInfo* info) {
    const char* arch = cml_json_string(config, "architecture");
    const LayeredDesign* design = NULL;
    for (size_t i = 0; i < sizeof kDesigns / sizeof kDesigns[0]; i++) if (arch && !strcmp(arch, kDesigns[i].architecture)) design = &kDesigns[i];
    Layered* m = design ? (Layered*)calloc(1, sizeof *m) : NULL;
    if (!m) return NULL;
    m->design = design;
    m->f32 = options->dtype == DTYPE_FLOAT32;
    m->max_sequences = options->max_sequences;
    char file[4096];
    snprintf(file, sizeof file, "%s/model.safetensors", path);
    CMLSafetensors* st = NULL;
    int rc = read_config(config, m) || !(st = cml_safetensors_open(file)) || load_shared(m, st);
    for (int i = 0; i < m->num_layers && !rc; i++) {
        if (m->layers[i].source == i) rc = load_layer(m, st, i);
        if (!rc) rc = make_rotation(&m->layers[i]);
    }
    cml_safetensors_close(st);
    if (rc || make_activations(m, options->max_step_rows)) { layered_free(m); return NULL; }
    info->vocab = m->vocab;
    for (int i = 0; i < m->num_layers; i++) {
        const int window = window_of(&m->layers[i]);
        if (window <= 0) { info->window = 0; break; }
        if (window > info->window) info->window = window;
        info->keep_first = lml_most(info->keep_first, m->layers[i].attn.keep);
    }
    return m;
}

#define LAYERED_CLASS(name) {.architecture = name, .load = layered_load, .free = layered_free, .make_pools = layered_make_pools, .forward = layered_forward, \
                             .head = layered_head, .check = layered_check}
static const CMLLMClass kLayeredClasses[] = {LAYERED_CLASS("Rarolorn"), LAYERED_CLASS("Situlorn"), LAYERED_CLASS("Lenedra"), LAYERED_CLASS("Zevilorn")};

__attribute__((constructor)) static void register_layered(void) {
    for (size_t i = 0; i < sizeof kLayeredClasses / sizeof kLayeredClasses[0]; i++) cml_lm_register(&kLayeredClasses[i]);
}
