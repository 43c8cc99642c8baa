/* Decoder-only models described layer by layer in config.json and stored as safetensors. A design is a row
 * of switches (LayeredDesign below); sizes, windows, scales and the order of layers come from the file.
 *
 *   config.json     architecture, vocab, width, norm.eps, layers: [{type, mixer, mlp, weights_of?}]
 *   mixer           grouped heads: heads, kv_heads, dim, vdim, scale, mask.size, q_temp {coef, every}
 *                   latents: heads, dim, rot_dim, vdim, kv_rank, scale, mask.size, rot {base, dims, scaling {factor,
 *                   original, fast, slow}}, kv_from (the layer whose cache this one reads)
 *   mlp             {kind: "dense", ff}, {kind: "moe", expert {ff, limit}, router {experts, top}} or null
 *   weights_of      index of the layer whose tensors this one uses; its cache is its own
 *   tensors         embed, final.norm, head, l<i>.norm1 / norm1b / norm2 / norm2b (as the design has them),
 *                   l<i>.mix.q / k / v / g / o / q.norm / k.norm, or q / dkv / dkv.norm / uk / uv / g / o,
 *                   l<i>.mlp.gate / up / down, up / down / act, or router and e<j>.gate / up / down; linear weights [out, in]
 *
 * On the device a layer's q, k, v and gate rows are one matrix, and the feed-forward's gate and up rows one
 * matrix interleaved in groups of 16 (the epilogues of both products pair them). Between two sublayers runs
 * one kernel: norm of the finished sublayer's output, residual add, norm for the next one. The residual, norms,
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

#include "cml_lm_internal.h"
#include "cml_safetensors.h"

#define SKINNY_ROWS 32
#define MAX_LAYERS 4096
#define EXPERT_ROWS 128            /* row tile of the experts' tensor-core product */
#define EXPAND_KEYS 65536          /* keys the scratch cache of long portions holds at most (CMLB200_EXPAND_KEYS: another number) */
#define DEV(call) do { if (CML_DEV_FAIL((call), __func__)) return -1; } while (0)

typedef struct MixerKind {
    const char* type;
    int latent;                  /* latent attention; 0: grouped heads */
    int wide_gate;               /* latent: sigmoid gate on every element of the heads' output */
} MixerKind;

typedef enum { FF_GATED, FF_POLY_NORM } DenseForm;

typedef struct LayeredDesign {
    const char* architecture;
    MixerKind mixers[2];
    double position_base;        /* > 0: sinusoidal position vector with that base added to the embedding */
    int input_norms;             /* each sublayer reads a normed residual; 0: the residual itself */
    const char* output_norms[2]; /* tensors of the norm on each sublayer's output before it joins the residual; NULL: none */
    int wide_qk_norm;            /* RMS norm of the whole q and k projections */
    int linear_bias;             /* scores lose slope_h * distance, slope_h = 2^(-8 (h + 1) / heads) */
    int sink;                    /* one added to the softmax denominator */
    int head_gate;               /* sigmoid gate per head */
    DenseForm dense;             /* of a dense feed-forward */
    int act;                     /* of a gated feed-forward, or of the experts */
    int experts;                 /* feed-forwards of experts are known */
} LayeredDesign;

static const LayeredDesign kDesigns[] = {
    {"Rarolorn", {{"attention", 0, 0}}, 10000.0, 1, {"norm1b", "norm2b"}, 1, 1, 1, 1, FF_GATED, CMLB200_ACT_GELU_TANH, 0},
    {"Situlorn", {{"latent_attention", 1, 0}, {"latent_attention_2", 1, 1}}, 0.0, 0, {"norm1", "norm2"}, 0, 0, 0, 0, FF_POLY_NORM, CMLB200_ACT_CLAMPED, 1},
};

typedef struct LayerWeights {    /* device tensors of a layer that owns some */
    cmlb200_dense wqkvg, wo, wgu, wd;        /* latent layers: q, dkv and g rows; wgu without a gate: the up rows alone */
    float *norm1, *norm1b, *norm2, *norm2b, *q_norm, *k_norm, *slopes;
    float *c_norm, *coef;
    void* wukt;                  /* per head, transposed */
    cmlb200_dense wukv;          /* all Wuk rows, then all Wuv rows (per head padded to 16); in the 32-bit form Wuv alone */
    cmlb200_dense router, experts_gu, experts_down;
} LayerWeights;

typedef struct Layer {
    int source;                  /* the layer whose weights it uses */
    int ff;                      /* 0: no feed-forward */
    int experts, top;            /* 0: a dense feed-forward; ff is an expert's */
    float limit;
    const MixerKind* kind;
    cmlb200_attn attn;
    cmlb200_latent lat;
    int kv_from;                 /* the layer whose latents it reads: itself, as a rule */
    double rot_base, rot_scaling[4];         /* scaling[0]: factor, 0 without */
    float* freq;
    LayerWeights w;
} Layer;

typedef struct Layered {
    const LayeredDesign* design;
    int f32, vocab, width, num_layers;
    float eps;
    Layer* layers;
    void* embed;
    float *freq, *final_norm;
    cmlb200_dense head;
    int max_rows, max_sequences, ld_h, ld_qkvg, ld_att, ld_y, ld_f, ld_gu;
    float *x, *qkvg, *y, *gu;
    void *h, *att, *f;           /* operands of the matrix products: bf16, or fp32 in the 32-bit form */
    /* latent layers */
    int q_rows;                  /* rows whose queries are transformed at a time */
    void *q, *o;                 /* transformed queries (fp16 or fp32) and weighted latents (bf16 or fp32) */
    int expand_keys, *expand_table;
    void *expand_k, *expand_v, *expand_c;
    int slots, table_ld;
    /* experts */
    cmlb200_moe plan;
    void* xp;
    float* router;
    int ld_router;
} Layered;

static int round_up(int v, int to) { return (v + to - 1) / to * to; }

/* ---- configuration ---------------------------------------------------------------------------------- */
static int is_object(const CMLJson* j) { return j && j->type == CML_JSON_OBJECT; }

static int read_grouped(const CMLJson* mixer, Layer* l, int index, const LayeredDesign* design) {
    const CMLJson *mask = cml_json_get(mixer, "mask"), *temp = cml_json_get(mixer, "q_temp");
    cmlb200_attn* a = &l->attn;
    double scale = 0.0, coef = 0.0, every = 0.0;
    if (cml_json_int(mixer, "heads", &a->heads) || cml_json_int(mixer, "kv_heads", &a->kv_heads) || cml_json_int(mixer, "dim", &a->dim) ||
        cml_json_int(mixer, "vdim", &a->vdim) || cml_json_double(mixer, "scale", &scale) || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads ||
        a->dim <= 0 || a->vdim <= 0 || a->heads > 65535 || a->dim > 256 || a->vdim > 256) {
        LOG_ERROR("layer %d: heads, kv_heads, dim, vdim (up to 256) or scale are missing or do not fit", index);
        return -1;
    }
    if (is_object(mask) && (cml_json_int(mask, "size", &a->window) || a->window <= 0)) { LOG_ERROR("layer %d: mask.size", index); return -1; }
    if (is_object(temp) && (cml_json_double(temp, "coef", &coef) || cml_json_double(temp, "every", &every) || every <= 0.0)) { LOG_ERROR("layer %d: q_temp", index); return -1; }
    a->scale = (float)scale;
    a->temp_coef = (float)coef;
    a->temp_every = (float)every;
    a->dim_ld = round_up(a->dim, 16);
    a->vdim_ld = round_up(a->vdim, 16);
    a->sink = design->sink;
    a->gate_col = design->head_gate ? a->heads * a->dim + a->kv_heads * (a->dim + a->vdim) : -1;
    return 0;
}

static int read_latent(const CMLJson* mixer, Layer* l, int index) {
    const CMLJson *mask = cml_json_get(mixer, "mask"), *rot = cml_json_get(mixer, "rot"), *scaling = cml_json_get(rot, "scaling");
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
    if (cml_json_double(rot, "base", &l->rot_base) || cml_json_int(rot, "dims", &dims) || dims != a->rot_dim || l->rot_base <= 0.0 || l->rot_base == 1.0) {
        LOG_ERROR("layer %d: rot.base is missing or rot.dims is not rot_dim", index);
        return -1;
    }
    if (is_object(scaling))
        for (int k = 0; k < 4; k++)
            if (cml_json_double(scaling, keys[k], &l->rot_scaling[k]) || l->rot_scaling[k] <= 0.0) { LOG_ERROR("layer %d: rot.scaling.%s", index, keys[k]); return -1; }
    const CMLJson* from = cml_json_get(mixer, "kv_from");
    if (from && from->type != CML_JSON_NULL && cml_json_int(mixer, "kv_from", &l->kv_from)) { LOG_ERROR("layer %d: kv_from", index); return -1; }
    const int q = a->heads * (a->dim + a->rot_dim), kv = a->rank + a->rot_dim;
    a->scale = (float)scale;
    a->ld = round_up(kv, 16);
    a->ld_rank = round_up(a->rank, 64);
    a->kv_col = l->kv_from == index ? q : -1;
    a->gate_col = l->kind->wide_gate ? q + (l->kv_from == index ? kv : 0) : -1;
    return 0;
}

static int read_feed_forward(const CMLJson* mlp, Layer* l, int index, const LayeredDesign* design) {
    const char* kind = cml_json_string(mlp, "kind");
    if (kind && !strcmp(kind, "dense") && !cml_json_int(mlp, "ff", &l->ff) && l->ff > 0) return 0;
    const CMLJson *expert = cml_json_get(mlp, "expert"), *router = cml_json_get(mlp, "router");
    double limit = 0.0;
    if (design->experts && kind && !strcmp(kind, "moe") && !cml_json_int(expert, "ff", &l->ff) && l->ff > 0 && !cml_json_double(expert, "limit", &limit) &&
        !cml_json_int(router, "experts", &l->experts) && !cml_json_int(router, "top", &l->top) && l->experts > 0 && l->experts <= 1024 && l->top > 0 &&
        l->top <= l->experts) {
        l->limit = (float)limit;
        return 0;
    }
    LOG_ERROR("layer %d: feed-forward of kind '%s' is not known or incomplete", index, kind ? kind : "(none)");
    return -1;
}

static int read_layer(const CMLJson* j, Layer* l, int index, const LayeredDesign* design) {
    const CMLJson *mixer = cml_json_get(j, "mixer"), *mlp = cml_json_get(j, "mlp");
    const char* type = cml_json_string(j, "type");
    for (size_t k = 0; k < sizeof design->mixers / sizeof design->mixers[0]; k++)
        if (type && design->mixers[k].type && !strcmp(type, design->mixers[k].type)) l->kind = &design->mixers[k];
    if (!l->kind) { LOG_ERROR("layer %d: mixer type '%s' is not known to %s", index, type ? type : "(none)", design->architecture); return -1; }
    l->kv_from = index;
    if (l->kind->latent ? read_latent(mixer, l, index) : read_grouped(mixer, l, index, design)) return -1;
    if (is_object(mlp) && read_feed_forward(mlp, l, index, design)) return -1;
    l->source = index;
    int of;
    if (!cml_json_int(j, "weights_of", &of)) l->source = of;
    return 0;
}

static int window_of(const Layer* l) { return l->kind->latent ? l->lat.window : l->attn.window; }

static int same_shape(const Layer* a, const Layer* b) {
    if (a->kind != b->kind || a->ff != b->ff || a->experts != b->experts) return 0;
    if (a->kind->latent)
        return a->lat.heads == b->lat.heads && a->lat.dim == b->lat.dim && a->lat.rot_dim == b->lat.rot_dim && a->lat.vdim == b->lat.vdim &&
               a->lat.rank == b->lat.rank && (a->lat.kv_col < 0) == (b->lat.kv_col < 0);
    return a->attn.heads == b->attn.heads && a->attn.kv_heads == b->attn.kv_heads && a->attn.dim == b->attn.dim && a->attn.vdim == b->attn.vdim;
}

/* A layer that reads another one's cache: an earlier one, which fills its own, with the same latents and rotation. */
static int check_kv_from(const Layered* m, int i) {
    const Layer* l = &m->layers[i];
    if (!l->kind->latent || l->kv_from == i) return 0;
    const Layer* f = l->kv_from >= 0 && l->kv_from < i ? &m->layers[l->kv_from] : NULL;
    if (f && f->kind->latent && f->kv_from == l->kv_from && f->lat.rank == l->lat.rank && f->lat.rot_dim == l->lat.rot_dim && f->rot_base == l->rot_base &&
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
    m->num_layers = layers->count;
    m->layers = (Layer*)calloc((size_t)m->num_layers, sizeof(Layer));
    if (!m->layers) return -1;
    int i = 0;
    for (const CMLJson* j = layers->child; j; j = j->next, i++)
        if (read_layer(j, &m->layers[i], i, m->design)) return -1;
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
static float element(const CMLSafetensor* t, size_t i) {
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

static int find(const CMLSafetensors* st, const char* prefix, const char* name, int rows, int cols, CMLSafetensor* t) {
    char full[160];
    snprintf(full, sizeof full, "%s%s", prefix, name);
    if (cml_safetensors_find(st, full, t)) { LOG_ERROR("tensor '%s' is missing", full); return -1; }
    if (t->dtype == DTYPE_INT32 || t->ndim != (cols ? 2 : 1) || t->shape[0] != rows || (cols && t->shape[1] != cols)) {
        LOG_ERROR("tensor '%s' has another shape or type than config.json says ([%d, %d] expected)", full, rows, cols);
        return -1;
    }
    return 0;
}

static int upload(void** dst, const void* src, size_t bytes) {
    if (CML_DEV_FAIL(cmlb200_malloc(dst, bytes), "upload") || CML_DEV_FAIL(cmlb200_memcpy_h2d(*dst, src, bytes, NULL), "upload") ||
        CML_DEV_FAIL(cmlb200_stream_sync(NULL), "upload"))
        return -1;
    return 0;
}

/* Frequencies of the rotated pairs and the factor on sine and cosine. With scaling, the pairs that turn fewer than `slow`
 * times within `original` positions are slowed down by the factor, those that turn more than `fast` times are not, and a
 * ramp over the pairs lies between. */
static int make_rotation(Layer* l) {
    cmlb200_latent* a = &l->lat;
    const double n = a->rot_dim, *s = l->rot_scaling;
    float* f = (float*)malloc((size_t)(a->rot_dim / 2) * sizeof(float));
    if (!f) return -1;
    double lo = 0.0, hi = 0.0;
    if (s[0] > 0.0) {
        const double two_pi = 6.283185307179586476925;
        lo = fmax(floor(n * log(s[1] / (two_pi * s[2])) / (2.0 * log(l->rot_base))), 0.0);
        hi = fmin(ceil(n * log(s[1] / (two_pi * s[3])) / (2.0 * log(l->rot_base))), n - 1.0);
    }
    for (int i = 0; i < a->rot_dim / 2; i++) {
        const double plain = pow(l->rot_base, -2.0 * i / n);
        const double ramp = s[0] > 0.0 ? fmin(fmax((i - lo) / fmax(hi - lo, 0.001), 0.0), 1.0) : 0.0;
        f[i] = (float)(ramp > 0.0 ? plain / s[0] * ramp + plain * (1.0 - ramp) : plain);
    }
    a->rot_mul = s[0] > 0.0 ? (float)(0.1 * log(s[0]) + 1.0) : 1.0f;
    const int rc = upload((void**)&l->freq, f, (size_t)(a->rot_dim / 2) * sizeof(float));
    free(f);
    a->freq = l->freq;
    return rc;
}

static int load_vector(const CMLSafetensors* st, const char* prefix, const char* name, int n, float** dst) {
    CMLSafetensor t;
    if (find(st, prefix, name, n, 0, &t)) return -1;
    float* v = (float*)malloc((size_t)n * sizeof(float));
    if (!v) return -1;
    for (int i = 0; i < n; i++) v[i] = element(&t, (size_t)i);
    const int rc = upload((void**)dst, v, (size_t)n * sizeof(float));
    free(v);
    return rc;
}

static void put_row(const Layered* m, uint8_t* dst, const CMLSafetensor* t, int row, int cols) {
    const size_t at = (size_t)row * (size_t)cols;
    if (!m->f32 && t->dtype == DTYPE_BFLOAT16) memcpy(dst, (const uint8_t*)t->data + 2 * at, (size_t)cols * 2);
    else if (m->f32) for (int c = 0; c < cols; c++) ((float*)(void*)dst)[c] = element(t, at + (size_t)c);
    else for (int c = 0; c < cols; c++) ((uint16_t*)(void*)dst)[c] = to_bf16(element(t, at + (size_t)c));
}

/* Stacks up to four [rows, cols] tensors; interleave: two of them in turns of 16 rows, each padded to whole groups. */
static int load_matrix(const Layered* m, const CMLSafetensors* st, const char* prefix, const char* const* names, const int* rows, int parts, int cols,
                       int interleave, cmlb200_dense* out) {
    int total = 0;
    CMLSafetensor t[4];
    for (int p = 0; p < parts; p++) {
        if (find(st, prefix, names[p], rows[p], cols, &t[p])) return -1;
        total += interleave ? round_up(rows[p], 16) : rows[p];
    }
    const size_t es = m->f32 ? 4 : 2, ld = (size_t)round_up(cols, 64), bytes = (size_t)round_up(total, 16) * ld * es;
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
    const int rc = upload(&out->w, host, bytes);
    free(host);
    return rc;
}

static int alloc_matrix(const Layered* m, int rows, int cols, cmlb200_dense* out, uint8_t** host) {
    out->dtype = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    out->rows = rows;
    out->cols = cols;
    out->ld = round_up(cols, 64);
    *host = (uint8_t*)calloc((size_t)round_up(rows, 16) * (size_t)out->ld, m->f32 ? 4 : 2);
    if (!*host) LOG_ERROR("out of memory for a [%d, %d] weight", rows, cols);
    return *host ? 0 : -1;
}
static int upload_matrix(const Layered* m, cmlb200_dense* w, uint8_t* host) {
    const int rc = upload(&w->w, host, (size_t)round_up(w->rows, 16) * (size_t)w->ld * (m->f32 ? 4 : 2));
    free(host);
    return rc;
}

/* The experts' gate and up rows (interleaved as in load_matrix) and their down rows, one expert behind the other. */
static int load_experts(Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l) {
    LayerWeights* w = &l->w;
    const int gu = 2 * round_up(l->ff, 16), down = round_up(m->width, 16);
    const size_t es = m->f32 ? 4 : 2;
    const char* router[1] = {"mlp.router"};
    uint8_t *hg, *hd;
    if (load_matrix(m, st, prefix, router, &l->experts, 1, m->width, 0, &w->router) || alloc_matrix(m, l->experts * gu, m->width, &w->experts_gu, &hg)) return -1;
    if (alloc_matrix(m, l->experts * down, l->ff, &w->experts_down, &hd)) { free(hg); return -1; }
    int rc = 0;
    for (int e = 0; e < l->experts && !rc; e++) {
        char name[3][48];
        CMLSafetensor t[3];
        snprintf(name[0], sizeof name[0], "mlp.e%d.gate", e);
        snprintf(name[1], sizeof name[1], "mlp.e%d.up", e);
        snprintf(name[2], sizeof name[2], "mlp.e%d.down", e);
        rc = find(st, prefix, name[0], l->ff, m->width, &t[0]) || find(st, prefix, name[1], l->ff, m->width, &t[1]) || find(st, prefix, name[2], m->width, l->ff, &t[2]);
        for (int p = 0; p < 2 && !rc; p++)
            for (int r = 0; r < l->ff; r++)
                put_row(m, hg + ((size_t)e * gu + (size_t)(r / 16) * 32 + (size_t)(p * 16 + r % 16)) * (size_t)w->experts_gu.ld * es, &t[p], r, m->width);
        for (int r = 0; r < m->width && !rc; r++) put_row(m, hd + ((size_t)e * down + (size_t)r) * (size_t)w->experts_down.ld * es, &t[2], r, l->ff);
    }
    if (rc) { free(hg); free(hd); return -1; }
    rc = upload_matrix(m, &w->experts_gu, hg);
    return upload_matrix(m, &w->experts_down, hd) || rc ? -1 : 0;
}

/* Wuk and Wuv in the forms of the two ways a latent layer attends, or of the 32-bit one. */
static int load_latent_heads(const Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l) {
    const cmlb200_latent* a = &l->lat;
    LayerWeights* w = &l->w;
    CMLSafetensor uk, uv;
    const int H = a->heads, D = a->dim, V = a->vdim, R = a->rank;
    if (find(st, prefix, "mix.uk", H * D, R, &uk) || find(st, prefix, "mix.uv", H * V, R, &uv)) return -1;
    const int rp = m->f32 ? R : round_up(R, 16), dp = m->f32 ? D : round_up(D, 64);
    const size_t es = m->f32 ? 4 : 2, bytes = (size_t)H * (size_t)rp * (size_t)dp * es;
    uint8_t* t = (uint8_t*)calloc(bytes, 1);
    if (!t) { LOG_ERROR("out of memory for '%smix.uk'", prefix); return -1; }
    for (int h = 0; h < H; h++)
        for (int d = 0; d < D; d++)
            for (int r = 0; r < R; r++) {
                const size_t to = ((size_t)h * (size_t)rp + (size_t)r) * (size_t)dp + (size_t)d;
                const float v = element(&uk, (size_t)(h * D + d) * (size_t)R + (size_t)r);
                if (m->f32) ((float*)(void*)t)[to] = v;
                else ((uint16_t*)(void*)t)[to] = to_bf16(v);
            }
    int rc = upload(&w->wukt, t, bytes);
    free(t);
    if (rc) return -1;
    if (m->f32) {
        float* v = (float*)malloc((size_t)H * (size_t)V * (size_t)R * sizeof(float));
        if (!v) return -1;
        for (int r = 0; r < H * V; r++) put_row(m, (uint8_t*)(v + (size_t)r * (size_t)R), &uv, r, R);
        rc = upload(&w->wukv.w, v, (size_t)H * (size_t)V * (size_t)R * sizeof(float));
        free(v);
        return rc;
    }
    const int vp = round_up(V, 16);
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

static int load_mixer(Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l) {
    LayerWeights* w = &l->w;
    const char* out[1] = {"mix.o"};
    const int out_rows[1] = {m->width};
    if (l->kind->latent) {
        const cmlb200_latent* a = &l->lat;
        const char* proj[3] = {"mix.q"};
        int rows[3] = {a->heads * (a->dim + a->rot_dim)}, parts = 1;
        if (a->kv_col >= 0) { proj[parts] = "mix.dkv"; rows[parts++] = a->rank + a->rot_dim; }
        if (a->gate_col >= 0) { proj[parts] = "mix.g"; rows[parts++] = a->heads * a->vdim; }
        return (a->kv_col >= 0 && load_vector(st, prefix, "mix.dkv.norm", a->rank, &w->c_norm)) || load_matrix(m, st, prefix, proj, rows, parts, m->width, 0, &w->wqkvg) ||
               load_latent_heads(m, st, prefix, l) || load_matrix(m, st, prefix, out, out_rows, 1, a->heads * a->vdim, 0, &w->wo) ? -1 : 0;
    }
    const cmlb200_attn* a = &l->attn;
    const char* proj[4] = {"mix.q", "mix.k", "mix.v", "mix.g"};
    const int proj_rows[4] = {a->heads * a->dim, a->kv_heads * a->dim, a->kv_heads * a->vdim, a->heads};
    if ((m->design->wide_qk_norm && (load_vector(st, prefix, "mix.q.norm", proj_rows[0], &w->q_norm) || load_vector(st, prefix, "mix.k.norm", proj_rows[1], &w->k_norm))) ||
        load_matrix(m, st, prefix, proj, proj_rows, m->design->head_gate ? 4 : 3, m->width, 0, &w->wqkvg) ||
        load_matrix(m, st, prefix, out, out_rows, 1, a->heads * a->vdim, 0, &w->wo))
        return -1;
    if (m->design->linear_bias) {
        float* s = (float*)malloc((size_t)a->heads * sizeof(float));
        if (!s) return -1;
        for (int h = 0; h < a->heads; h++) s[h] = (float)exp2(-8.0 * (h + 1) / a->heads);
        const int rc = upload((void**)&w->slopes, s, (size_t)a->heads * sizeof(float));
        free(s);
        return rc;
    }
    return 0;
}

static int load_layer(Layered* m, const CMLSafetensors* st, int index) {
    Layer* l = &m->layers[index];
    LayerWeights* w = &l->w;
    const LayeredDesign* d = m->design;
    char prefix[32];
    snprintf(prefix, sizeof prefix, "l%d.", index);
    const char *gu[2] = {"mlp.gate", "mlp.up"}, *up[1] = {"mlp.up"}, *down[1] = {"mlp.down"};
    const int out_rows[1] = {m->width}, ff_rows[2] = {l->ff, l->ff};
    if ((d->input_norms && load_vector(st, prefix, "norm1", m->width, &w->norm1)) ||
        (d->output_norms[0] && load_vector(st, prefix, d->output_norms[0], m->width, &w->norm1b)) || load_mixer(m, st, prefix, l))
        return -1;
    if (!l->ff) return 0;
    if ((d->input_norms && load_vector(st, prefix, "norm2", m->width, &w->norm2)) ||
        (d->output_norms[1] && load_vector(st, prefix, d->output_norms[1], m->width, &w->norm2b)))
        return -1;
    if (l->experts) return load_experts(m, st, prefix, l);
    if (d->dense == FF_POLY_NORM ? load_matrix(m, st, prefix, up, ff_rows, 1, m->width, 0, &w->wgu) || load_vector(st, prefix, "mlp.act", 4, &w->coef)
                                 : load_matrix(m, st, prefix, gu, ff_rows, 2, m->width, 1, &w->wgu))
        return -1;
    return load_matrix(m, st, prefix, down, out_rows, 1, l->ff, 0, &w->wd);
}

static int load_shared(Layered* m, const CMLSafetensors* st) {
    CMLSafetensor t;
    const char* head[1] = {"head"};
    const int head_rows[1] = {m->vocab};
    if (find(st, "", "embed", m->vocab, m->width, &t)) return -1;
    const size_t row = (size_t)m->width * (m->f32 ? 4 : 2);
    uint8_t* e = (uint8_t*)malloc((size_t)m->vocab * row);
    float* fr = (float*)malloc((size_t)(m->width / 2 + 1) * sizeof(float));
    int rc = e && fr ? 0 : -1;
    for (int i = 0; i < m->vocab && !rc; i++) put_row(m, e + (size_t)i * row, &t, i, m->width);
    rc = rc || upload(&m->embed, e, (size_t)m->vocab * row);
    if (!rc && m->design->position_base > 0.0) {
        for (int i = 0; i <= m->width / 2; i++) fr[i] = (float)pow(m->design->position_base, -2.0 * i / m->width);
        rc = upload((void**)&m->freq, fr, (size_t)(m->width / 2 + 1) * sizeof(float));
    }
    free(e);
    free(fr);
    return rc || load_vector(st, "", "final.norm", m->width, &m->final_norm) || load_matrix(m, st, "", head, head_rows, 1, m->width, 0, &m->head) ? -1 : 0;
}

/* ---- activations and caches --------------------------------------------------------------------------- */
static int zeroed(void** dst, size_t bytes) {
    DEV(cmlb200_malloc(dst, bytes));
    DEV(cmlb200_memset(*dst, 0, bytes, NULL));
    return 0;
}

static int most(int a, int b) { return a > b ? a : b; }

/* Operand buffers have strides that are multiples of 64 and start out zero: the decode product reads up
 * to the padded width, where its weights are zero. */
static int make_activations(Layered* m, int rows) {
    int q = 0, att = 0, ff = 0, z = 0, latent_q = 0, latent_o = 0, experts = 0, top = 0;
    long positions = 0, tiles = 0;
    for (int i = 0; i < m->num_layers; i++) {
        const Layer* l = &m->layers[i];
        q = most(q, m->layers[l->source].w.wqkvg.rows);
        ff = most(ff, l->ff);
        if (l->kind->latent) {
            const cmlb200_latent* a = &l->lat;
            att = most(att, a->heads * a->vdim);
            latent_q = most(latent_q, a->heads * (m->f32 ? a->rank + a->rot_dim : a->ld));
            latent_o = most(latent_o, a->heads * (m->f32 ? a->rank : a->ld_rank));
        } else {
            att = most(att, l->attn.heads * l->attn.vdim);
        }
        if (l->experts) {
            const long p = cmlb200_moe_positions(rows, l->top, l->experts, EXPERT_ROWS);
            if (p > positions) positions = p;
            if (p / EXPERT_ROWS + l->experts + 1 > tiles) tiles = p / EXPERT_ROWS + l->experts + 1;
            experts = most(experts, l->experts);
            top = most(top, l->top);
        } else if (l->ff) {
            z = most(z, m->design->dense == FF_POLY_NORM ? l->ff : (m->f32 ? 2 * round_up(l->ff, 16) : 0));
        }
        if (l->experts && m->f32) z = most(z, 2 * round_up(l->ff, 16));
    }
    m->max_rows = rows;
    m->ld_h = round_up(m->width, 64);
    m->ld_qkvg = round_up(q, 16);
    m->ld_att = round_up(att, 64);
    m->ld_y = round_up(m->width, 16);
    m->ld_f = round_up(ff ? ff : 1, 64);
    m->ld_gu = round_up(z, 16);
    m->ld_router = round_up(experts, 16);
    const size_t R = (size_t)rows, P = (size_t)(positions > rows ? positions : rows), es = m->f32 ? 4 : 2;
    const size_t head = R > 256 ? R : 256;                 /* the head normalises up to 256 rows at once into h */
    if (zeroed((void**)&m->x, R * (size_t)m->width * 4) || zeroed(&m->h, head * (size_t)m->ld_h * es) || zeroed((void**)&m->qkvg, R * (size_t)m->ld_qkvg * 4) ||
        zeroed(&m->att, R * (size_t)m->ld_att * es) || zeroed((void**)&m->y, P * (size_t)m->ld_y * 4) || zeroed(&m->f, P * (size_t)m->ld_f * es) ||
        (z && zeroed((void**)&m->gu, (m->f32 ? P : R) * (size_t)m->ld_gu * 4)))
        return -1;
    if (latent_q) {
        const long q_rows = (long)m->max_sequences * 64;
        m->q_rows = q_rows < rows ? (int)q_rows : rows;
        if (zeroed(&m->q, (size_t)m->q_rows * (size_t)latent_q * es) || zeroed(&m->o, (size_t)m->q_rows * (size_t)latent_o * es)) return -1;
    }
    if (experts) {
        cmlb200_moe* p = &m->plan;
        const size_t pairs = R * (size_t)top * 4, pos = P * 4, per = (size_t)experts * 4;
        if (zeroed((void**)&m->router, R * (size_t)m->ld_router * 4) || (!m->f32 && zeroed(&m->xp, P * (size_t)m->ld_h * es)) || zeroed((void**)&p->ids, pairs) ||
            zeroed((void**)&p->weight, pairs) || zeroed((void**)&p->pos, pairs) || zeroed((void**)&p->src, pos) || zeroed((void**)&p->expert, pos) ||
            zeroed((void**)&p->start, per) || zeroed((void**)&p->count, per) || zeroed((void**)&p->active, per) || zeroed((void**)&p->num_active, 4) ||
            zeroed((void**)&p->tiles, (size_t)tiles * 16) || zeroed((void**)&p->num_tiles, 4))
            return -1;
    }
    return CML_DEV_FAIL(cmlb200_stream_sync(NULL), "make_activations") ? -1 : 0;
}

/* The scratch cache of long portions: keys and values per head for as many tokens as a step may expand at a time. */
static int make_expansion(Layered* m, int blocks, int block_size, int slots, int table_ld) {
    int k = 0, v = 0, c = 0;
    for (int i = 0; i < m->num_layers; i++) {
        const cmlb200_latent* a = &m->layers[i].lat;
        if (!m->layers[i].kind->latent) continue;
        k = most(k, a->heads * round_up(a->dim + a->rot_dim, 16));
        v = most(v, a->heads * round_up(a->vdim, 16));
        c = most(c, a->ld_rank);
    }
    if (!k || m->f32) return 0;
    m->slots = slots;
    m->table_ld = table_ld;
    const char* env = getenv("CMLB200_EXPAND_KEYS");
    int keys = env && atoi(env) > 0 && atoi(env) < (1 << 28) ? round_up(atoi(env), block_size) : EXPAND_KEYS;
    if ((long)blocks * block_size < keys) keys = blocks * block_size;
    m->expand_keys = keys;
    const size_t n = (size_t)m->expand_keys;
    return zeroed(&m->expand_k, n * (size_t)k * 2) || zeroed(&m->expand_v, n * (size_t)v * 2) || zeroed(&m->expand_c, n * (size_t)c * 2) ||
           zeroed((void**)&m->expand_table, (size_t)slots * (size_t)table_ld * sizeof(int)) ? -1 : 0;
}

static int layered_make_pools(void* model, int blocks, int block_size, int slots, int table_ld) {
    Layered* m = (Layered*)model;
    const size_t es = m->f32 ? 4 : 2, tokens = (size_t)blocks * (size_t)block_size;
    for (int i = 0; i < m->num_layers; i++) {
        Layer* l = &m->layers[i];
        const LayerWeights* w = &m->layers[l->source].w;
        if (l->kind->latent) {
            cmlb200_latent* a = &l->lat;
            a->cache_dtype = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_F16;
            a->block_size = block_size;
            a->pool_blocks = blocks;
            a->c_norm = w->c_norm;
            a->eps = m->eps;
            if (l->kv_from != i) a->pool = m->layers[l->kv_from].lat.pool;
            else if (zeroed(&a->pool, tokens * (size_t)a->ld * es)) return -1;
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
        if (zeroed(&a->k_pool, heads * (size_t)a->dim_ld * es) || zeroed(&a->v_pool, heads * (size_t)a->vdim_ld * es)) return -1;
    }
    if (make_expansion(m, blocks, block_size, slots, table_ld)) return -1;
    DEV(cmlb200_stream_sync(NULL));
    return 0;
}

/* ---- a step ------------------------------------------------------------------------------------------- */
static int product(const Layered* m, const cmlb200_dense* w, const void* x, int ldx, int rows, float* y, int ldy, void* st) {
    if (m->f32) DEV(cmlb200_linear_dense_f32(w, (const float*)x, ldx, rows, y, ldy, st));
    else if (rows <= SKINNY_ROWS) DEV(cmlb200_gemv_dense(w, (const uint16_t*)x, ldx, rows, y, ldy, st));
    else DEV(cmlb200_gemm_dense(w, (const uint16_t*)x, ldx, rows, y, ldy, st));
    return 0;
}

/* Router, plan, the chosen experts' products; y then holds a row per (row, expert) pair. */
static int expert_layer(const Layered* m, const Layer* l, const LayerWeights* w, int rows, cmlb200_moe* plan, void* st) {
    const int act = m->design->act;
    *plan = m->plan;
    plan->experts = l->experts;
    plan->top = l->top;
    if (product(m, &w->router, m->h, m->ld_h, rows, m->router, m->ld_router, st)) return -1;
    DEV(cmlb200_moe_route(plan, m->router, m->ld_router, rows, m->f32 || rows <= SKINNY_ROWS ? 1 : EXPERT_ROWS, st));
    if (m->f32) {
        DEV(cmlb200_moe_linear_f32(plan, &w->experts_gu, (const float*)m->h, m->ld_h, 1, rows, 2 * round_up(l->ff, 16), m->gu, m->ld_gu, st));
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
    const int act = m->design->act;
    if (m->design->dense == FF_POLY_NORM) {
        if (product(m, &w->wgu, m->h, m->ld_h, rows, m->gu, m->ld_gu, st)) return -1;
        DEV(cmlb200_poly_norm(m->gu, m->ld_gu, rows, l->ff, w->coef, m->eps, m->f, m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16, m->ld_f, st));
    } else if (m->f32) {
        DEV(cmlb200_linear_dense_f32(&w->wgu, (const float*)m->h, m->ld_h, rows, m->gu, m->ld_gu, st));
        DEV(cmlb200_glu_rows_f32(m->gu, m->ld_gu, rows, l->ff, act, (float*)m->f, m->ld_f, st));
    } else if (rows <= SKINNY_ROWS) {
        DEV(cmlb200_gemv_dense_glu(&w->wgu, (const uint16_t*)m->h, m->ld_h, rows, l->ff, act, (uint16_t*)m->f, m->ld_f, st));
    } else {
        DEV(cmlb200_gemm_dense_glu(&w->wgu, (const uint16_t*)m->h, m->ld_h, rows, l->ff, act, (uint16_t*)m->f, m->ld_f, st));
    }
    return product(m, &w->wd, m->f, m->ld_f, rows, m->y, m->ld_y, st);
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
    s.dim_ld = round_up(s.dim, 16);
    s.vdim_ld = round_up(s.vdim, 16);
    s.scale = a->scale;
    s.window = a->window;
    s.gate_col = a->gate_col;
    s.gate_wide = a->gate_col >= 0;
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
            keys += round_up(k, a->block_size);
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
    if (l->kind->latent) return attend_latent(m, l, w, b, st);
    cmlb200_attn a = l->attn;
    a.block_table = b->d_table;
    a.table_ld = b->table_ld;
    if (m->f32) {
        DEV(cmlb200_qk_norm_append(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, b->rows, st));
        DEV(cmlb200_attention_rows_f32(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, b->rows, (float*)m->att, m->ld_att, st));
        return 0;
    }
    const int one = b->one_rows, more = b->rows - one;
    if (more) {
        DEV(cmlb200_qk_norm_append(&a, m->qkvg + (size_t)one * m->ld_qkvg, m->ld_qkvg, b->d_pos + one, b->d_slot + one, more, st));
        DEV(cmlb200_attention_tiles(&a, m->qkvg, m->ld_qkvg, b->d_tiles, b->tiles, (uint16_t*)m->att, m->ld_att, st));
    }
    if (one) DEV(cmlb200_attention_one(&a, m->qkvg, m->ld_qkvg, b->d_pos, b->d_slot, one, b->max_keys, (uint16_t*)m->att, m->ld_att, st));
    return 0;
}

/* A sublayer's output joins the residual; `next`: the norm in front of what reads it next (designs with input norms). */
static int join(const Layered* m, const float* post, const float* next, const cmlb200_moe* parts, int rows, void* st) {
    const int out = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    if (m->design->input_norms) DEV(cmlb200_residual_norm(m->x, m->y, m->ld_y, post, next, m->eps, rows, m->width, NULL, m->h, out, m->ld_h, st));
    else DEV(cmlb200_residual_add(m->x, m->y, m->ld_y, parts, post, m->eps, rows, m->width, m->h, out, m->ld_h, st));
    return 0;
}

static int layered_forward(void* model, const CMLLMBatch* b, void* st) {
    const Layered* m = (const Layered*)model;
    const int rows = b->rows, out = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    if (rows > m->max_rows) { LOG_ERROR("layered_forward: %d rows of %d", rows, m->max_rows); return -1; }
    DEV(cmlb200_embed_rows(m->embed, out, b->d_tokens, b->d_pos, m->freq, rows, m->width, m->vocab, m->x, st));
    if (m->design->input_norms) DEV(cmlb200_residual_norm(m->x, NULL, 0, NULL, m->layers[m->layers[0].source].w.norm1, m->eps, rows, m->width, NULL, m->h, out, m->ld_h, st));
    else DEV(cmlb200_residual_add(m->x, NULL, 0, NULL, NULL, m->eps, rows, m->width, m->h, out, m->ld_h, st));
    for (int i = 0; i < m->num_layers; i++) {
        const Layer* l = &m->layers[i];
        const LayerWeights* w = &m->layers[l->source].w;
        const float* next = i + 1 < m->num_layers ? m->layers[m->layers[i + 1].source].w.norm1 : NULL;
        cmlb200_moe plan;
        if (product(m, &w->wqkvg, m->h, m->ld_h, rows, m->qkvg, m->ld_qkvg, st) || attend(m, l, w, b, st) ||
            product(m, &w->wo, m->att, m->ld_att, rows, m->y, m->ld_y, st) || join(m, w->norm1b, l->ff ? w->norm2 : next, NULL, rows, st))
            return -1;
        if (!l->ff) continue;
        if (l->experts ? expert_layer(m, l, w, rows, &plan, st) : feed_forward(m, l, w, rows, st)) return -1;
        if (join(m, w->norm2b, next, l->experts ? &plan : NULL, rows, st)) return -1;
    }
    return 0;
}

static int layered_head(void* model, const int* d_rows, int n, float* d_logits, void* st) {
    const Layered* m = (const Layered*)model;
    DEV(cmlb200_residual_norm(m->x, NULL, 0, NULL, m->final_norm, m->eps, n, m->width, d_rows, m->h, m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16, m->ld_h, st));
    return product(m, &m->head, m->h, m->ld_h, n, d_logits, m->vocab, st);
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
        void* bufs[] = {w->wqkvg.w, w->wo.w, w->wgu.w, w->wd.w, w->norm1, w->norm1b, w->norm2, w->norm2b, w->q_norm, w->k_norm, w->slopes, w->c_norm, w->coef,
                        w->wukt, w->wukv.w, w->router.w, w->experts_gu.w, w->experts_down.w, l->freq, l->attn.k_pool, l->attn.v_pool,
                        l->kv_from == i ? l->lat.pool : NULL};
        for (size_t k = 0; k < sizeof bufs / sizeof bufs[0]; k++) cmlb200_free(bufs[k]);
    }
    const cmlb200_moe* p = &m->plan;
    void* bufs[] = {m->embed, m->freq, m->final_norm, m->head.w, m->x, m->qkvg, m->y, m->gu, m->h, m->att, m->f, m->q, m->o, m->expand_table, m->expand_k,
                    m->expand_v, m->expand_c, m->xp, m->router, p->ids, p->weight, p->pos, p->src, p->expert, p->start, p->count, p->active, p->num_active,
                    p->tiles, p->num_tiles};
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
        if (!rc && m->layers[i].kind->latent) rc = make_rotation(&m->layers[i]);
    }
    cml_safetensors_close(st);
    if (rc || make_activations(m, options->max_step_rows)) { layered_free(m); return NULL; }
    info->vocab = m->vocab;
    for (int i = 0; i < m->num_layers; i++) {
        const int window = window_of(&m->layers[i]);
        if (window <= 0) { info->window = 0; break; }
        if (window > info->window) info->window = window;
    }
    return m;
}

#define LAYERED_CLASS(name) {.architecture = name, .load = layered_load, .free = layered_free, .make_pools = layered_make_pools, .forward = layered_forward, \
                             .head = layered_head, .check = layered_check}
static const CMLLMClass kLayeredClasses[] = {LAYERED_CLASS("Rarolorn"), LAYERED_CLASS("Situlorn")};

__attribute__((constructor)) static void register_layered(void) {
    for (size_t i = 0; i < sizeof kLayeredClasses / sizeof kLayeredClasses[0]; i++) cml_lm_register(&kLayeredClasses[i]);
}
