/* Decoder-only models described layer by layer in config.json and stored as safetensors. A design is a row
 * of switches (LayeredDesign below); sizes, windows, scales and the order of layers come from the file.
 *
 *   config.json     architecture, vocab, width, norm.eps, layers: [{type, mixer, mlp, weights_of?}]
 *   mixer           heads, kv_heads, dim, vdim, scale, mask.size, q_temp {coef, every}
 *   mlp             {kind: "dense", ff} or null
 *   weights_of      index of the layer whose tensors this one uses; its cache is its own
 *   tensors         embed, final.norm, head, l<i>.norm1 / norm1b / norm2 / norm2b,
 *                   l<i>.mix.q / k / v / g / o / q.norm / k.norm, l<i>.mlp.gate / up / down; linear weights [out, in]
 *
 * On the device a layer's q, k, v and gate rows are one matrix, and the feed-forward's gate and up rows one
 * matrix interleaved in groups of 16 (the epilogues of both products pair them). Between two sublayers runs
 * one kernel: norm of the finished sublayer's output, residual add, norm for the next one. The residual, norms,
 * scores and weights are fp32; in the bfloat16 form matrix operands are bf16 and cached keys and values
 * fp16. Up to 32 rows a step streams its weights through the decode product, above that tcgen05 tiles. */
#include <math.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include "cml_lm_internal.h"
#include "cml_safetensors.h"

#define SKINNY_ROWS 32
#define MAX_LAYERS 4096
#define DEV(call) do { if (CML_DEV_FAIL((call), __func__)) return -1; } while (0)

typedef struct LayeredDesign {
    const char* architecture;
    double position_base;        /* > 0: sinusoidal position vector with that base added to the embedding */
    int output_norms;            /* each sublayer's output is normed before it joins the residual */
    int wide_qk_norm;            /* RMS norm of the whole q and k projections */
    int linear_bias;             /* scores lose slope_h * distance, slope_h = 2^(-8 (h + 1) / heads) */
    int sink;                    /* one added to the softmax denominator */
    int head_gate;               /* sigmoid gate per head */
    int act;                     /* of the gated feed-forward */
} LayeredDesign;

static const LayeredDesign kDesigns[] = {
    {"Rarolorn", 10000.0, 1, 1, 1, 1, 1, CMLB200_ACT_GELU_TANH},
};

typedef struct LayerWeights {    /* device tensors of a layer that owns some */
    cmlb200_dense wqkvg, wo, wgu, wd;
    float *norm1, *norm1b, *norm2, *norm2b, *q_norm, *k_norm, *slopes;
} LayerWeights;

typedef struct Layer {
    int source;                  /* the layer whose weights it uses */
    int ff;                      /* 0: no feed-forward */
    cmlb200_attn attn;
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
    int max_rows, ld_h, ld_qkvg, ld_att, ld_y, ld_f, ld_gu;
    float *x, *qkvg, *y, *gu;
    void *h, *att, *f;           /* operands of the matrix products: bf16, or fp32 in the 32-bit form */
} Layered;

static int round_up(int v, int to) { return (v + to - 1) / to * to; }

/* ---- configuration ---------------------------------------------------------------------------------- */
static int read_layer(const CMLJson* j, Layer* l, int index, const LayeredDesign* design) {
    const CMLJson *mixer = cml_json_get(j, "mixer"), *mask = cml_json_get(mixer, "mask"), *temp = cml_json_get(mixer, "q_temp"), *mlp = cml_json_get(j, "mlp");
    const char* type = cml_json_string(j, "type");
    cmlb200_attn* a = &l->attn;
    double scale = 0.0, coef = 0.0, every = 0.0;
    if (!type || strcmp(type, "attention")) { LOG_ERROR("layer %d: mixer type '%s' is not known to %s", index, type ? type : "(none)", design->architecture); return -1; }
    if (cml_json_int(mixer, "heads", &a->heads) || cml_json_int(mixer, "kv_heads", &a->kv_heads) || cml_json_int(mixer, "dim", &a->dim) ||
        cml_json_int(mixer, "vdim", &a->vdim) || cml_json_double(mixer, "scale", &scale) || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads ||
        a->dim <= 0 || a->vdim <= 0 || a->heads > 65535 || a->dim > 256 || a->vdim > 256) {
        LOG_ERROR("layer %d: heads, kv_heads, dim, vdim (up to 256) or scale are missing or do not fit", index);
        return -1;
    }
    if (mask && mask->type == CML_JSON_OBJECT && (cml_json_int(mask, "size", &a->window) || a->window <= 0)) { LOG_ERROR("layer %d: mask.size", index); return -1; }
    if (temp && temp->type == CML_JSON_OBJECT && (cml_json_double(temp, "coef", &coef) || cml_json_double(temp, "every", &every) || every <= 0.0)) { LOG_ERROR("layer %d: q_temp", index); return -1; }
    if (mlp && mlp->type == CML_JSON_OBJECT) {
        const char* kind = cml_json_string(mlp, "kind");
        if (!kind || strcmp(kind, "dense") || cml_json_int(mlp, "ff", &l->ff) || l->ff <= 0) { LOG_ERROR("layer %d: feed-forward of kind '%s'", index, kind ? kind : "(none)"); return -1; }
    }
    a->scale = (float)scale;
    a->temp_coef = (float)coef;
    a->temp_every = (float)every;
    a->dim_ld = round_up(a->dim, 16);
    a->vdim_ld = round_up(a->vdim, 16);
    a->sink = design->sink;
    a->gate_col = design->head_gate ? a->heads * a->dim + a->kv_heads * (a->dim + a->vdim) : -1;
    l->source = index;
    int of;
    if (!cml_json_int(j, "weights_of", &of)) l->source = of;
    return 0;
}

static int same_shape(const Layer* a, const Layer* b) {
    return a->attn.heads == b->attn.heads && a->attn.kv_heads == b->attn.kv_heads && a->attn.dim == b->attn.dim && a->attn.vdim == b->attn.vdim && a->ff == b->ff;
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

static int load_layer(Layered* m, const CMLSafetensors* st, int index) {
    Layer* l = &m->layers[index];
    LayerWeights* w = &l->w;
    const cmlb200_attn* a = &l->attn;
    char prefix[32];
    snprintf(prefix, sizeof prefix, "l%d.", index);
    const char* proj[4] = {"mix.q", "mix.k", "mix.v", "mix.g"};
    const int proj_rows[4] = {a->heads * a->dim, a->kv_heads * a->dim, a->kv_heads * a->vdim, a->heads};
    const char *out[1] = {"mix.o"}, *gu[2] = {"mlp.gate", "mlp.up"}, *down[1] = {"mlp.down"};
    const int out_rows[1] = {m->width}, gu_rows[2] = {l->ff, l->ff};
    if (load_vector(st, prefix, "norm1", m->width, &w->norm1) ||
        (m->design->output_norms && load_vector(st, prefix, "norm1b", m->width, &w->norm1b)) ||
        (m->design->wide_qk_norm && (load_vector(st, prefix, "mix.q.norm", proj_rows[0], &w->q_norm) || load_vector(st, prefix, "mix.k.norm", proj_rows[1], &w->k_norm))) ||
        load_matrix(m, st, prefix, proj, proj_rows, m->design->head_gate ? 4 : 3, m->width, 0, &w->wqkvg) ||
        load_matrix(m, st, prefix, out, out_rows, 1, a->heads * a->vdim, 0, &w->wo))
        return -1;
    if (l->ff && (load_vector(st, prefix, "norm2", m->width, &w->norm2) || (m->design->output_norms && load_vector(st, prefix, "norm2b", m->width, &w->norm2b)) ||
                  load_matrix(m, st, prefix, gu, gu_rows, 2, m->width, 1, &w->wgu) || load_matrix(m, st, prefix, down, out_rows, 1, l->ff, 0, &w->wd)))
        return -1;
    if (m->design->linear_bias) {
        float* s = (float*)malloc((size_t)a->heads * sizeof(float));
        if (!s) return -1;
        for (int h = 0; h < a->heads; h++) s[h] = (float)exp2(-8.0 * (h + 1) / a->heads);
        const int rc = upload((void**)&w->slopes, s, (size_t)a->heads * sizeof(float));
        free(s);
        if (rc) return -1;
    }
    return 0;
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

/* Operand buffers have strides that are multiples of 64 and start out zero: the decode product reads up
 * to the padded width, where its weights are zero. */
static int make_activations(Layered* m, int rows) {
    int q = 0, att = 0, ff = 0;
    for (int i = 0; i < m->num_layers; i++) {
        const Layer* l = &m->layers[i];
        const int n = m->layers[l->source].w.wqkvg.rows;
        if (n > q) q = n;
        if (l->attn.heads * l->attn.vdim > att) att = l->attn.heads * l->attn.vdim;
        if (l->ff > ff) ff = l->ff;
    }
    m->max_rows = rows;
    m->ld_h = round_up(m->width, 64);
    m->ld_qkvg = round_up(q, 16);
    m->ld_att = round_up(att, 64);
    m->ld_y = round_up(m->width, 16);
    m->ld_f = round_up(ff ? ff : 1, 64);
    m->ld_gu = 2 * round_up(ff ? ff : 1, 16);
    const size_t R = (size_t)rows, es = m->f32 ? 4 : 2, head = R > 256 ? R : 256;      /* the head normalises up to 256 rows at once into h */
    return zeroed((void**)&m->x, R * (size_t)m->width * 4) || zeroed(&m->h, head * (size_t)m->ld_h * es) || zeroed((void**)&m->qkvg, R * (size_t)m->ld_qkvg * 4) ||
           zeroed(&m->att, R * (size_t)m->ld_att * es) || zeroed((void**)&m->y, R * (size_t)m->ld_y * 4) || zeroed(&m->f, R * (size_t)m->ld_f * es) ||
           (m->f32 && zeroed((void**)&m->gu, R * (size_t)m->ld_gu * 4)) || CML_DEV_FAIL(cmlb200_stream_sync(NULL), "make_activations") ? -1 : 0;
}

static int layered_make_pools(void* model, int blocks, int block_size) {
    Layered* m = (Layered*)model;
    for (int i = 0; i < m->num_layers; i++) {
        cmlb200_attn* a = &m->layers[i].attn;
        const LayerWeights* w = &m->layers[m->layers[i].source].w;
        const size_t es = m->f32 ? 4 : 2, slots = (size_t)blocks * (size_t)block_size * (size_t)a->kv_heads;
        a->cache_dtype = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_F16;
        a->block_size = block_size;
        a->q_norm = w->q_norm;
        a->k_norm = w->k_norm;
        a->eps = m->eps;
        a->slopes = w->slopes;
        if (zeroed(&a->k_pool, slots * (size_t)a->dim_ld * es) || zeroed(&a->v_pool, slots * (size_t)a->vdim_ld * es)) return -1;
    }
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

static int feed_forward(const Layered* m, const Layer* l, const LayerWeights* w, int rows, void* st) {
    const int act = m->design->act;
    if (m->f32) {
        DEV(cmlb200_linear_dense_f32(&w->wgu, (const float*)m->h, m->ld_h, rows, m->gu, m->ld_gu, st));
        DEV(cmlb200_glu_rows_f32(m->gu, m->ld_gu, rows, l->ff, act, (float*)m->f, m->ld_f, st));
    } else if (rows <= SKINNY_ROWS) {
        DEV(cmlb200_gemv_dense_glu(&w->wgu, (const uint16_t*)m->h, m->ld_h, rows, l->ff, act, (uint16_t*)m->f, m->ld_f, st));
    } else {
        DEV(cmlb200_gemm_dense_glu(&w->wgu, (const uint16_t*)m->h, m->ld_h, rows, l->ff, act, (uint16_t*)m->f, m->ld_f, st));
    }
    return product(m, &w->wd, m->f, m->ld_f, rows, m->y, m->ld_y, st);
}

static int attend(const Layered* m, const Layer* l, const CMLLMBatch* b, void* st) {
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

static int layered_forward(void* model, const CMLLMBatch* b, void* st) {
    const Layered* m = (const Layered*)model;
    const int rows = b->rows, out = m->f32 ? CMLB200_DT_F32 : CMLB200_DT_BF16;
    if (rows > m->max_rows) { LOG_ERROR("layered_forward: %d rows of %d", rows, m->max_rows); return -1; }
    DEV(cmlb200_embed_rows(m->embed, out, b->d_tokens, b->d_pos, m->freq, rows, m->width, m->vocab, m->x, st));
    DEV(cmlb200_residual_norm(m->x, NULL, 0, NULL, m->layers[m->layers[0].source].w.norm1, m->eps, rows, m->width, NULL, m->h, out, m->ld_h, st));
    for (int i = 0; i < m->num_layers; i++) {
        const Layer* l = &m->layers[i];
        const LayerWeights* w = &m->layers[l->source].w;
        const float* next = i + 1 < m->num_layers ? m->layers[m->layers[i + 1].source].w.norm1 : NULL;
        if (product(m, &w->wqkvg, m->h, m->ld_h, rows, m->qkvg, m->ld_qkvg, st) || attend(m, l, b, st) ||
            product(m, &w->wo, m->att, m->ld_att, rows, m->y, m->ld_y, st))
            return -1;
        DEV(cmlb200_residual_norm(m->x, m->y, m->ld_y, w->norm1b, l->ff ? w->norm2 : next, m->eps, rows, m->width, NULL, m->h, out, m->ld_h, st));
        if (!l->ff) continue;
        if (feed_forward(m, l, w, rows, st)) return -1;
        DEV(cmlb200_residual_norm(m->x, m->y, m->ld_y, w->norm2b, next, m->eps, rows, m->width, NULL, m->h, out, m->ld_h, st));
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
    if (m->f32 || b->rows <= SKINNY_ROWS) return 0;
    DEV(cmlb200_gemm_dense_status(&status, 1));
    return status ? -1 : 0;
}

/* ---- class --------------------------------------------------------------------------------------------- */
static void layered_free(void* model) {
    Layered* m = (Layered*)model;
    if (!m) return;
    for (int i = 0; m->layers && i < m->num_layers; i++) {
        LayerWeights* w = &m->layers[i].w;
        void* bufs[] = {w->wqkvg.w, w->wo.w, w->wgu.w, w->wd.w, w->norm1, w->norm1b, w->norm2, w->norm2b, w->q_norm, w->k_norm, w->slopes,
                        m->layers[i].attn.k_pool, m->layers[i].attn.v_pool};
        for (size_t k = 0; k < sizeof bufs / sizeof bufs[0]; k++) cmlb200_free(bufs[k]);
    }
    void* bufs[] = {m->embed, m->freq, m->final_norm, m->head.w, m->x, m->qkvg, m->y, m->gu, m->h, m->att, m->f};
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
    char file[4096];
    snprintf(file, sizeof file, "%s/model.safetensors", path);
    CMLSafetensors* st = NULL;
    int rc = read_config(config, m) || !(st = cml_safetensors_open(file)) || load_shared(m, st);
    for (int i = 0; i < m->num_layers && !rc; i++)
        if (m->layers[i].source == i) rc = load_layer(m, st, i);
    cml_safetensors_close(st);
    if (rc || make_activations(m, options->max_step_rows)) { layered_free(m); return NULL; }
    info->vocab = m->vocab;
    for (int i = 0; i < m->num_layers; i++) {
        if (m->layers[i].attn.window <= 0) { info->window = 0; break; }
        if (m->layers[i].attn.window > info->window) info->window = m->layers[i].attn.window;
    }
    return m;
}

static const CMLLMClass kLayeredClass = {.architecture = "Rarolorn", .load = layered_load, .free = layered_free, .make_pools = layered_make_pools,
                                         .forward = layered_forward, .head = layered_head, .check = layered_check};

__attribute__((constructor)) static void register_layered(void) { cml_lm_register(&kLayeredClass); }
