/* What the sources of the layered models share: the description of a design, a layer and a model, and the helpers that
 * load weights and run products. See cml_lm_layered.c. */
#ifndef CML_LM_LAYERED_H
#define CML_LM_LAYERED_H

#include "cml_lm_internal.h"
#include "cml_safetensors.h"

#define SKINNY_ROWS 32
#define EXPERT_ROWS 128            /* row tile of the experts' tensor-core product */
#define MAX_PARTS 16               /* tensors stacked into one matrix at most */
#define DEV(call) do { if (CML_DEV_FAIL((call), __func__)) return -1; } while (0)

/* grouped heads; latent attention; grouped heads beside a recurrence */
typedef enum { MIXER_GROUPED, MIXER_LATENT, MIXER_PARALLEL } MixerForm;
/* beside grouped heads: a gated delta rule, both outputs scaled and added; a minimal gated recurrence, half the sum of both outputs' norms */
typedef enum { BESIDE_DELTA, BESIDE_GRU } Beside;
typedef enum { GATE_NONE, GATE_WIDE, GATE_HEAD } HeadsGate;      /* sigmoid on the heads' output: none, per element, per head */
/* neighbouring entries of queries and keys turn: not at all; with frequencies divided by a factor where the file gives one; or stretched by wavelength */
typedef enum { ROTATE_NONE, ROTATE_LINEAR, ROTATE_BANDS } Rotate;
typedef enum { NORM_NONE, NORM_WIDE, NORM_HEAD } HeadNorm;       /* of q and k: none, over all heads, per head */
typedef enum { SINK_NONE, SINK_ONE, SINK_LEARNED } Sink;         /* what joins the softmax denominator: nothing, one, exp of a number per head */

typedef struct GroupedForm {       /* switches of grouped heads */
    HeadNorm norm;
    Sink sink;
    int linear_bias;               /* scores lose slope_h * distance, slope_h = 2^(-8 (h + 1) / heads) */
    int head_gate;                 /* sigmoid gate per head */
    int chunked;                   /* mask.size is that of chunks counted from position 0; 0: of a window, mask.keep_first tokens kept in sight */
    int in_bias, out_bias;         /* biases of the projections, of the output projection */
    int keys_as_values;            /* no v projection: values are the projected keys before their norm */
    Rotate rotate;
    int conv;                      /* q, k and v are convolved over time */
    int talk;                      /* scores are capped and every head's is a combination of all heads' */
} GroupedForm;

typedef struct MixerKind {
    const char* type;
    MixerForm form;
    HeadsGate gate;                /* latent */
    int q_latent;                  /* latent: queries come out of a normed latent of their own */
    Sink sink;                     /* latent */
    Beside beside;                 /* parallel */
    GroupedForm grouped;
} MixerKind;

typedef enum { FF_GATED, FF_POLY_NORM } DenseForm;
/* not known; softmax scores as they are; scores corrected for the choice, groups, identity experts, weights that sum to a
 * constant, a shared expert; sigmoid scores as they are, groups by their two best, experts without a gate */
typedef enum { EXPERTS_NONE, EXPERTS_PLAIN, EXPERTS_GROUPED, EXPERTS_SIGMOID } ExpertsForm;

typedef struct LayeredDesign {
    const char* architecture;
    MixerKind mixers[3];
    double position_base;          /* > 0: sinusoidal position vector with that base added to the embedding */
    int input_norms;               /* each sublayer reads a normed residual; 0: the residual itself */
    const char* output_norms[2];   /* tensors of the norm on each sublayer's output before it joins the residual; NULL: none */
    float norm_offset;             /* added to the stored weights of the model's norms */
    int streams;                   /* the residual is `streams` streams, read, mixed and written with learned coefficients */
    int side_by_side;              /* mixer and feed-forward read the same normed residual and join it together, each through a gate (rg1, rg2) */
    int loops;                     /* config.json may run a stretch of layers several times */
    DenseForm dense;               /* of a dense feed-forward */
    int act;                       /* of a gated feed-forward, or of the experts */
    ExpertsForm experts;
} LayeredDesign;

typedef struct Sublayer {          /* device tensors around a mixer or feed-forward */
    float *norm, *post;            /* in front of it, on its output */
    float *in, *out, *mix;         /* streams */
} Sublayer;

typedef struct LayerWeights {      /* device tensors of a layer that owns some */
    cmlb200_dense wqkvg, wo, wgu, wd;        /* latent layers: q, dkv and g rows; wgu without a gate: the up rows alone */
    Sublayer sub[2];
    float *q_norm, *k_norm, *slopes, *sinks;
    float *c_norm, *coef;
    void* wukt;                    /* per head, transposed */
    cmlb200_dense wukv;            /* all Wuk rows, then all Wuv rows (per head padded to 16); in the 32-bit form Wuv alone */
    cmlb200_dense router, experts_gu, experts_down, shared_gu, shared_down;
    float* correction;
    /* gated delta rule */
    float *conv, *rate, *dt_bias, *o_norm;
    cmlb200_dense wa, wg;          /* second factors of the decay's and the gate's projections; the first are rows of wqkvg */
    cmlb200_dense wuq, wo2;        /* queries out of their latent; output of a second mixer with a product of its own */
    float *dq_norm, *talk, *left_out, *right_out;
} LayerWeights;

typedef struct Layer {             /* a layer of config.json, or one more pass over it */
    int index;                     /* in config.json */
    int again;                     /* the embedding is added to the residual in front of it */
    int source;                    /* the layer whose weights it uses */
    int ff;                        /* 0: no feed-forward */
    int experts, top;              /* 0: a dense feed-forward; ff is an expert's */
    int identity, groups, keep, shared_ff;
    float limit, router_scale;
    const MixerKind* kind;
    cmlb200_attn attn;
    cmlb200_latent lat;
    cmlb200_delta delta;
    cmlb200_gru gru;
    int q_rank, proj_col;          /* of a queries' latent; the column that the projection's output begins with */
    int gate_cols, router_col;     /* columns of a side-by-side layer: the sublayers' gate logits, the router's */
    int a_rank, g_rank;            /* of the decay's and the gate's projections; their columns follow the beta logits */
    int kv_from;                   /* the layer whose latents it reads: itself, as a rule */
    double rot_base, rot_scaling[4];         /* scaling[0]: factor, 0 without */
    float* freq;
    LayerWeights w;
} Layer;

typedef struct Layered {
    const LayeredDesign* design;
    int f32, vocab, width, num_layers;
    int streams;                   /* 0: one residual, no streams */
    float eps, embed_scale, cap;
    Layer* layers;
    void* embed;
    float *freq, *final_norm;
    cmlb200_dense head;
    int max_rows, max_sequences, ld_h, ld_qkvg, ld_att, ld_y, ld_f, ld_gu;
    float *x, *qkvg, *y, *gu;
    void *h, *att, *f;             /* operands of the matrix products: bf16, or fp32 in the 32-bit form */
    /* latent layers */
    int q_rows;                    /* rows whose queries are transformed at a time */
    void *q, *o;                   /* transformed queries (fp16 or fp32) and weighted latents (bf16 or fp32) */
    int expand_keys, *expand_table;
    void *expand_k, *expand_v, *expand_c;
    int slots, table_ld;
    /* experts */
    cmlb200_moe plan;
    void* xp;
    float *router, *y_shared;
    int ld_router;
    /* gated delta rule */
    int ld_dec, ld_gate, ld_low;
    float *dec, *gate, *delta_work;
    void* low;                     /* packed operand of wa and wg */
    /* side by side */
    float *y_mix, *y_mix2;
    /* queries' latents; convolved queries; scores that are made ahead of attention */
    int ld_cq;
    void *cq, *q_rows_out;
    float* scores;
    size_t scores_room;            /* floats */
    int scores_keys;               /* keys in reach of a row at most */
} Layered;

static inline int lml_round_up(int v, int to) { return (v + to - 1) / to * to; }
static inline int lml_most(int a, int b) { return a > b ? a : b; }

/* Tensor prefix + name of that shape (cols 0: a vector; rows < 0: any number, which t then holds); logs what is wrong with it. */
int lml_find(const CMLSafetensors* st, const char* prefix, const char* name, int rows, int cols, CMLSafetensor* t);
float lml_element(const CMLSafetensor* t, size_t i);
int lml_upload(void** dst, const void* src, size_t bytes);
int lml_load_vector(const CMLSafetensors* st, const char* prefix, const char* name, int n, float offset, float** dst);
/* Stacks [rows, cols] tensors; interleave: two of them in turns of 16 rows, each padded to whole groups. */
int lml_load_matrix(const Layered* m, const CMLSafetensors* st, const char* prefix, const char* const* names, const int* rows, int parts, int cols,
                    int interleave, cmlb200_dense* out);
int lml_zeroed(void** dst, size_t bytes);
/* Stacks tensors [channels of the part, taps] as [taps][channels of all parts]. */
int lml_load_taps(const CMLSafetensors* st, const char* prefix, const char* const* names, const int* channels, int parts, int taps, float** dst);
int lml_product(const Layered* m, const cmlb200_dense* w, const void* x, int ldx, int rows, float* y, int ldy, void* st);

/* cml_lm_delta.c: the gated delta rule of a MIXER_PARALLEL layer. Its projections are rows of wqkvg from column delta.col on, its output
 * columns of the heads' output from column `col` on. */
int cml_delta_read(const CMLJson* mixer, Layer* l, int index, int col);
int cml_delta_ranks(const CMLSafetensors* st, const char* prefix, Layer* l, int width);
int cml_delta_load(Layered* m, const CMLSafetensors* st, const char* prefix, Layer* l);
int cml_delta_activations(Layered* m, int rows);
int cml_delta_make_state(Layered* m, Layer* l, const LayerWeights* w, int slots);
int cml_delta_run(const Layered* m, const Layer* l, const LayerWeights* w, const CMLLMBatch* b, int col, void* st);

/* cml_lm_gru.c: the minimal gated recurrence of a MIXER_PARALLEL layer, projected from column gru.col on. */
int cml_gru_read(const CMLJson* mixer, Layer* l, int index);
int cml_gru_make_state(Layer* l, int slots);
int cml_gru_run(const Layered* m, const Layer* l, const CMLLMBatch* b, int col, void* st);

/* cml_lm_talk.c: grouped heads with scores made ahead of the softmax (cap, talking heads) and projections convolved over time. */
int cml_talk_read(const CMLJson* mixer, Layer* l, int index);
int cml_talk_load(const CMLSafetensors* st, const char* prefix, Layer* l);
int cml_talk_make_state(Layer* l, const LayerWeights* w, int slots);
int cml_talk_make_scores(Layered* m, int slots, int table_ld, int block_size);
int cml_talk_run(const Layered* m, const cmlb200_attn* a, const CMLLMBatch* b, void* st);

#endif
