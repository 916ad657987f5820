/*
 * vuib200_lm.h - C ABI of libvuib200_lm: token language models (decoder-only, slot cache) on sm_100a.
 *
 * The same conventions as vuib200.h: status codes, borrowed device pointers, the caller's stream and workspace, no
 * device allocation inside the library, one host thread per handle.  A model is a list of layer descriptors, each
 * naming its mechanisms and their constants; a new design combines them in another order or adds one beside them.
 *
 *   mixers   VUIB_LM_MIX_LATENT        latent attention: queries through a normed latent, ONE cached row per position
 *                                      [normed latent c | rotated key part] shared by all heads, interleaved rotation,
 *                                      causal softmax, element-wise sigmoid output gate
 *            VUIB_LM_MIX_GROUPED       grouped-query attention: rotation of component i with i + rot_dims/2, optional RMS norm
 *                                      (no weight) of rotated queries and keys, soft-capped scores, sliding window, biases
 *            VUIB_LM_MIX_DELTA         gated delta rule: short causal convolutions, unit queries and keys, a recurrent
 *                                      matrix per head in 32 bits, output norm and silu gate per head
 *   MLPs     VUIB_LM_MLP_NONE
 *            VUIB_LM_MLP_CLAMPED_GLU   g = min(a, limit), u = clamp(b, +-limit): g * sigmoid(slope g) * (u + shift)
 *            VUIB_LM_MLP_RELU2         relu(a)^2
 *   blocks   VUIB_LM_BLOCK_LN2         parallel, two layer norms: x += mixer(LN1(x)) + mlp(LN2(x))
 *            VUIB_LM_BLOCK_RMS         parallel, one RMS norm: x += mixer(n) + mlp(n), n = RMS(x)
 *
 * Latent layers with the clamped MLP come in the first block, the other mechanisms in the second.  A layer that runs
 * several times in a model is listed several times: every run has its own cache, and all may be given the same weights.
 *
 * dtype 0 stores matrices, activations and cache rows in bf16; dtype 1 stores everything in 32 bits and multiplies
 * in 32 bits.  Residual stream, norms, rotation, scores, softmax weights, gate arguments and logits are 32-bit in both.
 */
#ifndef VUIB200_LM_H
#define VUIB200_LM_H

#include <stddef.h>
#include <stdint.h>

#include "vuib200.h"

#ifdef __cplusplus
extern "C" {
#endif

#define VUIB_LM_ABI_VERSION 2
#define VUIB_LM_MAX_LAYERS 1024

#define VUIB_LM_BF16 0
#define VUIB_LM_F32 1

#define VUIB_LM_MIX_LATENT 1
#define VUIB_LM_MIX_GROUPED 2
#define VUIB_LM_MIX_DELTA 3
#define VUIB_LM_MLP_NONE 0
#define VUIB_LM_MLP_CLAMPED_GLU 1
#define VUIB_LM_MLP_RELU2 2
#define VUIB_LM_BLOCK_LN2 0
#define VUIB_LM_BLOCK_RMS 1

typedef struct VuibLmConfig {
    int32_t vocab, width, n_layers;
    int32_t dtype, block;
    int32_t n_slots;           /* cache slots = max_rows + 1 (spare slot = padding target) */
    int32_t max_seq;           /* positions per slot */
    int32_t max_rows;          /* most rows (streams) of one decode step */
    int32_t max_prefill_rows;  /* most rows (tokens) of one prefill call */
    float norm_eps, embed_scale, logit_scale;
} VuibLmConfig;

/* What a layer is: mechanisms, sizes, constants. */
typedef struct VuibLmLayer {
    int32_t mixer, mlp;
    int32_t heads, kv_heads, dim, rot_dim, rot_dims, vdim, kv_rank, q_rank; /* rot_dims components are rotated: of rot_dim extra ones (latent), of dim (grouped) */
    int32_t window;                             /* grouped: keys a query sees, itself among them; 0: all */
    int32_t qk_norm;                            /* grouped: divide rotated queries and keys by their root mean square */
    int32_t taps;                               /* delta: of the convolutions */
    int32_t ff;
    float scale;                                /* of the attention scores; delta: of the unit query */
    float softcap;                              /* grouped; 0: none */
    float unit_eps;                             /* delta: added to the squared length of queries and keys */
    float mlp_limit, mlp_slope, mlp_shift;
} VuibLmLayer;

/* How the layer's tensors are packed (vuib_lm_layer_dims): matrices row-major [rows, k], rows padded to multiples of
 * 128 and k to multiples of 64, all padding zero. */
typedef struct VuibLmDims {
    int32_t k_in;       /* padded width: K of w_in */
    int32_t n_gate;     /* gate rows of w_in end here */
    int32_t n_mlp;      /* first MLP row of w_in; clamped GLU: unit u has its gate in row n_mlp + 2u, its up row next to it; relu2: its row is n_mlp + u */
    int32_t n_in;       /* rows of w_in */
    int32_t k_out, off_y, n_out; /* w_out: columns [0, off_y) from the mixer's output, [off_y, off_y + ff) from the MLP */
    /* latent */
    int32_t n_dq, n_kv; /* w_in: query-latent rows end at n_dq, [c | rotated] rows at n_kv, gate rows follow */
    int32_t rp, rotp, dp; /* cache row: rp columns of c, rotp rotated, dp in all; dkv rows of w_in have this layout too */
    int32_t k_q, n_q;   /* w_q: n_q >= heads * dp rows; head h has rp rows W_uk[h]^T W_uq[h] (plain part), then rotp rows */
    int32_t x_ok;       /* 1: the layer has an expanded prefill (dtype 0 and sizes within its kernels) */
    int32_t n_xq;       /* w_xq: heads * (dimp + rotp) rows over k_q: the queries themselves */
    int32_t k_kv, n_xkv; /* w_xkv over k_kv columns: heads * dimp key rows, then heads * vdp value rows */
    /* grouped and delta: w_in has queries (grouped: heads, delta: kv_heads) at row 0, kv_heads keys at n_key, values (grouped:
     * kv_heads, delta: heads) at n_value, every head padded to dimp / vdp rows; delta: heads step-size rows at n_ab, then heads
     * decay rows.  The product's 32-bit rows end at n_raw; delta: the gate's heads * vdp rows follow up to n_gate.  Grouped
     * heads keep the two members of a rotated pair next to each other: components 0, r/2, 1, r/2 + 1, ..., then the rest. */
    int32_t dimp, vdp;  /* padded query/key and value sizes of a head (latent: of the expanded form) */
    int32_t n_key, n_value, n_ab, n_raw;
    int32_t cap;        /* grouped: positions of a slot's rings */
    int32_t reserved;
    int64_t off_v;      /* grouped: where a slot's V ring starts, in elements; delta: where the convolution inputs start, in floats */
    int64_t slot_bytes; /* of the layer's cache */
} VuibLmDims;

/* Borrowed device pointers of one layer; matrices in the model's dtype, vectors and tables fp32. */
typedef struct VuibLmLayerWeights {
    const float *norm1_w, *norm1_b, *norm2_w, *norm2_b;  /* (width); RMS blocks: norm1_w alone */
    const float *q_norm, *kv_norm;                       /* (q_rank), (kv_rank) */
    const void *w_in, *w_q, *w_uv, *w_out;               /* w_uv: (heads, vdim, rp) */
    const void *w_xq, *w_xkv;                            /* expanded prefill (NULL when x_ok is 0) */
    const float* trig;                                   /* (max_seq, rot_dims / 2, 2): cos, sin */
    const float *b_in, *b_out;                           /* grouped: (n_raw), (n_out) biases, padded with zeros; may be NULL */
    const float *conv;                                   /* delta: (taps, channels = n_ab), last row for the current token */
    const float *neg_a, *dt_bias, *head_norm;            /* delta: (heads) -exp(A_log), (heads), (vdp) */
} VuibLmLayerWeights;

typedef struct VuibLmHeadWeights {
    const void* embed;        /* (vocab, width), dtype */
    const float *final_w, *final_b;   /* RMS blocks: no final_b */
    const void* head;         /* (vocab padded to 128, k_in), dtype */
} VuibLmHeadWeights;

typedef struct VuibLm VuibLm;

int32_t vuib_lm_abi_version(void);
int32_t vuib_lm_create(const VuibLmConfig* cfg, const VuibLmLayer* layers, VuibLm** out);
int32_t vuib_lm_destroy(VuibLm* e);
int32_t vuib_lm_last_error(VuibLm* e, char* buf, size_t n);
int32_t vuib_lm_layer_dims(VuibLm* e, int32_t layer, VuibLmDims* out);

int32_t vuib_lm_workspace_bytes(VuibLm* e, size_t* bytes);
int32_t vuib_lm_bind_workspace(VuibLm* e, void* dev, size_t bytes);   /* 256-byte aligned, zeroed by the caller */
int32_t vuib_lm_bind_weights(VuibLm* e, const VuibLmHeadWeights* head, const VuibLmLayerWeights* layers);
/* cache[l]: n_slots * slot_bytes of layer l, 16-byte aligned, zeroed once; seq_lens: int32[n_slots].  Recurrent state and
 * rings need no clearing when a slot changes hands: a portion from position 0 does not look at what the slot held. */
int32_t vuib_lm_bind_cache(VuibLm* e, void* const* cache_dev, int32_t* seq_lens_dev);

/* Runs n_segs portions: portion s brings len[s] tokens of slot[s] from position pos[s] on (host arrays); tokens_dev is
 * int64 with the portions one after the other.  Appends to the cache and sets seq_lens[slot] = pos + len.  Logits fp32
 * (n_want, vocab) of the rows want_rows_dev (int32, indices into the call's rows); n_want may be 0.  With delta layers a
 * slot appears once in a call, and pos is its length so far. */
int32_t vuib_lm_prefill(VuibLm* e, int32_t n_segs, const int32_t* slot, const int32_t* pos, const int32_t* len,
                        const int64_t* tokens_dev, int32_t n_want, const int32_t* want_rows_dev, float* logits_out_dev,
                        void* stream);

/* One token for each of B rows at its slot's length; seq_lens[slot] += seq_inc[row] (1 when NULL).  Logits fp32
 * (B, vocab).  Fixed launches: can be captured in a graph and replayed. */
int32_t vuib_lm_decode(VuibLm* e, int32_t B, const int32_t* slots_dev, const int32_t* seq_inc_dev,
                       const int64_t* tokens_dev, float* logits_out_dev, void* stream);

/* Temperature, top_k_cb0, rep_penalty, rep_window and seed of VuibSampling apply to tokens. */
int32_t vuib_lm_set_sampling(VuibLm* e, const VuibSampling* s, void* stream);
/* One draw per row from logits (B, vocab) fp32, which a repetition penalty rewrites; slot's draw counter advances. */
int32_t vuib_lm_sample(VuibLm* e, int32_t B, const int32_t* slots_dev, float* logits_dev, int64_t* tokens_out_dev,
                       void* stream);
/* Clears a slot's draw counter and penalty state (slot -1: all). */
int32_t vuib_lm_reset_slot(VuibLm* e, int32_t slot, void* stream);

/* Optional tap (NULL disables): (n_layers, max(max_rows, max_prefill_rows), width) fp32, the residual rows after every layer. */
int32_t vuib_lm_set_taps(VuibLm* e, float* layer_rows_dev);
/* Portions of at least `rows` rows in all use the prefill forms of the mixers: expanded latent attention, tiled grouped
 * attention, chunked delta rule (0 restores the default, a large value disables them). */
int32_t vuib_lm_set_expand_min(VuibLm* e, int32_t rows);
int32_t vuib_lm_set_wait_limit(VuibLm* e, uint32_t polls);
int32_t vuib_lm_check_device_flag(VuibLm* e, void* stream);
int64_t vuib_lm_launch_count(VuibLm* e);

#ifdef __cplusplus
}
#endif
#endif
