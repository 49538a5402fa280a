/*
 * vesper_b200 -- C ABI of the operators of hybrid decoders: latent attention with a sliding window and
 * sinks, sigmoid attention with mixed heads, the Mamba-2 and the per-channel selective state-space mixers,
 * mixtures of experts, and the embedding / norm / looped-layer steps that go with them.  Same conventions as vesper_b200.h: every pointer is borrowed device memory, nothing is
 * allocated or freed, launches are asynchronous on the caller's stream, the return value is VB200_OK or
 * a negative vb200_status.
 *
 * Number formats: `dtype` VB200_BF16 keeps weights and activations in bf16 with fp32 accumulation;
 * VB200_F32 keeps everything in fp32 (CUDA cores, no reduced-precision products).  In both, positions,
 * angles, attention scores and weights, norms, the residual stream, step sizes, decays and the recurrent
 * state are fp32 (angles: fp64 product, reduced before the fp32 sine).
 *
 * Per-sequence state lives in slots: `slots` [B] int32 maps the rows of a call to slots, NULL = row b is
 * slot b.  `pos` [B] int32 is the position of each row's first token (what vb200_embed_sequence writes to
 * step_pos).  A sequence at position 0 ignores whatever its slot holds, so a slot can be reused at once.
 */
#ifndef VESPER_B200_HYBRID_H
#define VESPER_B200_HYBRID_H

#include "vesper_b200_block.h"

#ifdef __cplusplus
extern "C" {
#endif

/* ---- embedding of a step --------------------------------------------------------------------------
 * h[m, :] = table[id] (+ bigram[row]) (+ add), row = (previous id * mul_prev + id * mul_cur) mod buckets, or
 * `buckets` (the last row) for the first token of a sequence.  embed_copy (nullable) receives h before
 * `add`.  scaled_out (nullable, bf16) = bf16(h * scale): the producer half of a deferred RMSNorm (scale NULL = 1).
 * Also advances the sequences: step_pos[b] = lens[b]; lens[b] += T; prev[slot] = last id of the row. */
typedef struct vb200_embed_args {
    size_t struct_size;
    int32_t device;
    void* stream;
    int32_t dtype;               /* of the tables */
    const int32_t* ids;          /* [B, T] */
    int32_t B, T, dim, vocab;
    const void* table;           /* [vocab, dim] */
    const void* bigram;          /* [buckets + 1, dim] or NULL */
    int64_t buckets, mul_prev, mul_cur;
    const int32_t* slots;
    int32_t* lens;               /* [B] */
    int32_t* step_pos;           /* [B] out */
    int32_t* prev;               /* [slots] */
    float* h;                    /* [B*T, dim] fp32 */
    float* embed_copy;           /* nullable */
    const float* add;            /* [dim] or NULL */
    const float* scale;          /* [dim] or NULL */
    void* scaled_out;            /* [B*T, dim] bf16 or NULL */
} vb200_embed_args;
int vb200_embed_sequence(const vb200_embed_args* a);

/* h += addend (nullable) + vec (nullable), and scaled_out (nullable) = bf16(h * scale): re-entry into a looped
 * range of layers as a launch of its own. */
int vb200_residual_add(int device, void* stream, float* h, const float* addend, const float* vec, int32_t M, int32_t dim,
                       const float* scale, void* scaled_out);

/* out = x / sqrt(mean(x^2) + eps) * w in fp32 (x, out [M, dim] contiguous); mean over `count` columns (padding holds zeros). */
int vb200_rms_norm_f32(int device, void* stream, const float* x, const float* w, float* out, int32_t M, int32_t dim, int32_t count, float eps);

/* The end of a sublayer whose output is normed: x[m, :] += y[m, :] / sqrt(mean(y^2) + eps) * w (all fp32, rows of `dim` columns, mean
 * over `count`).  With `gather` the row normed is y[m, :] + sum_k rows[gather[m * n_gather + k], :] (bf16 rows, row stride dim; y nullable
 * then).  copy_out (nullable, bf16) = bf16(x * scale), scale nullable: the next sublayer's operand. */
typedef struct vb200_norm_add_args {
    size_t struct_size;
    int32_t device;
    void* stream;
    int32_t M, dim, count;
    float eps;
    float* x;                    /* [M, dim] */
    const float* y;              /* [M, dim] or NULL with gather */
    const float* w;              /* [dim] */
    const void* rows;            /* bf16 */
    const int32_t* gather;       /* [M, n_gather] or NULL */
    int32_t n_gather;
    const float* scale;          /* [dim] or NULL */
    void* copy_out;              /* [M, dim] bf16 or NULL */
} vb200_norm_add_args;
int vb200_norm_add(const vb200_norm_add_args* a);

/* fp32 y = x W^T with the epilogues of vb200_linear (VB200_EPI_F32, VB200_EPI_ADD_F32, VB200_EPI_RELU2, and the gated ones), bias [N] and
 * addend [M, N] (row stride ldo) nullable, added before the epilogue's own step. */
int vb200_linear_f32_ex(int device, void* stream, const float* x, int64_t ldx, const float* w, int64_t ldw, const float* bias,
                        const float* addend, float* out, int64_t ldo, int32_t M, int32_t N, int32_t K, int32_t epilogue);

/* ---- latent attention ------------------------------------------------------------------------------
 * Per token: q [H, dim + rot_dim] (last rot_dim rotated), a latent c [rank] (RMS-normed) and one rotated key part
 * [rot_dim] shared by all heads.  Key of head h = [W_uk_h c, rotated part], value = W_uv_h c, scores scaled by
 * `scale`; query i sees the keys j with 0 <= i - j < window; the softmax denominator also holds exp(sink_h).
 * Rotation: dimension i of the part pairs with i + rot_dim/2, angle = position * inv_freq[i].
 *
 * Cache: ring [slots, ring, ldc] of rows [c | zero pad | rotated part | zero pad], the part at column
 * vb200_latent_rot_offset(rank); position p lives in row p mod ring, ring = the window (or the longest sequence if
 * that is shorter). */
static inline int32_t vb200_latent_rot_offset(int32_t rank) { return (rank + 7) / 8 * 8; }
static inline int32_t vb200_latent_row(int32_t rank, int32_t rot_dim) { return (rank + 7) / 8 * 8 + (rot_dim + 7) / 8 * 8; }

typedef struct vb200_latent_args {
    size_t struct_size;
    int32_t device;
    void* stream;
    int32_t dtype;
    int32_t B, T, H, dim, rot_dim, vdim, rank;
    int32_t window, ring;
    float scale, eps;
    const double* inv_freq;      /* device [rot_dim / 2] */
    void* proj;  int64_t ldp;    /* [B*T, ldp]: q [H * (dim + rot_dim)] | c before its norm [rank] | key part before rotation [rot_dim];
                                    a prompt pass rotates q in place */
    const float* c_norm;         /* [rank] */
    const void* w_uk;            /* [H * dim, ldu] */
    const void* w_uv;            /* [H * vdim, ldu] */
    int64_t ldu;                 /* >= rank, multiple of 8, columns past rank zero */
    const float* sink;           /* [H] or NULL */
    const int32_t* slots;
    const int32_t* pos;          /* [B] */
    void* cache; int64_t ldc;    /* ring of every slot; ldc = vb200_latent_row() */
    void* out;   int64_t ldo;    /* [B*T, H * vdim], heads merged */
    /* prompt pass (T > 1): all rows start at start_pos; workspace: latent rows and expanded keys / values of the context */
    int32_t start_pos;
    void* ctx_latent;            /* [B, n_ctx, ldc] */
    void* ctx_kv; int64_t ldkv;  /* [B, n_ctx, H * (dim + vdim)]: keys then values; filled by the caller between the two calls */
    /* decode (T == 1) */
    int32_t max_len;             /* longest sequence length the step can meet (0 = ring): plans the key splits */
    void* workspace; size_t workspace_bytes;
} vb200_latent_args;

/* Context rows a prompt pass attends to: min(start_pos, window - 1) earlier ones and the T new ones. */
static inline int32_t vb200_latent_context(int32_t start_pos, int32_t T, int32_t window) {
    return (start_pos < window - 1 ? start_pos : window - 1) + T;
}
size_t vb200_latent_workspace_bytes(const vb200_latent_args* a);
/* Prompt pass, first call: norm and rotation of the new latents, rotation of q, the ring update, and ctx_latent. */
int vb200_latent_append(const vb200_latent_args* a);
/* Prompt pass, second call: attention over ctx_kv (expanded by the caller from ctx_latent with the stacked [W_uk; W_uv]). */
int vb200_latent_prefill(const vb200_latent_args* a);
/* One token per row in the absorbed form: q' = W_uk_h^T q, attention over the latents themselves, then W_uv_h. */
int vb200_latent_decode(const vb200_latent_args* a);
/* Name of the attention kernel the calling thread's last prefill / decode call launched. */
const char* vb200_last_latent_kernel(void);

/* ---- Mamba-2 mixer ---------------------------------------------------------------------------------
 * proj row: [z: H*P | x: H*P | B: G*N | C: G*N | dt: H].  x, B, C pass a causal depthwise convolution (taps, bias) and silu;
 * dt = softplus(dt + dt_bias); head h (group h / (H/G)):  S = exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x.
 * out = rmsnorm over norm_groups equal parts of (y * silu(z)), times norm_w.
 * State: conv ring [slots, taps, channels] (input of position p in row p mod taps; channels = H*P + 2*G*N) in `dtype`,
 * and S [slots, H, N, Pp] fp32, Pp = P rounded up to 4, padding zero. */
typedef struct vb200_ssd_args {
    size_t struct_size;
    int32_t device;
    void* stream;
    int32_t dtype;
    int32_t B, T, H, P, N, G, taps, norm_groups;
    float eps;
    const void* proj; int64_t ldp;
    const float* conv_w;         /* [channels, taps] */
    const float* conv_b;         /* [channels] */
    const float* dt_bias;        /* [H] */
    const float* A_log;          /* [H] */
    const float* D;              /* [H] */
    const float* norm_w;         /* [H * P] */
    const int32_t* slots;
    const int32_t* pos;
    void* conv_state;
    float* state;
    void* out; int64_t ldo;      /* [B*T, H * P] */
    void* workspace; size_t workspace_bytes;
    int32_t form;                /* 0 = choose, 1 = token by token, 2 = chunked (bf16), 3 = chunked with warp-level products only */
} vb200_ssd_args;
size_t vb200_ssd_workspace_bytes(const vb200_ssd_args* a);
int vb200_ssd_forward(const vb200_ssd_args* a);
/* Name of the recurrence kernel the calling thread's last vb200_ssd_forward launched. */
const char* vb200_last_ssd_kernel(void);

/* ---- sigmoid attention with mixed heads --------------------------------------------------------------
 * H query heads, G key / value heads, query head g in the group floor(g / (H/G)).  Queries and keys are divided by their
 * root mean square per head; the query at position p is multiplied by 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)
 * (temp_every 0: not).  With n = i - j >= 0,
 *   s_g = scale * q_g . k_group(g),   weight_h = sigmoid( sum_g talk[h, g] s_g + bias[h, min(n, n_bias - 1)] ),
 *   out_h = sigmoid(gate_h) * sum_j weight_h v_group(h)        (weights are not normalised)
 * `bias` holds everything that depends on head and distance only (a mixed relative bias, a per-head offset).
 * Heads are mixed before the product with the keys: q'[h, group, :] = scale * sum_{g in group} talk[h, g] q_g turns the
 * score into one dot product of q'_h with the concatenated keys of a position.
 * Values: value_role 1 stores the step's values to first_values, 2 replaces v by (1 - lambda) v + lambda * first_values.
 * Cache: k [slots, cap, ldk] rows of G * dim normed keys, v [slots, cap, ldv] rows of G * vdim values. */
typedef struct vb200_sigattn_args {
    size_t struct_size;
    int32_t device;
    void* stream;
    int32_t dtype;
    int32_t B, T, H, G, dim, vdim;
    float scale, eps;
    float temp_coef; int32_t temp_every;
    const void* proj;  int64_t ldp;  /* [B*T, ldp]: q [H * dim] | k [G * dim] | v [G * vdim] | gate [H] */
    const float* talk;               /* [H, H] */
    const float* bias;               /* [H, n_bias] */
    int32_t n_bias;
    int32_t value_role;
    float lambda;
    void* first_values;              /* [B*T, G * vdim], in dtype */
    const int32_t* slots;
    const int32_t* pos;              /* [B] */
    void* k_cache; int64_t ldk;      /* rows: multiples of 8 elements */
    void* v_cache; int64_t ldv;
    int32_t cap;
    void* out; int64_t ldo;          /* [B*T, H * vdim] */
    int32_t start_pos;               /* all rows' position when T > 1 */
    int32_t max_len;                 /* longest length a one-token step can meet (0 = cap): plans the key splits */
    void* workspace; size_t workspace_bytes;
    int32_t form;                    /* 0 = choose, 1 = CUDA cores, 2 = prompts on single SMs only */
} vb200_sigattn_args;
size_t vb200_sigattn_workspace_bytes(const vb200_sigattn_args* a);
int vb200_sigattn_forward(const vb200_sigattn_args* a);
/* Name of the attention kernel the calling thread's last vb200_sigattn_forward launched. */
const char* vb200_last_sigattn_kernel(void);

/* ---- selective state-space mixer (per channel) -------------------------------------------------------
 * proj row: [x: inner | z: inner].  x passes a causal depthwise convolution (taps, bias) and silu; [dt | B | C] = W_x x with dt of `rank`,
 * B and C of N columns; dt = softplus(W_dt dt + dt_bias) per channel;
 *   S[c, n] = exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,   y_c = sum_n S[c, n] C_n + D_c x_c,   out = y * silu(z).
 * Sizes are padded by the caller: inner, rank and N multiples of 8 (weights of the padding zero: it then stays zero).
 * State: conv ring [slots, taps, inner] in `dtype` and S [slots, inner, N] fp32. */
typedef struct vb200_selective_args {
    size_t struct_size;
    int32_t device;
    void* stream;
    int32_t dtype;
    int32_t B, T, inner, N, rank, taps;
    const void* proj; int64_t ldp;
    const float* conv_w;         /* [inner, taps] */
    const float* conv_b;         /* [inner] */
    const void* w_x;             /* [rank + 2 N, inner] */
    const void* w_dt;            /* [inner, rank] */
    const float* dt_bias;        /* [inner] */
    const float* A;              /* [inner, N], negative */
    const float* D;              /* [inner] */
    const int32_t* slots;
    const int32_t* pos;
    void* conv_state;
    float* state;
    void* out; int64_t ldo;      /* [B*T, inner] */
    void* workspace; size_t workspace_bytes;
} vb200_selective_args;
size_t vb200_selective_workspace_bytes(const vb200_selective_args* a);
int vb200_selective_forward(const vb200_selective_args* a);
/* Name of the recurrence kernel the calling thread's last vb200_selective_forward launched. */
const char* vb200_last_selective_kernel(void);

/* ---- mixture of experts -------------------------------------------------------------------------------
 * s = sigmoid(W_router x) in fp32; experts rank by s + correction.  groups > 0: consecutive experts are put together, as many to each of the
 * groups; groups rank by their best two experts' ranks added up, and experts outside the first `keep` groups are out of the running.
 * The first `top` experts get the weights s / (sum of their s + 1e-20) * scale.
 * y[m, :] = sum of weight * W_down_e (silu(W_gate_e x) * (W_up_e x)), plus the same of the shared expert (if any) with weight 1.
 * Gate and up rows are interleaved (row 2j = gate_j, row 2j + 1 = up_j).
 * Prompts (vb200_moe_rows(a) > 0): y receives the shared expert only, and the weighted outputs of the chosen experts stay as bf16 rows
 * in the workspace, to be added by vb200_norm_add with (rows, gather) from vb200_moe_rows_of. */
typedef struct vb200_moe_args {
    size_t struct_size;
    int32_t device;
    void* stream;
    int32_t dtype;
    int32_t M, dim, ff, ff_shared;           /* dim: row of x and y (multiple of 8); ff_shared 0 = none */
    int32_t experts, top, groups, keep;
    float scale;
    const void* x;                           /* [M, dim] in dtype */
    const void* w_router;                    /* [experts, dim] in dtype */
    const float* correction;                 /* [experts] or NULL */
    const void* w_in;                        /* [experts, 2 ff, dim] */
    const void* w_out;  int64_t ld_out;      /* [experts, dim, ld_out], ld_out = ff padded to 8 */
    const void* w_shared_in;                 /* [2 ff_shared, dim] */
    const void* w_shared_out; int64_t ld_shared;
    float* y;                                /* [M, dim] fp32 */
    void* workspace; size_t workspace_bytes;
    int32_t form;                            /* 0 = choose, 1 = one token at a time, 2 = grouped by expert (bf16) */
} vb200_moe_args;
size_t vb200_moe_workspace_bytes(const vb200_moe_args* a);
int vb200_moe_forward(const vb200_moe_args* a);
/* Rows per token that a call leaves to vb200_norm_add (0: y is complete), and where they are. */
int32_t vb200_moe_rows(const vb200_moe_args* a);
int vb200_moe_rows_of(const vb200_moe_args* a, const void** rows, const int32_t** gather);
/* The choice alone: ids and weights [M, top] of given logits [M, experts]. */
int vb200_moe_route(int device, void* stream, const float* logits, const float* correction, int32_t M, int32_t experts, int32_t top, int32_t groups, int32_t keep,
                    float scale, int32_t* ids, float* weights);
const char* vb200_last_moe_kernel(void);

#ifdef __cplusplus
}
#endif
#endif /* VESPER_B200_HYBRID_H */
