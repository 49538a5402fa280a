/*
 * vesper_b200 -- C ABI of the sequence-mixing operators of hybrid decoders: latent attention with a
 * sliding window and sinks, the Mamba-2 state-space mixer, and the embedding / looped-layer steps that
 * go with them.  Same conventions as vesper_b200.h: every pointer is borrowed device memory, nothing is
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
 * `add`.  scaled_out (nullable, bf16) = bf16(h * scale): the producer half of a deferred RMSNorm.
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
    const float* scale;          /* [dim], with scaled_out */
    void* scaled_out;            /* [B*T, dim] bf16 or NULL */
} vb200_embed_args;
int vb200_embed_sequence(const vb200_embed_args* a);

/* h += addend (nullable) + vec (nullable), and scaled_out (nullable) = bf16(h * scale): re-entry into a looped
 * range of layers as a launch of its own. */
int vb200_residual_add(int device, void* stream, float* h, const float* addend, const float* vec, int32_t M, int32_t dim,
                       const float* scale, void* scaled_out);

/* out = x / sqrt(mean(x^2) + eps) * w in fp32 (x, out [M, dim] contiguous); mean over `count` columns (padding holds zeros). */
int vb200_rms_norm_f32(int device, void* stream, const float* x, const float* w, float* out, int32_t M, int32_t dim, int32_t count, float eps);

/* fp32 y = x W^T with the epilogues of vb200_linear (VB200_EPI_F32, VB200_EPI_ADD_F32, VB200_EPI_RELU2), bias [N] and
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

#ifdef __cplusplus
}
#endif
#endif /* VESPER_B200_HYBRID_H */
