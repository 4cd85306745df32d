/* C ABI of libllvq_dense.so: the kernels of models whose weights are dense (bf16 or f32), beside the archive-code
 * library of llvq_b200.h. Conventions are the same: every entry point validates its arguments, records a message
 * (llvq_dn_last_error) and returns 0 or a negative status of llvq_b200.h; all pointers are device memory unless a
 * comment says otherwise; work is issued on `stream` and not synchronised. Sizes are elements.
 *
 * Element types: LLVQ_DN_F32 (everything in 32-bit) and LLVQ_DN_BF16 (weights, prompt activations and caches in
 * bf16; norms, rotations, scores, softmax and the residual stream in f32). Matrices are row-major [out, ld] with
 * ld a multiple of a 16-byte vector (8 bf16, 4 f32) and zeros beyond the row's length; norm weights are f32
 * factors as applied. */
#ifndef LLVQ_DENSE_H
#define LLVQ_DENSE_H
#include <stddef.h>
#include <stdint.h>
#ifdef __cplusplus
extern "C" {
#endif

enum { LLVQ_DN_F32 = 0, LLVQ_DN_BF16 = 1 };
typedef void* llvq_dn_stream;

const char* llvq_dn_last_error(void);
uint64_t llvq_dn_launch_count(void);
/* Read and clear the error word of the current device (synchronises): bit 0 = a kernel's bounded wait ran out. */
int llvq_dn_poll_error(int32_t* out);
/* Programmatic overlap of consecutive launches (on by default). */
int llvq_dn_set_overlap(int32_t on);

/* ---- one token: y = W a + bias with the activation formed in the kernel ---- */
enum {
    LLVQ_DN_PLAIN = 0, /* a = x */
    LLVQ_DN_EMBED = 1, /* a = scale * table[*token] */
    LLVQ_DN_NORM = 2   /* t = alpha x + delta (with a table: t = scale * table[*token]); a = t / sqrt(mean(t^2) + eps) * norm_w */
};
typedef struct {
    int32_t dtype, prologue;
    int32_t glu;            /* rows are (gate, up) pairs: y[i] = g sigmoid(gain g) (u + shift), g = min(gate_i, limit), u = clamp(up_i, +-limit) */
    int32_t n_out, k, ldw;
    int32_t ld_table, table_rows;
    float alpha, eps, scale, limit, gain, shift;
    float softcap;          /* llvq_dn_head only: logits <- softcap * tanh(logits / softcap); 0 = none */
    const void* w;
    const float* bias;      /* or NULL */
    float* y;               /* [n_out], or [n_out / 2] with glu; llvq_dn_head: the logits, may be NULL */
    const float* x;
    const float* delta;     /* or NULL */
    const float* norm_w;
    float* a_out;           /* EMBED, NORM: the activation is also stored here (or NULL); not x itself */
    const void* table;      /* EMBED; NORM: or NULL */
    const int64_t* token;   /* with a table or a route */
    /* The rest may be zero. */
    float glu_scale;        /* times the gated unit; 0 = 1 */
    int32_t rows2, glu2;    /* NORM: second rows over the same t, [rows2, ldw]; glu2: they are (gate, up) pairs */
    int32_t k_r, ld_r;      /* PLAIN: routed columns (w_r) */
    int32_t route_rows, top, matrices;
    const float* residual;  /* [n_out] added to y (may be y), not with glu */
    float* t_out;           /* NORM: t (not x itself) */
    const void* w2;         /* routed: the stack [matrices, rows2 / top, ldw]: rows of matrix route[*token][j] follow one another */
    const float* norm_w2;
    float* y2;              /* [rows2], or [rows2 / 2] with glu2 */
    const void* w_r;        /* [matrices, n_out, ld_r]: y += sum_j w_r[route[*token][j]] x_j, x_j the k_r values at x + ldw + j ld_r;
                               with it w may be NULL and k, ldw 0 */
    const int32_t* route;   /* [route_rows, top], or NULL: nothing is routed */
} llvq_dn_gemv_desc;
int llvq_dn_gemv(const llvq_dn_gemv_desc* d, llvq_dn_stream stream);
/* The same over the vocabulary rows, with the greedy pick: best logit and its row (the lowest row on ties).
 * scratch: 8192 bytes. */
int llvq_dn_head(const llvq_dn_gemv_desc* d, void* scratch, float* val_out, int64_t* idx_out, llvq_dn_stream stream);

/* ---- latent attention ---- */
typedef struct {
    int32_t dtype;
    int32_t heads, dim, rot_dim, vdim, kv_rank; /* per head: dim unrotated and rot_dim rotated key dimensions, vdim values */
    int32_t ldk;                 /* row stride of uk and uv */
    int32_t slots, ld;           /* ring of cached rows [latent kv_rank | rotated rot_dim | zeros], position p in slot p % slots */
    int32_t rot_dims;            /* rotated dimensions of the rotated part (even); tables are [positions, rot_dims / 2] */
    int32_t window;              /* visible positions including the token itself */
    int32_t splits;
    float scale, eps;
    void* ring;
    const float* cos_t;
    const float* sin_t;
    const void* uk;              /* [heads * dim, ldk] */
    const void* uv;              /* [heads * vdim, ldk] */
    const float* kv_norm;        /* [kv_rank] */
    const float* sink;           /* [heads] or NULL */
    float* qlat;                 /* scratch [heads, ld] */
    float* part;                 /* scratch [heads * splits * (kv_rank + 2)] */
} llvq_dn_latent;
/* q [heads * (dim + rot_dim)] of the token at *pos into qlat; with y_kv [kv_rank + rot_dim] (its down projection) the
 * token's row is stored into the ring, without it the ring already holds it. */
int llvq_dn_latent_query(const llvq_dn_latent* a, const float* q, const float* y_kv, const int64_t* pos, llvq_dn_stream stream);
/* Attention of qlat over the ring: partial results per split. */
int llvq_dn_latent_decode(const llvq_dn_latent* a, const int64_t* pos, llvq_dn_stream stream);
/* Partial results -> ctx [heads * vdim]. */
int llvq_dn_latent_value(const llvq_dn_latent* a, float* ctx, llvq_dn_stream stream);

/* Attention of a prompt portion: q [n_q, heads * (dim + rot_dim)] before rotation, kv [n_k, ld_kv] = expanded
 * [heads * dim keys | heads * vdim values], kr [n_k, ld_kr] rotated key parts; query i is position pos0 + i, key j
 * position key0 + j. out [n_q, heads * vdim]. Reads window, scale, sink, rot_dims, tables and sizes of `a`.
 * vt: NULL, or, where llvq_dn_latent_prefill_transposes says 1 (the tcgen05 kernel serves the portion), the values apart
 * and transposed, [heads * vdim, ld_vt], ld_vt a multiple of 8 and zeros from n_k to the next one; kv then holds keys only.
 * kernel: 0 = by size and type, 1 = the generic one. */
int llvq_dn_latent_prefill_transposes(const llvq_dn_latent* a, int32_t n_q);
int llvq_dn_latent_prefill(const llvq_dn_latent* a, const void* q, const void* kv, int32_t ld_kv, const void* kr, int32_t ld_kr,
                           const void* vt, int32_t ld_vt, int32_t n_q, int32_t n_k, int64_t pos0, int64_t key0, void* out, int32_t kernel,
                           llvq_dn_stream stream);

/* ---- rows of a prompt portion ---- */
int llvq_dn_embed_rows(int32_t dtype, const void* table, int32_t ld, int32_t table_rows, const int64_t* tokens, int32_t rows, int32_t n,
                       float scale, float* x, void* xt, llvq_dn_stream stream);
/* t = alpha x + y (+ bias); out = t / sqrt(mean(t^2) + eps) * w as f32 and as the element type (either may be NULL). */
int llvq_dn_postnorm_rows(int32_t dtype, const float* x, const void* y, const float* bias, const float* w, float alpha, float eps,
                          void* xt, float* out, int32_t rows, int32_t n, llvq_dn_stream stream);
/* y [rows, ldy] = [q_rank | kv_rank | rot_dim]: the query latent normed into cq [rows, q_rank]; with store_kv the cache
 * rows of positions pos0 .. pos0 + rows - 1 (rows <= slots). */
int llvq_dn_latent_rows(const llvq_dn_latent* a, const void* y, int32_t ldy, int32_t q_rank, const float* q_norm, void* cq,
                        int64_t pos0, int32_t rows, int32_t store_kv, llvq_dn_stream stream);
/* gate_up and bias in (gate, up) pairs: [rows, n, 2] and [n, 2] -> [rows, n]. */
int llvq_dn_glu_rows(int32_t dtype, const void* gate_up, const float* bias, void* out, int32_t rows, int32_t n, float limit, float gain,
                     float shift, llvq_dn_stream stream);
/* The same into rows of stride ld_out, times `scale`. */
int llvq_dn_gated_rows(int32_t dtype, const void* gate_up, const float* bias, void* out, int32_t ld_out, int32_t rows, int32_t n, float limit, float gain,
                       float shift, float scale, llvq_dn_stream stream);
/* x += y (+ sum of rows places[row * top ..] of `routed`); h1, h2 = the sum's norms with weights w1, w2. y, routed, (w1, h1) and
 * (w2, h2) may be NULL. */
int llvq_dn_add_norms_rows(int32_t dtype, float* x, const void* y, const void* routed, const int32_t* places, int32_t top, const float* w1, void* h1,
                           const float* w2, void* h2, float eps, int32_t rows, int32_t n, llvq_dn_stream stream);
int llvq_dn_softcap(float* y, size_t n, float cap, llvq_dn_stream stream);

/* ---- grouped-query attention with normed queries and keys, windowed ---- */
typedef struct {
    int32_t dtype;
    int32_t heads, kv_heads, dim, vdim;
    int32_t slots, ld, kd, vd;   /* ring rows [kv_heads * kd keys | kv_heads * vd values]: heads padded with zeros to whole 16-byte vectors */
    int32_t window, splits;      /* visible positions including the token itself; splits of the token step (at most 128) */
    float scale, eps, out_scale; /* out_scale: times the token step's result */
    void* ring;                  /* position p in slot p % slots */
    const float* q_norm;         /* [dim] */
    const float* k_norm;
    const float* q;              /* token step: projections of the token */
    const float* k;
    const float* v;
    const float* gate;           /* [heads * vdim], sigmoid applied here; or NULL */
    float* part;                 /* scratch [heads * splits * (vdim + 2)] */
    uint32_t* arrived;           /* scratch [kv_heads * ceil(heads / kv_heads / 4)], zero before the first call */
    float* out;                  /* [heads * vdim] */
} llvq_dn_gqa;
/* ---- real-gated linear recurrence behind a short convolution ---- */
typedef struct {
    int32_t dtype;
    int32_t blocks, n, taps, ldw; /* width = blocks * n */
    float out_scale;
    const float* conv_w;         /* [width, taps], last column the current token's */
    const float* conv_b;
    const float* b;              /* [blocks, 2 n]: biases of r, then of i */
    const float* lam;            /* [width]: softplus of the stored value */
    float* conv;                 /* [taps, width]: input of position p in row p % taps */
    float* state;                /* [2, width]: state before position p in half p % 2 */
    const void* w;               /* [blocks, 2 n, ldw]: rows of Ra, then of Ri */
    const float* x;              /* token step: input of the convolution, gate branch before gelu */
    const float* y;
    float* out;
} llvq_dn_lru;
/* The token at *pos through either mixer, or both side by side in one launch. Running it again at the same position with
 * the same inputs changes nothing; position 0 starts from an empty state. */
int llvq_dn_mixer_token(const llvq_dn_gqa* a, const llvq_dn_lru* r, const int64_t* pos, llvq_dn_stream stream);

/* A portion's rows of one product (stride ldy): queries normed into qn [rows, heads * dim], keys and values of positions
 * pos0 .. into the ring. */
int llvq_dn_gqa_rows(const llvq_dn_gqa* a, const void* q, const void* k, const void* v, int32_t ldy, void* qn, int64_t pos0, int32_t rows, llvq_dn_stream stream);
/* Attention of a portion: query i is position pos0 + i, row j of `rows` (laid out as the ring's) position key0 + j; out [n_q, heads * vdim].
 * vt: NULL, or, where ..._transposes says 1, the values transposed, [kv_heads * vdim, ld_vt], zeros from n_k to the next multiple of 8. */
int llvq_dn_gqa_prefill_transposes(const llvq_dn_gqa* a, int32_t n_q);
int llvq_dn_gqa_prefill(const llvq_dn_gqa* a, const void* qn, const void* rows, const void* vt, int32_t ld_vt, int32_t n_q, int32_t n_k, int64_t pos0,
                        int64_t key0, void* out, int32_t kernel, llvq_dn_stream stream);
/* out = x * sigmoid(gate) * scale, row strides ldx, ldg, ldo. */
int llvq_dn_gate_rows(int32_t dtype, const void* x, int32_t ldx, const void* gate, int32_t ldg, void* out, int32_t ldo, int32_t rows, int32_t n, float scale,
                      llvq_dn_stream stream);

/* Causal convolution per channel over x + x_bias (rows of stride ldx), its past from `ring`; then (a call of its own, behind every
 * reader) the last taps inputs into the ring. */
int llvq_dn_conv_rows(int32_t dtype, const void* x, int32_t ldx, const float* x_bias, const float* w, const float* bias, const float* ring, void* out,
                      int32_t channels, int32_t taps, int64_t pos0, int32_t rows, llvq_dn_stream stream);
int llvq_dn_conv_keep(int32_t dtype, const void* x, int32_t ldx, const float* x_bias, float* ring, int32_t channels, int32_t taps, int64_t pos0, int32_t rows,
                      llvq_dn_stream stream);
/* u [rows, width] of conv_rows, z [blocks, rows, 2 n] = the gate matrices times u in f32, y [rows, ldy]: out = S gelu(y + y_bias) out_scale. */
int llvq_dn_lru_rows(const llvq_dn_lru* a, const void* u, const float* z, const void* y, int32_t ldy, const float* y_bias, void* out, int32_t ldo, int64_t pos0,
                     int32_t rows, llvq_dn_stream stream);

/* A portion's rows by expert: table [table_rows, top] names each token's. Place i of the sorted list (by expert, then by row) belongs to
 * row source[i]; places[row * top + j] is where choice j of a row sits; ends[e] is the end of expert e's places. */
int llvq_dn_route_rows(const int32_t* table, int32_t table_rows, int32_t top, int32_t experts, const int64_t* tokens, int32_t rows, int32_t* source,
                       int32_t* places, int32_t* ends, llvq_dn_stream stream);

/* ---- gated delta rule ---- */
typedef struct {
    int32_t dtype;
    int32_t heads, kv_heads, dim, vdim, vp, taps; /* vp: vdim in whole vectors of 4 */
    float eps;
    const float* conv_w;         /* [channels, taps], channels = [kv_heads * dim q | kv_heads * dim k | heads * vdim v] */
    const float* decay;          /* [heads]: exp(A_log) */
    const float* dt_bias;
    const float* norm;           /* [vdim] */
    float* conv;                 /* [taps, channels], as llvq_dn_lru */
    float* state;                /* [2, heads, dim, vp], as llvq_dn_lru; zero beyond vdim */
    const float* x;              /* token step: [channels] */
    const float* gate;           /* [heads * vdim], silu applied here */
    const float* beta;           /* [heads] before the sigmoid */
    const float* alpha;          /* [heads]: added to dt_bias */
    float* o;                    /* scratch [heads * vp] */
    uint32_t* arrived;           /* scratch [heads], zero before the first call */
    float* out;                  /* [heads * vdim] */
} llvq_dn_delta;
int llvq_dn_delta_token(const llvq_dn_delta* a, const int64_t* pos, llvq_dn_stream stream);
/* x rows [channels], ba [rows, 2 heads] f32 (beta, then alpha), gate rows [heads * vdim] -> out rows [heads * vdim]. */
int llvq_dn_delta_scratch(const llvq_dn_delta* a, int32_t rows, size_t* floats);
int llvq_dn_delta_rows(const llvq_dn_delta* a, const void* x, int32_t ldx, const float* ba, const void* gate, int32_t ldg, float* scratch, void* out, int32_t ldo,
                       int64_t pos0, int32_t rows, llvq_dn_stream stream);

#ifdef __cplusplus
}
#endif
#endif /* LLVQ_DENSE_H */
