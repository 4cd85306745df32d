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
    LLVQ_DN_NORM = 2   /* t = alpha x + delta; a = t / sqrt(mean(t^2) + eps) * norm_w */
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
    const void* table;
    const int64_t* token;
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
int llvq_dn_softcap(float* y, size_t n, float cap, llvq_dn_stream stream);

#ifdef __cplusplus
}
#endif
#endif /* LLVQ_DENSE_H */
