// C ABI of libllvq_dense.so (include/llvq_dense.h): models with dense bf16 or f32 weights.
#include <cuda_runtime.h>

#include <algorithm>

#include "../../include/llvq_dense.h"
#include "dense_gemv.cuh"
#include "delta_rule.cuh"
#include "dense_rows.cuh"
#include "gqa_attn.cuh"
#include "host_util.cuh"
#include "latent_attn.cuh"
#include "latent_prefill.cuh"
#include "latent_prefill_tc.cuh"
#include "linear_recurrence.cuh"

using namespace llvq;

static_assert(kHeadMaxGrid * sizeof(HeadBest) == 8192, "scratch of llvq_dn_head");

namespace {

constexpr size_t kMaxSmem = 227 * 1024;

bool bad_dtype(int dt) { return dt != LLVQ_DN_F32 && dt != LLVQ_DN_BF16; }
int elem_size(int dt) { return dt == LLVQ_DN_BF16 ? 2 : 4; }

int sm_count() {
    static std::atomic<int> cached{0};
    int n = cached.load();
    if (!n) {
        int dev = 0;
        cudaGetDevice(&dev);
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) n = 148;
        cached = n;
    }
    return n;
}

int check_gemv(const llvq_dn_gemv_desc* d, const char* who) {
    if (!d || bad_dtype(d->dtype)) return fail(kStatusInvalid, "%s: null descriptor or element type", who);
    const int vn = 16 / elem_size(d->dtype);
    const bool routed_only = !d->w && d->w_r && d->k == 0 && d->ldw == 0;
    if (d->n_out <= 0 || (!routed_only && (!d->w || d->k <= 0 || d->ldw < d->k || d->ldw % vn || ((uintptr_t)d->w & 15))))
        return fail(kStatusInvalid, "%s: matrix of %d x %d, row stride %d (a multiple of %d, 16-byte aligned)", who, d->n_out, d->k, d->ldw, vn);
    if (d->glu && d->n_out % 2) return fail(kStatusInvalid, "%s: %d rows are not (gate, up) pairs", who, d->n_out);
    switch (d->prologue) {
        case LLVQ_DN_PLAIN:
            if (!d->x) return fail(kStatusInvalid, "%s: null activation", who);
            break;
        case LLVQ_DN_NORM:
            if ((!d->x && !d->table) || !d->norm_w || (d->x && (d->a_out == d->x || d->t_out == d->x)))
                return fail(kStatusInvalid, "%s: norm needs x, norm_w and another buffer to store to", who);
            if (d->table && (!d->token || d->ld_table < d->ldw || d->ld_table % vn || ((uintptr_t)d->table & 15) || d->table_rows <= 0))
                return fail(kStatusInvalid, "%s: norm of a table row needs a token and rows of %d", who, d->ldw);
            break;
        case LLVQ_DN_EMBED:
            if (!d->table || !d->token || d->ld_table < d->k || d->table_rows <= 0) return fail(kStatusInvalid, "%s: embed needs a table and a token", who);
            break;
        default: return fail(kStatusInvalid, "%s: prologue %d", who, d->prologue);
    }
    if (d->route && (!d->token || d->route_rows <= 0 || d->top <= 0 || d->matrices <= 0 || !(d->rows2 || d->w_r)))
        return fail(kStatusInvalid, "%s: a route of %d matrices of %d", who, d->top, d->matrices);
    if (d->rows2) {
        const int unit = (d->route ? d->top : 1) * (d->glu2 ? 2 : 1);
        if (d->prologue != LLVQ_DN_NORM || d->rows2 < 0 || d->rows2 % unit || !d->w2 || ((uintptr_t)d->w2 & 15) || !d->norm_w2 || !d->y2)
            return fail(kStatusInvalid, "%s: %d second rows", who, d->rows2);
    }
    if (d->w_r && (d->prologue != LLVQ_DN_PLAIN || !d->route || d->k_r <= 0 || d->ld_r < d->k_r || d->ld_r % vn || ((uintptr_t)d->w_r & 15)))
        return fail(kStatusInvalid, "%s: routed columns of %d, row stride %d", who, d->k_r, d->ld_r);
    if (d->residual && d->glu) return fail(kStatusInvalid, "%s: a residual beside a gated unit", who);
    return kStatusOk;
}

__device__ unsigned int g_device_error;  // bits set by kernels whose bounded wait ran out

unsigned int* device_error() {
    static std::atomic<unsigned int*> cached[64];
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return nullptr;
    if (!cached[dev].load()) {
        void* p = nullptr;
        if (cudaGetSymbolAddress(&p, g_device_error) != cudaSuccess) return nullptr;
        cached[dev] = (unsigned int*)p;
    }
    return cached[dev].load();
}

template <int VPL, int PRO, bool HEAD>
int launch_stream_vpl(const DenseGemvArgs& a, int grid, size_t smem, cudaStream_t s) {
    const int st = ensure_dyn_smem((const void*)dense_gemv_stream_kernel<VPL, PRO, HEAD>, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(dense_gemv_stream_kernel<VPL, PRO, HEAD>, dim3(grid), dim3(kGvThreads), smem, s, a));
    g_launches++;
    return kStatusOk;
}

template <int PRO, bool HEAD>
int launch_stream(const DenseGemvArgs& a, int grid, size_t smem, cudaStream_t s) {
    if (a.segv <= 3 * 32) return launch_stream_vpl<3, PRO, HEAD>(a, grid, smem, s);
    if (a.segv <= 6 * 32) return launch_stream_vpl<6, PRO, HEAD>(a, grid, smem, s);
    return launch_stream_vpl<kGsMaxVpl, PRO, HEAD>(a, grid, smem, s);
}

// Deals the CTAs of a grid to the two sets of rows; returns the most rows a CTA gets (pairs stay together).
int deal_rows(DenseGemvArgs& a, int grid) {
    a.cta2 = grid;
    if (!a.rows2) return a.n_out / grid + 2;
    a.cta2 = std::max(1, std::min(grid - 1, (int)((long long)grid * a.n_out / (a.n_out + a.rows2))));
    return std::max(a.n_out / a.cta2, a.rows2 / (grid - a.cta2)) + 2;
}

// Column segments, ring and grid of the stream kernel; false when a row is too long for it.
bool plan_stream(DenseGemvArgs& a, int* grid, size_t* smem) {
    const int vecs = a.ldw / 8;
    if (a.w_r) {  // segments of one length for the matrix and for each routed one
        const int vecs_r = a.ld_r / 8, total = vecs + a.top * vecs_r;
        bool found = false;
        for (int n = std::min(kGvWarps, (total + 6 * 32 - 1) / (6 * 32)); n <= kGvWarps && !found; ++n) {
            a.segv = (total + n - 1) / n - 1;
            while (!found && ++a.segv <= kGsMaxVpl * 32) {
                a.seg_r = (vecs_r + a.segv - 1) / a.segv;
                a.nseg = (vecs + a.segv - 1) / a.segv + a.top * a.seg_r;
                found = a.nseg <= n;
            }
        }
        if (!found) return false;
    } else {
        a.nseg = 1;
        while (a.nseg < kGvWarps && (vecs + a.nseg - 1) / a.nseg > 6 * 32) a.nseg *= 2;
        a.segv = (vecs + a.nseg - 1) / a.nseg;
        if (a.segv > kGsMaxVpl * 32 || (a.nseg - 1) * a.segv >= vecs) return false;
    }
    a.slots = std::max(2, std::min(kGsMaxSlots, kGsRingBytes / (a.segv * 16)));
    const int groups = kGvWarps / a.nseg;
    *grid = std::max(a.rows2 ? 2 : 1, std::min((a.n_out + a.rows2 + groups - 1) / groups, sm_count()));
    *smem = (size_t)kGvWarps * a.slots * a.segv * 16 + (size_t)deal_rows(a, *grid) * a.nseg * sizeof(float);
    return *smem <= kMaxSmem - 2048;
}

template <typename T, int PRO, bool HEAD>
int launch_gemv(DenseGemvArgs a, int grid, cudaStream_t s) {
    const int rows = deal_rows(a, grid);
    const size_t smem = ((size_t)a.ldw + (a.w_r ? (size_t)a.top * a.ld_r : 0) + (size_t)rows * a.kslices) * sizeof(float);
    if (smem > kMaxSmem) return fail(kStatusUnsupported, "dn_gemv: %d columns need %zu bytes of shared memory", a.k, smem);
    if (smem > 40 * 1024) {
        const int st = ensure_dyn_smem((const void*)dense_gemv_kernel<T, PRO, HEAD>, smem);
        if (st) return st;
    }
    CUDA_TRY(launch_dep(dense_gemv_kernel<T, PRO, HEAD>, dim3(grid), dim3(kGvThreads), smem, s, a));
    g_launches++;
    return kStatusOk;
}

template <typename T>
int gemv_t(const llvq_dn_gemv_desc* d, HeadBest* best, int* grid_out, cudaStream_t s) {
    DenseGemvArgs a{};
    a.w = d->w, a.bias = d->bias, a.y = d->y, a.x = d->x, a.delta = d->delta, a.norm_w = d->norm_w, a.a_out = d->a_out;
    a.table = d->table, a.token = (const long long*)d->token, a.best = best;
    a.n_out = d->n_out, a.k = d->k, a.ldw = d->ldw, a.ld_table = d->ld_table, a.table_rows = d->table_rows;
    a.glu = d->glu;
    a.glu_scale = d->glu_scale == 0.0f ? 1.0f : d->glu_scale;
    a.residual = d->residual, a.t_out = d->t_out;
    a.w2 = d->w2, a.norm_w2 = d->norm_w2, a.y2 = d->y2, a.rows2 = d->rows2, a.glu2 = d->glu2;
    a.w_r = d->w_r, a.k_r = d->k_r, a.ld_r = d->ld_r;
    if (d->route) a.route = d->route, a.route_rows = d->route_rows, a.top = d->top, a.matrices = d->matrices, a.rows_m = d->rows2 / d->top;
    a.alpha = d->alpha, a.eps = d->eps, a.scale = d->scale, a.limit = d->limit, a.gain = d->gain, a.shift = d->shift, a.cap = d->softcap;
    // column slices: enough lanes for a row's vectors; rows of a CTA are shared by the row groups that are left
    if constexpr (sizeof(T) == 2) {
        size_t smem = 0;
        int grid = 0;
        a.err = device_error();
        a.vec_x = !(((uintptr_t)a.x | (uintptr_t)a.delta | (uintptr_t)a.norm_w | (uintptr_t)a.norm_w2) & 15);
        if (a.err && plan_stream(a, &grid, &smem)) {
            if (grid_out) *grid_out = grid;
            if (best) {
                if (d->prologue == LLVQ_DN_NORM) return launch_stream<kGvNorm, true>(a, grid, smem, s);
                if (d->prologue == LLVQ_DN_PLAIN) return launch_stream<kGvPlain, true>(a, grid, smem, s);
                return fail(kStatusUnsupported, "dn_head: prologue %d (plain or norm)", d->prologue);
            }
            switch (d->prologue) {
                case LLVQ_DN_PLAIN: return launch_stream<kGvPlain, false>(a, grid, smem, s);
                case LLVQ_DN_EMBED: return launch_stream<kGvEmbed, false>(a, grid, smem, s);
                default: return launch_stream<kGvNorm, false>(a, grid, smem, s);
            }
        }
    }
    const int vecs = (d->ldw + (d->w_r ? d->top * d->ld_r : 0)) / Vec16<T>::N;
    a.kslices = vecs > 128 ? 8 : vecs > 64 ? 4 : vecs > 32 ? 2 : 1;
    const int rows_step = kGvWarps / a.kslices * kGvRows;
    int grid = std::max(d->rows2 ? 2 : 1, std::min((d->n_out + d->rows2 + rows_step - 1) / rows_step, 4 * sm_count()));
    if (best) grid = std::min(grid, kHeadMaxGrid);
    if (grid_out) *grid_out = grid;
    if (best) {
        if (d->prologue == LLVQ_DN_NORM) return launch_gemv<T, kGvNorm, true>(a, grid, s);
        if (d->prologue == LLVQ_DN_PLAIN) return launch_gemv<T, kGvPlain, true>(a, grid, s);
        return fail(kStatusUnsupported, "dn_head: prologue %d (plain or norm)", d->prologue);
    }
    switch (d->prologue) {
        case LLVQ_DN_PLAIN: return launch_gemv<T, kGvPlain, false>(a, grid, s);
        case LLVQ_DN_EMBED: return launch_gemv<T, kGvEmbed, false>(a, grid, s);
        default: return launch_gemv<T, kGvNorm, false>(a, grid, s);
    }
}

int check_latent(const llvq_dn_latent* a, const char* who) {
    if (!a || bad_dtype(a->dtype)) return fail(kStatusInvalid, "%s: null descriptor or element type", who);
    const int vn = 16 / elem_size(a->dtype);
    if (a->heads <= 0 || a->dim <= 0 || a->rot_dim < 0 || a->vdim <= 0 || a->kv_rank <= 0 || a->window <= 0)
        return fail(kStatusInvalid, "%s: a size is not positive", who);
    if (a->rot_dims < 0 || a->rot_dims > a->rot_dim || a->rot_dims % 2 || (a->rot_dims && (!a->cos_t || !a->sin_t)))
        return fail(kStatusInvalid, "%s: %d rotated of %d dimensions", who, a->rot_dims, a->rot_dim);
    if (a->ld % vn || a->ld < a->kv_rank + a->rot_dim || a->slots <= 0 || !a->ring || ((uintptr_t)a->ring & 15))
        return fail(kStatusInvalid, "%s: cache rows of %d elements, %d slots", who, a->ld, a->slots);
    if (a->ldk % vn || a->ldk < a->kv_rank) return fail(kStatusInvalid, "%s: row stride %d of the up projections", who, a->ldk);
    return kStatusOk;
}

LatentRing ring_of(const llvq_dn_latent* a) { return LatentRing{a->ring, a->slots, a->ld}; }
RotaryTable rot_of(const llvq_dn_latent* a) { return RotaryTable{a->cos_t, a->sin_t, a->rot_dims}; }

// Whether the token's attention runs on the tensor cores (bf16 rows of a size that fits one tile in shared memory).
bool decode_on_mma(const llvq_dn_latent* a) {
    return a->dtype == LLVQ_DN_BF16 && a->kv_rank <= 1024 && latent_decode_mma_smem(a->ld) <= kMaxSmem;
}

template <typename T, typename Q>
int latent_query_t(const llvq_dn_latent* a, const float* q, const float* y_kv, const int64_t* pos, cudaStream_t s) {
    LatentQueryArgs k{q, a->uk, a->qlat, y_kv, a->kv_norm, (const long long*)pos, ring_of(a), rot_of(a),
                      a->heads, a->dim, a->rot_dim, a->kv_rank, a->ldk, a->eps};
    const int slices = (a->ldk / Vec16<T>::N + 31) / 32;
    CUDA_TRY(launch_dep(latent_query_kernel<T, Q>, dim3(a->heads + (y_kv ? 1 : 0), slices), dim3(256), 0, s, k));
    g_launches++;
    return kStatusOk;
}

LatentDecodeArgs decode_args(const llvq_dn_latent* a, const int64_t* pos) {
    return LatentDecodeArgs{a->qlat, (const long long*)pos, a->part, a->part + (size_t)a->heads * a->splits * 2, ring_of(a), a->heads, a->kv_rank,
                            a->window, a->scale};
}

template <int CH>
int latent_decode_mma(const llvq_dn_latent* a, const int64_t* pos, cudaStream_t s) {
    const size_t smem = latent_decode_mma_smem(a->ld);
    const int st = ensure_dyn_smem((const void*)latent_decode_mma_kernel<CH>, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(latent_decode_mma_kernel<CH>, dim3((a->heads + kLmHeads - 1) / kLmHeads, a->splits), dim3(256), smem, s, decode_args(a, pos)));
    g_launches++;
    return kStatusOk;
}

template <typename T>
int latent_decode_t(const llvq_dn_latent* a, const int64_t* pos, cudaStream_t s) {
    const size_t smem = latent_decode_smem<T>(a->ld, a->kv_rank);
    if (smem > kMaxSmem) return fail(kStatusUnsupported, "dn_latent_decode: cache rows of %d elements need %zu bytes of shared memory", a->ld, smem);
    const int st = ensure_dyn_smem((const void*)latent_decode_kernel<T>, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(latent_decode_kernel<T>, dim3((a->heads + kLdHeads - 1) / kLdHeads, a->splits), dim3(256), smem, s, decode_args(a, pos)));
    g_launches++;
    return kStatusOk;
}

template <typename T>
int latent_value_t(const llvq_dn_latent* a, float* ctx, cudaStream_t s) {
    LatentValueArgs k{a->part, a->part + (size_t)a->heads * a->splits * 2, a->sink, a->uv, ctx, a->heads, a->vdim, a->kv_rank, a->ldk, a->splits};
    const size_t smem = ((size_t)a->ldk + a->splits) * sizeof(float);
    if (smem > kMaxSmem) return fail(kStatusUnsupported, "dn_latent_value: %d latent dimensions, %d splits", a->kv_rank, a->splits);
    const int st = ensure_dyn_smem((const void*)latent_value_kernel<T>, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(latent_value_kernel<T>, dim3(a->heads, (a->vdim + kLvRows - 1) / kLvRows), dim3(256), smem, s, k));
    g_launches++;
    return kStatusOk;
}

template <int NV, bool VEC>
int prefill_mma(const LatentPrefillArgs& p, size_t smem, cudaStream_t s) {
    const int st = ensure_dyn_smem((const void*)latent_prefill_mma_kernel<NV, VEC>, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(latent_prefill_mma_kernel<NV, VEC>, dim3((p.n_q + kLpM - 1) / kLpM, p.heads, (p.vdim + NV * 8 - 1) / (NV * 8)),
                        dim3(kLpThreads), smem, s, p));
    g_launches++;
    return kStatusOk;
}

template <typename T>
int prefill_simt(const LatentPrefillArgs& p, cudaStream_t s) {
    const size_t smem = (size_t)kLsWarps * (p.dim + p.rot_dim + p.vdim) * sizeof(float);
    if (smem > kMaxSmem) return fail(kStatusUnsupported, "dn_latent_prefill: head sizes %d + %d, %d", p.dim, p.rot_dim, p.vdim);
    const int st = ensure_dyn_smem((const void*)latent_prefill_simt_kernel<T>, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(latent_prefill_simt_kernel<T>, dim3((p.n_q + kLsWarps - 1) / kLsWarps, p.heads), dim3(kLsWarps * 32), smem, s, p));
    g_launches++;
    return kStatusOk;
}

// The tcgen05 kernel takes heads of whole 16-byte vectors whose tiles fit shared memory and TMEM, and portions that
// fill a good part of its query tiles.
bool prefill_fits_tc(int dtype, int n_q, int dim, int rot_dim, int vdim, float scale) {
    return dtype == LLVQ_DN_BF16 && n_q >= 64 && scale > 0.0f && !((dim | rot_dim | vdim) & 7) && tc_v_rows(vdim) <= 192 &&
           latent_prefill_tc_smem(dim + rot_dim, vdim) <= kMaxSmem - 1024;
}
bool prefill_on_tc(const llvq_dn_latent* a, int n_q) {
    return !(a->kv_rank & 7) && prefill_fits_tc(a->dtype, n_q, a->dim, a->rot_dim, a->vdim, a->scale);
}

int prefill_tc(const LatentPrefillArgs& p, const void* vt, int ld_vt, cudaStream_t s) {
    LatentPrefillTcArgs tc{p, vt, ld_vt, device_error()};
    if (!tc.err) return fail(kStatusCuda, "prompt attention: no error word");
    const size_t smem = latent_prefill_tc_smem(p.dim + p.rot_dim, p.vdim);
    const int st = ensure_dyn_smem((const void*)latent_prefill_tc_kernel, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(latent_prefill_tc_kernel, dim3((p.n_q + 2 * kTcM - 1) / (2 * kTcM), p.heads), dim3(kTcThreads), smem, s, tc));
    g_launches++;
    return kStatusOk;
}

// Values along the positions. kernel: 0 = by size and type, 1 = the generic one.
int prefill_plain(int dtype, const LatentPrefillArgs& p, int kernel, cudaStream_t s) {
    if (dtype == LLVQ_DN_F32) return prefill_simt<float>(p, s);
    const int nv = p.vdim <= 64 ? 8 : p.vdim <= 128 ? 16 : 32;
    const size_t smem = latent_prefill_smem(p.dim, p.rot_dim, nv);
    if (kernel == 1 || smem > kMaxSmem) return prefill_simt<bf16>(p, s);
    const bool vec = !((p.dim | p.rot_dim | p.vdim | p.ld_kv | p.ld_kr | p.k_head | p.v_head | p.v_off) & 7) &&
                     !(((uintptr_t)p.q | (uintptr_t)p.kv | (uintptr_t)p.kr | (uintptr_t)p.out) & 15);
    if (nv == 8) return vec ? prefill_mma<8, true>(p, smem, s) : prefill_mma<8, false>(p, smem, s);
    if (nv == 16) return vec ? prefill_mma<16, true>(p, smem, s) : prefill_mma<16, false>(p, smem, s);
    return vec ? prefill_mma<32, true>(p, smem, s) : prefill_mma<32, false>(p, smem, s);
}

}  // namespace

extern "C" {

const char* llvq_dn_last_error(void) { return g_error.c_str(); }
uint64_t llvq_dn_launch_count(void) { return g_launches.load(); }
int llvq_dn_poll_error(int32_t* out) {
    if (!out) return fail(kStatusInvalid, "dn_poll_error: null argument");
    unsigned int v = 0, zero = 0;
    CUDA_TRY(cudaMemcpyFromSymbol(&v, g_device_error, sizeof v));
    if (v) CUDA_TRY(cudaMemcpyToSymbol(g_device_error, &zero, sizeof zero));
    *out = (int32_t)v;
    return kStatusOk;
}
int llvq_dn_set_overlap(int32_t on) {
    g_overlap_ops = on ? 1 : 0;
    return kStatusOk;
}

int llvq_dn_gemv(const llvq_dn_gemv_desc* d, llvq_dn_stream stream) {
    const int st = check_gemv(d, "dn_gemv");
    if (st) return st;
    if (!d->y) return fail(kStatusInvalid, "dn_gemv: null result");
    return d->dtype == LLVQ_DN_BF16 ? gemv_t<bf16>(d, nullptr, nullptr, (cudaStream_t)stream) : gemv_t<float>(d, nullptr, nullptr, (cudaStream_t)stream);
}

int llvq_dn_head(const llvq_dn_gemv_desc* d, void* scratch, float* val_out, int64_t* idx_out, llvq_dn_stream stream) {
    int st = check_gemv(d, "dn_head");
    if (st) return st;
    if (d->glu || d->rows2 || d->residual) return fail(kStatusUnsupported, "dn_head: rows in pairs, second rows or a residual");
    if (!scratch || !val_out || !idx_out) return fail(kStatusInvalid, "dn_head: null argument");
    cudaStream_t s = (cudaStream_t)stream;
    int grid = 0;
    st = d->dtype == LLVQ_DN_BF16 ? gemv_t<bf16>(d, (HeadBest*)scratch, &grid, s) : gemv_t<float>(d, (HeadBest*)scratch, &grid, s);
    if (st) return st;
    CUDA_TRY(launch_dep(lm_head_pick_kernel, dim3(1), dim3(kHeadMaxGrid), 0, s, (const HeadBest*)scratch, grid, 0ll, val_out, (long long*)idx_out));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_latent_query(const llvq_dn_latent* a, const float* q, const float* y_kv, const int64_t* pos, llvq_dn_stream stream) {
    const int st = check_latent(a, "dn_latent_query");
    if (st) return st;
    if (!q || !pos || !a->uk || !a->qlat || (y_kv && !a->kv_norm)) return fail(kStatusInvalid, "dn_latent_query: null argument");
    cudaStream_t s = (cudaStream_t)stream;
    if (a->dtype == LLVQ_DN_F32) return latent_query_t<float, float>(a, q, y_kv, pos, s);
    return decode_on_mma(a) ? latent_query_t<bf16, bf16>(a, q, y_kv, pos, s) : latent_query_t<bf16, float>(a, q, y_kv, pos, s);
}

int llvq_dn_latent_decode(const llvq_dn_latent* a, const int64_t* pos, llvq_dn_stream stream) {
    const int st = check_latent(a, "dn_latent_decode");
    if (st) return st;
    if (!pos || !a->qlat || !a->part || a->splits < 1 || a->splits > 4096) return fail(kStatusInvalid, "dn_latent_decode: null argument or %d splits", a->splits);
    if (a->window > a->slots) return fail(kStatusInvalid, "dn_latent_decode: a window of %d over %d slots", a->window, a->slots);
    cudaStream_t s = (cudaStream_t)stream;
    if (a->dtype == LLVQ_DN_F32) return latent_decode_t<float>(a, pos, s);
    if (!decode_on_mma(a)) return latent_decode_t<bf16>(a, pos, s);
    if (a->kv_rank <= 128) return latent_decode_mma<1>(a, pos, s);
    if (a->kv_rank <= 256) return latent_decode_mma<2>(a, pos, s);
    return a->kv_rank <= 512 ? latent_decode_mma<4>(a, pos, s) : latent_decode_mma<8>(a, pos, s);
}

int llvq_dn_latent_value(const llvq_dn_latent* a, float* ctx, llvq_dn_stream stream) {
    const int st = check_latent(a, "dn_latent_value");
    if (st) return st;
    if (!ctx || !a->part || !a->uv || a->splits < 1 || a->splits > 4096) return fail(kStatusInvalid, "dn_latent_value: null argument or %d splits", a->splits);
    return a->dtype == LLVQ_DN_BF16 ? latent_value_t<bf16>(a, ctx, (cudaStream_t)stream) : latent_value_t<float>(a, ctx, (cudaStream_t)stream);
}

int llvq_dn_latent_prefill_transposes(const llvq_dn_latent* a, int32_t n_q) {
    return check_latent(a, "dn_latent_prefill_transposes") == kStatusOk && prefill_on_tc(a, n_q) ? 1 : 0;
}

int llvq_dn_latent_prefill(const llvq_dn_latent* a, const void* q, const void* kv, int32_t ld_kv, const void* kr, int32_t ld_kr,
                           const void* vt, int32_t ld_vt, int32_t n_q, int32_t n_k, int64_t pos0, int64_t key0, void* out, int32_t kernel, llvq_dn_stream stream) {
    const int st = check_latent(a, "dn_latent_prefill");
    if (st) return st;
    if (!q || !kv || !kr || !out) return fail(kStatusInvalid, "dn_latent_prefill: null argument");
    if (n_q <= 0 || n_k <= 0 || pos0 < 0 || key0 < 0 || key0 > pos0 || pos0 + n_q > key0 + n_k || ld_kv < a->heads * (a->dim + (vt ? 0 : a->vdim)) ||
        ld_kr < a->rot_dim || (vt && ld_vt < n_k))
        return fail(kStatusInvalid, "dn_latent_prefill: %d queries at %lld over %d keys at %lld", n_q, (long long)pos0, n_k, (long long)key0);
    LatentPrefillArgs p{q, kv, kr, a->sink, out, rot_of(a), pos0, key0, n_q, n_k, a->heads, a->dim, a->rot_dim, a->vdim, ld_kv, ld_kr,
                        a->window, a->scale, 1, a->dim, a->vdim, a->heads * a->dim};
    cudaStream_t s = (cudaStream_t)stream;
    if (vt) {
        if (!prefill_on_tc(a, n_q) || ((ld_kv | ld_kr | ld_vt) & 7) || (((uintptr_t)q | (uintptr_t)kv | (uintptr_t)kr | (uintptr_t)vt | (uintptr_t)out) & 15))
            return fail(kStatusInvalid, "dn_latent_prefill: transposed values where llvq_dn_latent_prefill_transposes says no, or rows not on 16 bytes");
        return prefill_tc(p, vt, ld_vt, s);
    }
    return prefill_plain(a->dtype, p, kernel, s);
}

int llvq_dn_embed_rows(int32_t dtype, const void* table, int32_t ld, int32_t table_rows, const int64_t* tokens, int32_t rows, int32_t n,
                       float scale, float* x, void* xt, llvq_dn_stream stream) {
    if (bad_dtype(dtype) || !table || !tokens || !x || rows <= 0 || n <= 0 || ld < n || table_rows <= 0) return fail(kStatusInvalid, "dn_embed_rows: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(embed_rows_kernel<bf16>, dim3(rows), dim3(kRowThreads), 0, s, (const bf16*)table, ld, table_rows, (const long long*)tokens, scale, x, (bf16*)xt, n));
    else
        CUDA_TRY(launch_dep(embed_rows_kernel<float>, dim3(rows), dim3(kRowThreads), 0, s, (const float*)table, ld, table_rows, (const long long*)tokens, scale, x, (float*)xt, n));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_postnorm_rows(int32_t dtype, const float* x, const void* y, const float* bias, const float* w, float alpha, float eps,
                          void* xt, float* out, int32_t rows, int32_t n, llvq_dn_stream stream) {
    if (bad_dtype(dtype) || !x || !w || rows <= 0 || n <= 0 || (size_t)n * 4 > kMaxSmem - 1024) return fail(kStatusInvalid, "dn_postnorm_rows: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    const int vec = n % 4 == 0 && !(((uintptr_t)x | (uintptr_t)y | (uintptr_t)bias | (uintptr_t)w | (uintptr_t)xt | (uintptr_t)out) & 15);
    const size_t smem = (size_t)n * 4;
    const void* f = dtype == LLVQ_DN_BF16 ? (const void*)postnorm_rows_kernel<bf16> : (const void*)postnorm_rows_kernel<float>;
    if (smem > 40 * 1024) {
        const int st = ensure_dyn_smem(f, smem);
        if (st) return st;
    }
    if (dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(postnorm_rows_kernel<bf16>, dim3(rows), dim3(kRowThreads), smem, s, x, (const bf16*)y, bias, w, alpha, eps, (bf16*)xt, out, n, vec));
    else
        CUDA_TRY(launch_dep(postnorm_rows_kernel<float>, dim3(rows), dim3(kRowThreads), smem, s, x, (const float*)y, bias, w, alpha, eps, (float*)xt, out, n, vec));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_latent_rows(const llvq_dn_latent* a, const void* y, int32_t ldy, int32_t q_rank, const float* q_norm, void* cq,
                        int64_t pos0, int32_t rows, int32_t store_kv, llvq_dn_stream stream) {
    const int st = check_latent(a, "dn_latent_rows");
    if (st) return st;
    if (!y || !q_norm || !cq || q_rank <= 0 || rows <= 0 || rows > a->slots || pos0 < 0 || (store_kv && !a->kv_norm) ||
        ldy < q_rank + (store_kv ? a->kv_rank + a->rot_dim : 0))
        return fail(kStatusInvalid, "dn_latent_rows: %d rows into %d slots, row stride %d", rows, a->slots, ldy);
    LatentRing ring = ring_of(a);
    if (!store_kv) ring.rows = nullptr;
    cudaStream_t s = (cudaStream_t)stream;
    if (a->dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(latent_rows_kernel<bf16>, dim3(rows), dim3(kRowThreads), 0, s, (const bf16*)y, ldy, q_rank, q_norm, (bf16*)cq, a->kv_norm, a->kv_rank,
                            a->rot_dim, rot_of(a), (long long)pos0, ring, a->eps));
    else
        CUDA_TRY(launch_dep(latent_rows_kernel<float>, dim3(rows), dim3(kRowThreads), 0, s, (const float*)y, ldy, q_rank, q_norm, (float*)cq, a->kv_norm, a->kv_rank,
                            a->rot_dim, rot_of(a), (long long)pos0, ring, a->eps));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_gated_rows(int32_t dtype, const void* gate_up, const float* bias, void* out, int32_t ld_out, int32_t rows, int32_t n, float limit, float gain,
                       float shift, float scale, llvq_dn_stream stream) {
    if (bad_dtype(dtype) || !gate_up || !out || rows <= 0 || n <= 0 || ld_out < n) return fail(kStatusInvalid, "dn_gated_rows: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    const int vec = n % 4 == 0 && ld_out % 4 == 0 && !(((uintptr_t)gate_up | (uintptr_t)bias | (uintptr_t)out) & 15);
    const dim3 grid(rows, (n + 8 * kRowThreads - 1) / (8 * kRowThreads));
    if (dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(glu_rows_kernel<bf16>, grid, dim3(kRowThreads), 0, s, (const bf16*)gate_up, bias, (bf16*)out, ld_out, n, limit, gain, shift, scale, vec));
    else
        CUDA_TRY(launch_dep(glu_rows_kernel<float>, grid, dim3(kRowThreads), 0, s, (const float*)gate_up, bias, (float*)out, ld_out, n, limit, gain, shift, scale, vec));
    g_launches++;
    return kStatusOk;
}
int llvq_dn_glu_rows(int32_t dtype, const void* gate_up, const float* bias, void* out, int32_t rows, int32_t n, float limit, float gain,
                     float shift, llvq_dn_stream stream) {
    return llvq_dn_gated_rows(dtype, gate_up, bias, out, n, rows, n, limit, gain, shift, 1.0f, stream);
}

int llvq_dn_add_norms_rows(int32_t dtype, float* x, const void* y, const void* routed, const int32_t* places, int32_t top, const float* w1, void* h1,
                           const float* w2, void* h2, float eps, int32_t rows, int32_t n, llvq_dn_stream stream) {
    if (bad_dtype(dtype) || !x || rows <= 0 || n <= 0 || (size_t)n * 4 > kMaxSmem - 1024 || (routed && (!places || top <= 0)) || (w1 && !h1) || (w2 && !h2))
        return fail(kStatusInvalid, "dn_add_norms_rows: bad argument");
    const int vec = n % 4 == 0 && !(((uintptr_t)x | (uintptr_t)y | (uintptr_t)routed | (uintptr_t)w1 | (uintptr_t)w2 | (uintptr_t)h1 | (uintptr_t)h2) & 15);
    AddNormsArgs k{x, y, routed, places, w1, w2, h1, h2, n, routed ? top : 0, vec, eps};
    const size_t smem = (size_t)n * 4;
    if (smem > 40 * 1024) {
        const int st = ensure_dyn_smem(dtype == LLVQ_DN_BF16 ? (const void*)add_norms_rows_kernel<bf16> : (const void*)add_norms_rows_kernel<float>, smem);
        if (st) return st;
    }
    if (dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(add_norms_rows_kernel<bf16>, dim3(rows), dim3(kRowThreads), smem, (cudaStream_t)stream, k));
    else
        CUDA_TRY(launch_dep(add_norms_rows_kernel<float>, dim3(rows), dim3(kRowThreads), smem, (cudaStream_t)stream, k));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_softcap(float* y, size_t n, float cap, llvq_dn_stream stream) {
    if (!y || !n || !(cap > 0.0f)) return fail(kStatusInvalid, "dn_softcap: bad argument");
    const int grid = (int)std::min<size_t>((n + kRowThreads - 1) / kRowThreads, 4096);
    CUDA_TRY(launch_dep(softcap_kernel, dim3(grid), dim3(kRowThreads), 0, (cudaStream_t)stream, y, n, cap));
    g_launches++;
    return kStatusOk;
}

}  // extern "C"

#include "mixer_api.cuh"
