// The mixers' part of the C ABI (include/llvq_dense.h): grouped-query attention, the gated linear recurrence, the gated
// delta rule. Included by dense_api.cu, whose helpers it uses.
#pragma once

#include <initializer_list>

namespace {

// Sizes are whole 16-byte vectors and pointers on 16-byte boundaries.
int whole_vectors(int dtype, std::initializer_list<int> sizes, std::initializer_list<const void*> pointers) {
    for (const int n : sizes)
        if (n % (16 / elem_size(dtype))) return 0;
    for (const void* p : pointers)
        if ((uintptr_t)p & 15) return 0;
    return 1;
}

GqaRing ring_of(const llvq_dn_gqa* a) { return GqaRing{a->ring, a->slots, a->ld, a->kd, a->vd}; }

int check_gqa(const llvq_dn_gqa* a, const char* who) {
    if (!a || bad_dtype(a->dtype)) return fail(kStatusInvalid, "%s: null descriptor or element type", who);
    const int vn = 16 / elem_size(a->dtype);
    if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 || a->window <= 0)
        return fail(kStatusInvalid, "%s: %d heads over %d, sizes %d and %d, window %d", who, a->heads, a->kv_heads, a->dim, a->vdim, a->window);
    if (!a->ring || ((uintptr_t)a->ring & 15) || a->slots <= 0 || a->kd < a->dim || a->kd % vn || a->vd < a->vdim || a->vd % vn || a->ld % vn ||
        a->ld < a->kv_heads * (a->kd + a->vd))
        return fail(kStatusInvalid, "%s: cache rows of %d elements (heads of %d and %d), %d slots", who, a->ld, a->kd, a->vd, a->slots);
    return kStatusOk;
}

int check_lru(const llvq_dn_lru* a, const char* who) {
    if (!a || bad_dtype(a->dtype)) return fail(kStatusInvalid, "%s: null descriptor or element type", who);
    if (a->blocks <= 0 || a->n <= 0 || a->taps <= 0 || !a->conv_w || !a->conv_b || !a->b || !a->lam || !a->conv || !a->state)
        return fail(kStatusInvalid, "%s: %d blocks of %d, %d taps, or a null argument", who, a->blocks, a->n, a->taps);
    return kStatusOk;
}

int check_delta(const llvq_dn_delta* a, const char* who) {
    if (!a || bad_dtype(a->dtype)) return fail(kStatusInvalid, "%s: null descriptor or element type", who);
    if (a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 || a->taps <= 0 || a->vp < a->vdim || a->vp % 4)
        return fail(kStatusInvalid, "%s: %d heads over %d, sizes %d and %d (%d), %d taps", who, a->heads, a->kv_heads, a->dim, a->vdim, a->vp, a->taps);
    if (!a->conv_w || !a->decay || !a->dt_bias || !a->norm || !a->conv || !a->state || ((uintptr_t)a->state & 15))
        return fail(kStatusInvalid, "%s: null argument", who);
    return kStatusOk;
}

template <typename T>
int mixer_token_t(const llvq_dn_gqa* a, const llvq_dn_lru* r, const int64_t* pos, cudaStream_t s) {
    GqaArgs g{};
    LruArgs l{};
    int attn = 0, rec = 0;
    size_t smem = 0;
    if (a) {
        if (a->vd / Vec16<T>::N > kGqThreads) return fail(kStatusUnsupported, "dn_mixer_token: values of %d", a->vdim);
        g = GqaArgs{a->q, a->k, a->v, a->gate, a->q_norm, a->k_norm, (const long long*)pos, a->part, a->part + (size_t)a->heads * a->splits * 2,
                    a->arrived, a->out, ring_of(a), a->heads, a->kv_heads, a->dim, a->vdim, a->window, a->splits, a->scale, a->eps, a->out_scale};
        attn = gqa_ctas(a->heads, a->kv_heads, a->splits);
        smem = gqa_token_smem<T>(a->kd, a->vd);
    }
    if (r) {
        l = LruArgs{r->x, r->y, r->conv_w, r->conv_b, r->w, r->b, r->lam, (const long long*)pos, r->conv, r->state, r->out, r->blocks, r->n, r->taps,
                    r->ldw, r->out_scale};
        rec = r->blocks * lru_tiles(r->n);
        smem = std::max(smem, (size_t)r->ldw * sizeof(float));
    }
    if (smem > kMaxSmem - 1024) return fail(kStatusUnsupported, "dn_mixer_token: %zu bytes of shared memory", smem);
    const int st = ensure_dyn_smem((const void*)mixer_token_kernel<T>, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(mixer_token_kernel<T>, dim3(attn + rec), dim3(256), smem, s, g, attn, l));
    g_launches++;
    return kStatusOk;
}

template <int LANES, int FOURS, int NC>
int delta_scan_t(const DeltaScanArgs& k, cudaStream_t s) {
    const dim3 grid((k.vdim + kDtCols - 1) / kDtCols, k.heads);
    // A CTA is bound by its own chain of tokens: two on one SM slow each other down. Where every CTA can have an SM, it
    // asks for more than half of the shared memory (CTAs launched into the tail of the kernel before would pile up).
    const size_t smem = std::max(delta_scan_smem(k.dim), (int)(grid.x * grid.y) <= sm_count() ? kMaxSmem / 2 + 1024 : 0);
    const int st = ensure_dyn_smem((const void*)delta_scan_kernel<LANES, FOURS, NC>, smem);
    if (st) return st;
    CUDA_TRY(launch_dep(delta_scan_kernel<LANES, FOURS, NC>, grid, dim3(kDtCols / NC * LANES), smem, s, k));
    g_launches++;
    return kStatusOk;
}

int delta_scan(const DeltaScanArgs& k, cudaStream_t s) {
    const int fours = delta_fours(k.dim);
    if (delta_lanes(k.dim) == 16) switch (fours) {
        case 1: return delta_scan_t<16, 1, 4>(k, s);
        case 2: return delta_scan_t<16, 2, 4>(k, s);
        case 3: return delta_scan_t<16, 3, 4>(k, s);
        default: return delta_scan_t<16, 4, 4>(k, s);
    }
    switch (fours) {
        case 3: return delta_scan_t<32, 3, 4>(k, s);
        case 4: return delta_scan_t<32, 4, 4>(k, s);
        case 5: return delta_scan_t<32, 5, 4>(k, s);
        case 6: return delta_scan_t<32, 6, 4>(k, s);
        case 7: return delta_scan_t<32, 7, 4>(k, s);
        case 8: return delta_scan_t<32, 8, 4>(k, s);
        default: return fail(kStatusUnsupported, "dn_delta_rows: keys of %d (at most 1024)", k.dim);
    }
}

}  // namespace

extern "C" {

int llvq_dn_mixer_token(const llvq_dn_gqa* a, const llvq_dn_lru* r, const int64_t* pos, llvq_dn_stream stream) {
    if ((!a && !r) || !pos) return fail(kStatusInvalid, "dn_mixer_token: null argument");
    if (a) {
        const int st = check_gqa(a, "dn_mixer_token");
        if (st) return st;
        if (!a->q || !a->k || !a->v || !a->q_norm || !a->k_norm || !a->part || !a->arrived || !a->out) return fail(kStatusInvalid, "dn_mixer_token: null argument");
        if (a->window > a->slots || a->splits < 1 || a->splits > kGqMaxSplits)
            return fail(kStatusInvalid, "dn_mixer_token: a window of %d over %d slots, %d splits", a->window, a->slots, a->splits);
    }
    if (r) {
        const int st = check_lru(r, "dn_mixer_token");
        if (st) return st;
        const int vn = 16 / elem_size(r->dtype);
        if (!r->x || !r->y || !r->w || ((uintptr_t)r->w & 15) || !r->out || r->ldw < r->n || r->ldw % vn || (a && a->dtype != r->dtype))
            return fail(kStatusInvalid, "dn_mixer_token: null argument, row stride %d, or unlike element types", r->ldw);
    }
    return (a ? a->dtype : r->dtype) == LLVQ_DN_BF16 ? mixer_token_t<bf16>(a, r, pos, (cudaStream_t)stream) : mixer_token_t<float>(a, r, pos, (cudaStream_t)stream);
}

int llvq_dn_gqa_rows(const llvq_dn_gqa* a, const void* q, const void* k, const void* v, int32_t ldy, void* qn, int64_t pos0, int32_t rows, llvq_dn_stream stream) {
    const int st = check_gqa(a, "dn_gqa_rows");
    if (st) return st;
    if (!q || !k || !v || !qn || !a->q_norm || !a->k_norm || ldy <= 0 || pos0 < 0 || rows <= 0 || rows > a->slots)
        return fail(kStatusInvalid, "dn_gqa_rows: null argument, or %d rows into %d slots", rows, a->slots);
    GqaRowsArgs p{q, k, v, qn, a->q_norm, a->k_norm, ring_of(a), pos0, ldy, a->heads, a->kv_heads, a->dim, a->vdim, a->eps, 0};
    p.vec = whole_vectors(a->dtype, {a->dim, a->vdim, ldy}, {q, k, v, qn});
    if (a->dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(gqa_rows_kernel<bf16>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, p));
    else
        CUDA_TRY(launch_dep(gqa_rows_kernel<float>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, p));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_gqa_prefill_transposes(const llvq_dn_gqa* a, int32_t n_q) {
    return check_gqa(a, "dn_gqa_prefill_transposes") == kStatusOk && prefill_fits_tc(a->dtype, n_q, a->dim, 0, a->vdim, a->scale) ? 1 : 0;
}

int llvq_dn_gqa_prefill(const llvq_dn_gqa* a, const void* qn, const void* rows, const void* vt, int32_t ld_vt, int32_t n_q, int32_t n_k, int64_t pos0,
                        int64_t key0, void* out, int32_t kernel, llvq_dn_stream stream) {
    const int st = check_gqa(a, "dn_gqa_prefill");
    if (st) return st;
    if (!qn || !rows || !out || n_q <= 0 || n_k <= 0 || pos0 < 0 || key0 < 0 || key0 > pos0 || pos0 + n_q > key0 + n_k || (vt && ld_vt < n_k))
        return fail(kStatusInvalid, "dn_gqa_prefill: %d queries at %lld over %d keys at %lld", n_q, (long long)pos0, n_k, (long long)key0);
    LatentPrefillArgs p{qn, rows, rows, nullptr, out, RotaryTable{nullptr, nullptr, 0}, pos0, key0, n_q, n_k, a->heads, a->dim, 0, a->vdim, a->ld, a->ld,
                        a->window, a->scale, a->heads / a->kv_heads, a->kd, a->vd, a->kv_heads * a->kd};
    if (vt) {
        if (!prefill_fits_tc(a->dtype, n_q, a->dim, 0, a->vdim, a->scale) || (ld_vt & 7) ||
            (((uintptr_t)qn | (uintptr_t)rows | (uintptr_t)vt | (uintptr_t)out) & 15))
            return fail(kStatusInvalid, "dn_gqa_prefill: transposed values where llvq_dn_gqa_prefill_transposes says no, or rows not on 16 bytes");
        return prefill_tc(p, vt, ld_vt, (cudaStream_t)stream);
    }
    return prefill_plain(a->dtype, p, kernel, (cudaStream_t)stream);
}

int llvq_dn_gate_rows(int32_t dtype, const void* x, int32_t ldx, const void* gate, int32_t ldg, void* out, int32_t ldo, int32_t rows, int32_t n, float scale,
                      llvq_dn_stream stream) {
    if (bad_dtype(dtype) || !x || !gate || !out || rows <= 0 || n <= 0 || ldx < n || ldg < n || ldo < n) return fail(kStatusInvalid, "dn_gate_rows: bad argument");
    const int vec = whole_vectors(dtype, {n, ldx, ldg, ldo}, {x, gate, out});
    const dim3 grid(rows, vec ? (n + 2047) / 2048 : (n + 1023) / 1024);
    if (dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(gate_rows_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)stream, (const bf16*)x, ldx, (const bf16*)gate, ldg, (bf16*)out, ldo, n, scale, vec));
    else
        CUDA_TRY(launch_dep(gate_rows_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)x, ldx, (const float*)gate, ldg, (float*)out, ldo, n, scale, vec));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_conv_rows(int32_t dtype, const void* x, int32_t ldx, const float* x_bias, const float* w, const float* bias, const float* ring, void* out,
                      int32_t channels, int32_t taps, int64_t pos0, int32_t rows, llvq_dn_stream stream) {
    if (bad_dtype(dtype) || !x || !w || !ring || !out || channels <= 0 || taps <= 0 || ldx < channels || pos0 < 0 || rows <= 0)
        return fail(kStatusInvalid, "dn_conv_rows: bad argument");
    const dim3 grid((channels + 255) / 256, (rows + kConvRun - 1) / kConvRun);
    if (dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(conv_rows_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)stream, (const bf16*)x, ldx, x_bias, w, bias, ring, (bf16*)out, channels,
                            taps, (long long)pos0, rows));
    else
        CUDA_TRY(launch_dep(conv_rows_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)x, ldx, x_bias, w, bias, ring, (float*)out, channels,
                            taps, (long long)pos0, rows));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_conv_keep(int32_t dtype, const void* x, int32_t ldx, const float* x_bias, float* ring, int32_t channels, int32_t taps, int64_t pos0, int32_t rows,
                      llvq_dn_stream stream) {
    if (bad_dtype(dtype) || !x || !ring || channels <= 0 || taps <= 0 || ldx < channels || pos0 < 0 || rows <= 0) return fail(kStatusInvalid, "dn_conv_keep: bad argument");
    const dim3 grid((channels + 255) / 256);
    if (dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(conv_keep_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)stream, (const bf16*)x, ldx, x_bias, ring, channels, taps, (long long)pos0, rows));
    else
        CUDA_TRY(launch_dep(conv_keep_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)x, ldx, x_bias, ring, channels, taps, (long long)pos0, rows));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_lru_rows(const llvq_dn_lru* a, const void* u, const float* z, const void* y, int32_t ldy, const float* y_bias, void* out, int32_t ldo, int64_t pos0,
                     int32_t rows, llvq_dn_stream stream) {
    const int st = check_lru(a, "dn_lru_rows");
    if (st) return st;
    const int width = a->blocks * a->n;
    if (!u || !z || !y || !y_bias || !out || ldy < width || ldo < width || pos0 < 0 || rows <= 0) return fail(kStatusInvalid, "dn_lru_rows: bad argument");
    LruScanArgs k{u, z, a->b, a->lam, y, y_bias, a->state, out, pos0, rows, a->blocks, a->n, ldy, ldo, a->out_scale};
    if (a->dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(lru_scan_kernel<bf16>, dim3((width + kScanCh - 1) / kScanCh), dim3(kScanWarps * 32), 0, (cudaStream_t)stream, k));
    else
        CUDA_TRY(launch_dep(lru_scan_kernel<float>, dim3((width + kScanCh - 1) / kScanCh), dim3(kScanWarps * 32), 0, (cudaStream_t)stream, k));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_route_rows(const int32_t* table, int32_t table_rows, int32_t top, int32_t experts, const int64_t* tokens, int32_t rows, int32_t* source,
                       int32_t* places, int32_t* ends, llvq_dn_stream stream) {
    if (!table || !tokens || !source || !places || !ends || table_rows <= 0 || top <= 0 || experts <= 0 || rows <= 0 || (long long)rows * top > INT32_MAX)
        return fail(kStatusInvalid, "dn_route_rows: bad argument");
    const size_t smem = ((size_t)experts + 1) * sizeof(int);
    if (smem > 40 * 1024) return fail(kStatusUnsupported, "dn_route_rows: %d experts", experts);
    CUDA_TRY(launch_dep(route_rows_kernel, dim3(1), dim3(kRouteThreads), smem, (cudaStream_t)stream, table, table_rows, top, experts, (const long long*)tokens, rows,
                        source, places, ends));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_delta_token(const llvq_dn_delta* a, const int64_t* pos, llvq_dn_stream stream) {
    const int st = check_delta(a, "dn_delta_token");
    if (st) return st;
    if (!pos || !a->x || !a->gate || !a->beta || !a->alpha || !a->o || !a->arrived || !a->out) return fail(kStatusInvalid, "dn_delta_token: null argument");
    DeltaArgs k{a->x, a->gate, a->beta, a->alpha, a->conv_w, a->decay, a->dt_bias, a->norm, (const long long*)pos, a->conv, a->state, a->o, a->arrived, a->out,
                a->heads, a->kv_heads, a->dim, a->vdim, a->vp, a->taps, a->eps};
    const size_t smem = delta_token_smem(a->dim);
    if (smem > kMaxSmem - 8192) return fail(kStatusUnsupported, "dn_delta_token: keys of %d", a->dim);
    const int st2 = ensure_dyn_smem((const void*)delta_token_kernel, smem);
    if (st2) return st2;
    CUDA_TRY(launch_dep(delta_token_kernel, dim3((a->vp + kDtCols - 1) / kDtCols, a->heads), dim3(kDtThreads), smem, (cudaStream_t)stream, k));
    g_launches++;
    return kStatusOk;
}

int llvq_dn_delta_scratch(const llvq_dn_delta* a, int32_t rows, size_t* floats) {
    const int st = check_delta(a, "dn_delta_scratch");
    if (st) return st;
    if (rows <= 0 || !floats) return fail(kStatusInvalid, "dn_delta_scratch: bad argument");
    const size_t groups = delta_groups(rows);
    *floats = groups * (kDeltaGroup * (size_t)2 * a->kv_heads * delta_padded(a->dim) + (size_t)a->heads * kDeltaScalars) + (size_t)2 * rows * a->heads * a->vdim;
    return kStatusOk;
}

int llvq_dn_delta_rows(const llvq_dn_delta* a, const void* x, int32_t ldx, const float* ba, const void* gate, int32_t ldg, float* scratch, void* out, int32_t ldo,
                       int64_t pos0, int32_t rows, llvq_dn_stream stream) {
    const int st = check_delta(a, "dn_delta_rows");
    if (st) return st;
    const int channels = 2 * a->kv_heads * a->dim + a->heads * a->vdim, hv = a->heads * a->vdim;
    if (!x || !ba || !gate || !scratch || ((uintptr_t)scratch & 15) || !out || ldx < channels || ldg < hv || ldo < hv || pos0 < 0 || rows <= 0)
        return fail(kStatusInvalid, "dn_delta_rows: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    const int dp = delta_padded(a->dim);
    float* qk = scratch;
    float* sc = qk + (size_t)delta_groups(rows) * kDeltaGroup * 2 * a->kv_heads * dp;
    float* v = sc + (size_t)delta_groups(rows) * a->heads * kDeltaScalars;
    float* o = v + (size_t)rows * hv;
    DeltaPrepArgs p{x, ba, a->conv_w, a->conv, a->decay, a->dt_bias, qk, v, sc, pos0, rows, ldx, a->heads, a->kv_heads, a->dim, a->vdim, a->taps, dp};
    if (a->taps == 4 && ((uintptr_t)a->conv_w & 15)) return fail(kStatusInvalid, "dn_delta_rows: convolution weights not on 16 bytes");
    const int elem = elem_size(a->dtype);
    const bool fours = a->taps == 4 && !((a->dim | a->vdim | ldx) & 3) && !((uintptr_t)x & (4 * elem - 1));
    const auto prep = a->dtype == LLVQ_DN_BF16 ? (fours ? delta_prep_kernel<bf16, 4> : delta_prep_kernel<bf16, 1>)
                                                : (fours ? delta_prep_kernel<float, 4> : delta_prep_kernel<float, 1>);
    CUDA_TRY(launch_dep(prep, dim3(delta_groups(rows)), dim3(256), 0, s, p));
    g_launches++;
    int st2 = llvq_dn_conv_keep(a->dtype, x, ldx, nullptr, a->conv, channels, a->taps, pos0, rows, stream);
    if (st2) return st2;
    const int vec = a->vdim <= 256 && a->vdim % 8 == 0 && whole_vectors(a->dtype, {a->vdim, ldg, ldo}, {gate, out, o});
    st2 = delta_scan(DeltaScanArgs{qk, v, sc, a->state, o, pos0, rows, a->heads, a->kv_heads, a->dim, a->vdim, a->vp}, s);
    if (st2) return st2;
    if (a->dtype == LLVQ_DN_BF16)
        CUDA_TRY(launch_dep(head_gate_rows_kernel<bf16>, dim3(rows), dim3(256), 0, s, (const float*)o, a->norm, (const bf16*)gate, ldg, (bf16*)out, ldo, a->heads, a->vdim, a->eps, vec));
    else
        CUDA_TRY(launch_dep(head_gate_rows_kernel<float>, dim3(rows), dim3(256), 0, s, (const float*)o, a->norm, (const float*)gate, ldg, (float*)out, ldo, a->heads, a->vdim, a->eps, vec));
    g_launches++;
    return kStatusOk;
}

}  // extern "C"
