// Attention of a prompt portion over keys and values laid out per position, causal, windowed, with a sink in the
// denominator: latent attention (expanded by a matrix product ahead of it, k = W_uk c, v = W_uv c) and, with nothing to
// rotate, grouped-query attention (query head h reads key/value head h / rep; heads may be padded). Queries are laid out head by head as
// [dim unrotated | rot_dim to be rotated], kv rows as [keys, k_head apart | values from v_off on, v_head apart], the rotated key
// part is read from the cached rows (one for all heads). Key j of the operands is position key0 + j, query i is
// position pos0 + i.
//
//   latent_prefill_mma_kernel   bf16 operands on the tensor cores, f32 scores and softmax. A CTA of 8 warps owns
//       128 queries of one head (and a slice of the value dimensions), the query tile is staged once with its
//       rotation applied; key and value tiles of 64 positions are double buffered with cp.async. Tiles outside
//       the window of the CTA are never loaded, a warp skips those outside its own 16 rows, and only tiles that
//       cross an edge of the window are masked.
//   latent_prefill_simt_kernel  any element type and any size, f32 arithmetic throughout: one warp per query
//       and head, lane = position for the scores, lane = value dimension for the sums.
#pragma once
#include "latent_attn.cuh"

namespace llvq {

struct LatentPrefillArgs {
    const void* q;     // [n_q, heads * (dim + rot_dim)] of T
    const void* kv;    // [n_k, ld_kv] of T
    const void* kr;    // [n_k, ld_kr] of T: the rotated key part of each position
    const float* sink; // [heads] or null
    void* out;         // [n_q, heads * vdim] of T
    RotaryTable rt;
    long long pos0, key0;
    int n_q, n_k, heads, dim, rot_dim, vdim, ld_kv, ld_kr;
    int window;
    float scale;
    int rep, k_head, v_head, v_off;
};

constexpr int kLpM = 128, kLpN = 64, kLpThreads = 256;

// Pitches in elements: an odd number of 16-byte vectors, so that eight rows of an ldmatrix fall into different banks.
__host__ __device__ inline int lp_qk_pitch(int dim, int rot_dim) { return (dim + rot_dim + 15) / 16 * 16 + 8; }
inline size_t latent_prefill_smem(int dim, int rot_dim, int nv) {
    const size_t qk = lp_qk_pitch(dim, rot_dim), v = (size_t)nv * 8 + 8;
    return (kLpM * qk + 2 * kLpN * (qk + v)) * sizeof(bf16);
}

// NV: 8-column tiles of the value slice a CTA accumulates (even). VEC: every row piece is a whole number of aligned
// 16-byte vectors; otherwise tiles are staged element by element.
template <int NV, bool VEC>
__global__ void __launch_bounds__(kLpThreads, 1)
latent_prefill_mma_kernel(LatentPrefillArgs A) {
    extern __shared__ __align__(16) unsigned char lp_raw[];
    const int qk = A.dim + A.rot_dim, pitch = lp_qk_pitch(A.dim, A.rot_dim), ksteps = (pitch - 8) / 16;
    constexpr int vp = NV * 8 + 8;
    bf16* sq = reinterpret_cast<bf16*>(lp_raw);
    bf16* sk = sq + kLpM * pitch;
    bf16* sv = sk + 2 * kLpN * pitch;
    const bf16* Q = reinterpret_cast<const bf16*>(A.q);
    const bf16* KV = reinterpret_cast<const bf16*>(A.kv);
    const bf16* KR = reinterpret_cast<const bf16*>(A.kr);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, hk = h / A.rep, v_lo = blockIdx.z * NV * 8, v_n = min(NV * 8, A.vdim - v_lo);
    // long rows first: the last CTAs of a portion see the most keys
    const int q_lo = ((int)gridDim.x - 1 - (int)blockIdx.x) * kLpM, q_n = min(kLpM, A.n_q - q_lo);
    llvq_dependent_enter();

    // keys are addressed by their place in the operands; query i sees places i + off - window + 1 .. i + off
    const int off = (int)(A.pos0 - A.key0);
    const int k_end = min(A.n_k, q_lo + q_n - 1 + off + 1);
    const int k_begin = max(0, q_lo + off - A.window + 1);
    const int tiles = (k_end - k_begin + kLpN - 1) / kLpN;

    auto stage = [&](int t) {
        const int base = k_begin + t * kLpN;
        bf16* dk = sk + (t & 1) * kLpN * pitch;
        bf16* dv = sv + (t & 1) * kLpN * vp;
        if constexpr (VEC) {
            const int cn = A.dim / 8, cr = A.rot_dim / 8, ct = (pitch - 8) / 8;
            for (int i = tid; i < kLpN * ct; i += kLpThreads) {
                const int r = i / ct, c = i - r * ct, j = base + r;
                const bool in = j < k_end && c < cn + cr;
                const bf16* src = !in ? KV : c < cn ? KV + (size_t)j * A.ld_kv + (size_t)hk * A.k_head + 8 * c : KR + (size_t)j * A.ld_kr + 8 * (c - cn);
                copy16_async(dk + r * pitch + 8 * c, src, in);
            }
            for (int i = tid; i < kLpN * NV; i += kLpThreads) {
                const int r = i / NV, c = i - r * NV, j = base + r;
                const bool in = j < k_end && 8 * c < v_n;
                copy16_async(dv + r * vp + 8 * c, in ? KV + (size_t)j * A.ld_kv + A.v_off + (size_t)hk * A.v_head + v_lo + 8 * c : KV, in);
            }
        } else {
            for (int i = tid; i < kLpN * (pitch - 8); i += kLpThreads) {
                const int r = i / (pitch - 8), c = i - r * (pitch - 8), j = base + r;
                bf16 v = __float2bfloat16_rn(0.0f);
                if (j < k_end && c < qk) v = c < A.dim ? KV[(size_t)j * A.ld_kv + (size_t)hk * A.k_head + c] : KR[(size_t)j * A.ld_kr + c - A.dim];
                dk[r * pitch + c] = v;
            }
            for (int i = tid; i < kLpN * NV * 8; i += kLpThreads) {
                const int r = i / (NV * 8), c = i - r * (NV * 8), j = base + r;
                bf16 v = __float2bfloat16_rn(0.0f);
                if (j < k_end && c < v_n) v = KV[(size_t)j * A.ld_kv + A.v_off + (size_t)hk * A.v_head + v_lo + c];
                dv[r * vp + c] = v;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (tiles > 0) stage(0);

    // query tile, rotated; rows beyond the portion and columns beyond dim + rot_dim are zero
    {
        const size_t qrow = (size_t)A.heads * qk;
        const int half = A.rt.dims / 2;
        if constexpr (VEC) {
            const int cn = A.dim / 8;
            for (int i = tid; i < kLpM * cn; i += kLpThreads) {
                const int r = i / cn, c = i - r * cn;
                copy16_async(sq + r * pitch + 8 * c, r < q_n ? Q + (size_t)(q_lo + r) * qrow + (size_t)h * qk + 8 * c : Q, r < q_n);
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        } else {
            for (int i = tid; i < kLpM * A.dim; i += kLpThreads) {
                const int r = i / A.dim, c = i - r * A.dim;
                sq[r * pitch + c] = r < q_n ? Q[(size_t)(q_lo + r) * qrow + (size_t)h * qk + c] : __float2bfloat16_rn(0.0f);
            }
        }
        const int rest = A.rot_dim - half;  // pairs, then what passes
        for (int i = tid; i < kLpM * rest; i += kLpThreads) {
            const int r = i / rest, c = i - r * rest;
            bf16* dst = sq + r * pitch + A.dim;
            const bf16* src = Q + (size_t)(q_lo + r) * qrow + (size_t)h * qk + A.dim;
            if (c < half) {
                float a = 0.0f, b = 0.0f;
                if (r < q_n) {
                    const size_t p = (size_t)(A.pos0 + q_lo + r) * half + c;
                    const float cs = A.rt.cos_t[p], sn = A.rt.sin_t[p], u = to_f32(src[c]), v = to_f32(src[c + half]);
                    a = u * cs - v * sn;
                    b = v * cs + u * sn;
                }
                dst[c] = from_f32<bf16>(a);
                dst[c + half] = from_f32<bf16>(b);
            } else {
                dst[c + half] = r < q_n ? src[c + half] : __float2bfloat16_rn(0.0f);
            }
        }
        const int pad = pitch - 8 - qk;
        for (int i = tid; i < kLpM * pad; i += kLpThreads) sq[(i / pad) * pitch + qk + i % pad] = __float2bfloat16_rn(0.0f);
    }

    float o[NV][4];
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[n][j] = 0.0f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    const float s2 = A.scale * kLog2e;
    const int qa = q_lo + warp * 16 + off;  // place of the warp's first query among the keys
    const int row_lo = qa + (lane >> 2);    // this thread's rows: row_lo and row_lo + 8
    const int nv_used = (v_n + 7) / 8;

    for (int t = 0; t < tiles; ++t) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // tile t is staged, and every warp is done with the buffer of tile t + 1
        if (t + 1 < tiles) stage(t + 1);
        const int base = k_begin + t * kLpN;
        if (base > qa + 15 || base + kLpN - 1 < qa - A.window + 1 || warp * 16 >= q_n) continue;  // warp-uniform
        const bf16* tk = sk + (t & 1) * kLpN * pitch;
        const bf16* tv = sv + (t & 1) * kLpN * vp;
        float s[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int j = 0; j < 4; ++j) s[n][j] = 0.0f;
#pragma unroll 2
        for (int k = 0; k < ksteps; ++k) {
            unsigned int a[4];
            ldmatrix4(a, sq + (warp * 16 + (lane & 15)) * pitch + k * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int n = 0; n < 8; n += 2) {
                unsigned int b[4];
                ldmatrix4(b, tk + (n * 8 + (lane & 7) + (lane >> 4) * 8) * pitch + k * 16 + ((lane >> 3) & 1) * 8);
                mma_bf16(s[n], a, b[0], b[1]);
                mma_bf16(s[n + 1], a, b[2], b[3]);
            }
        }
        const bool edge = base + kLpN - 1 > qa || base < qa + 15 - A.window + 1 || base + kLpN > k_end;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float v = s[n][j] * s2;
                if (edge) {
                    const int key = base + n * 8 + (lane & 3) * 2 + (j & 1), row = row_lo + (j >> 1) * 8;
                    if (key > row || row - key >= A.window || key >= k_end) v = -INFINITY;
                }
                s[n][j] = v;
                mx[j >> 1] = fmaxf(mx[j >> 1], v);
            }
        float corr[2], base_m[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float mn = fmaxf(m[r], mx[r]);
            base_m[r] = mn == -INFINITY ? 0.0f : mn;  // a row that has seen no key yet
            corr[r] = exp2f(m[r] - base_m[r]);
            m[r] = mn;
            l[r] *= corr[r];
        }
        unsigned int p[8][2];
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            float e[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                e[j] = exp2f(s[n][j] - base_m[j >> 1]);
                l[j >> 1] += e[j];
            }
            p[n][0] = pack_bf16(e[0], e[1]);
            p[n][1] = pack_bf16(e[2], e[3]);
        }
#pragma unroll
        for (int n = 0; n < NV; ++n)
#pragma unroll
            for (int j = 0; j < 4; ++j) o[n][j] *= corr[j >> 1];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const unsigned int a[4] = {p[2 * k][0], p[2 * k][1], p[2 * k + 1][0], p[2 * k + 1][1]};
#pragma unroll
            for (int n = 0; n < NV; n += 2) {
                if (n >= nv_used) break;
                unsigned int b[4];
                ldmatrix4_trans(b, tv + (k * 16 + (lane & 15)) * vp + n * 8 + (lane >> 4) * 8);
                mma_bf16(o[n], a, b[0], b[1]);
                mma_bf16(o[n + 1], a, b[2], b[3]);
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (warp * 16 >= q_n) return;
    bf16* O = reinterpret_cast<bf16*>(A.out);
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        float f = 1.0f, den = l[r];
        if (A.sink) {
            const float sk2 = A.sink[h] * kLog2e, top = fmaxf(m[r], sk2);
            f = exp2f(m[r] - top);
            den = l[r] * f + exp2f(sk2 - top);
        }
        f /= den;
        const int row = q_lo + warp * 16 + (lane >> 2) + 8 * r;
        if (row >= A.n_q) continue;
        bf16* dst = O + (size_t)row * A.heads * A.vdim + (size_t)h * A.vdim + v_lo;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int c = n * 8 + (lane & 3) * 2;
            if constexpr (VEC) {
                if (c < v_n) *reinterpret_cast<unsigned int*>(dst + c) = pack_bf16(o[n][2 * r] * f, o[n][2 * r + 1] * f);
            } else {
                if (c < v_n) dst[c] = from_f32<bf16>(o[n][2 * r] * f);
                if (c + 1 < v_n) dst[c + 1] = from_f32<bf16>(o[n][2 * r + 1] * f);
            }
        }
    }
}

constexpr int kLsWarps = 8;

// grid = (ceil(n_q / 8), heads). Dynamic shared memory per warp: dim + rot_dim query values and vdim sums.
template <typename T>
__global__ void __launch_bounds__(kLsWarps * 32)
latent_prefill_simt_kernel(LatentPrefillArgs A) {
    extern __shared__ __align__(16) float ls_smem[];
    const int qk = A.dim + A.rot_dim, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.y, hk = h / A.rep;
    float* q_s = ls_smem + (size_t)warp * (qk + A.vdim);
    float* o_s = q_s + qk;
    llvq_dependent_enter();
    const int i = blockIdx.x * kLsWarps + warp;
    if (i >= A.n_q) return;
    const T* KV = reinterpret_cast<const T*>(A.kv);
    const T* KR = reinterpret_cast<const T*>(A.kr);
    const T* q = reinterpret_cast<const T*>(A.q) + ((size_t)i * A.heads + h) * qk;
    const long long pos = A.pos0 + i;
    const int half = A.rt.dims / 2;
    for (int c = lane; c < A.dim; c += 32) q_s[c] = to_f32(q[c]);
    for (int c = lane; c < A.rot_dim - half; c += 32) {
        if (c < half) {
            const float cs = A.rt.cos_t[pos * half + c], sn = A.rt.sin_t[pos * half + c];
            const float u = to_f32(q[A.dim + c]), v = to_f32(q[A.dim + half + c]);
            q_s[A.dim + c] = u * cs - v * sn;
            q_s[A.dim + half + c] = v * cs + u * sn;
        } else {
            q_s[A.dim + half + c] = to_f32(q[A.dim + half + c]);
        }
    }
    for (int c = lane; c < A.vdim; c += 32) o_s[c] = 0.0f;
    __syncwarp();
    const int last = min(A.n_k - 1, (int)(pos - A.key0)), first = max(0, (int)(pos - A.key0) - A.window + 1);
    const float s2 = A.scale * kLog2e;
    float m = -INFINITY, l = 0.0f;
    for (int base = first; base <= last; base += 32) {
        const int j = base + lane, here = min(32, last - base + 1);
        float s = -INFINITY;
        if (j <= last) {
            const T* k = KV + (size_t)j * A.ld_kv + (size_t)hk * A.k_head;
            const T* kr = KR + (size_t)j * A.ld_kr;
            float a = 0.0f;
            for (int c = 0; c < A.dim; ++c) a = fmaf(q_s[c], to_f32(k[c]), a);
            for (int c = 0; c < A.rot_dim; ++c) a = fmaf(q_s[A.dim + c], to_f32(kr[c]), a);
            s = a * s2;
        }
        const float mn = fmaxf(m, warp_max_f(s)), corr = exp2f(m - mn), p = exp2f(s - mn);
        l = l * corr + warp_sum_f(p);
        m = mn;
        const T* v = KV + (size_t)base * A.ld_kv + A.v_off + (size_t)hk * A.v_head;
        for (int c0 = 0; c0 < A.vdim; c0 += 32) {  // every lane takes part in the shuffles
            const int c = c0 + lane;
            const bool in = c < A.vdim;
            float a = in ? o_s[c] * corr : 0.0f;
            for (int t = 0; t < here; ++t) {
                const float pt = __shfl_sync(0xffffffffu, p, t);
                if (in) a = fmaf(pt, to_f32(v[(size_t)t * A.ld_kv + c]), a);
            }
            if (in) o_s[c] = a;
        }
    }
    float f = 1.0f, den = l;
    if (A.sink) {
        const float sk2 = A.sink[h] * kLog2e, top = fmaxf(m, sk2);
        f = exp2f(m - top);
        den = l * f + exp2f(sk2 - top);
    }
    f /= den;
    T* dst = reinterpret_cast<T*>(A.out) + ((size_t)i * A.heads + h) * A.vdim;
    for (int c = lane; c < A.vdim; c += 32) dst[c] = from_f32<T>(o_s[c] * f);
}

}  // namespace llvq
