// Grouped-query attention over a ring of cached rows, the token step, and the row kernels of a prompt portion around
// its attention (whose kernels are those of latent_prefill*.cuh: keys and values of a head apart, nothing rotated).
//
// A cached row is [kv_heads keys | kv_heads values], every head padded with zeros to whole 16-byte vectors; position p
// sits in slot p % slots. Queries and keys are RMS normed per head with weights of their own before they meet.
//
//   gqa_token            a CTA takes four query heads of one key/value head and one split of the visible positions, in
//                        tiles of 64: thread = (position, quarter of the key) for the scores, (position group, value
//                        vector) for the sums; online softmax in base 2, f32. The CTA whose split holds the token itself
//                        norms its key; the first of a group stores the cache row. The last split to arrive merges them
//                        all in order, gates the heads and scales them: no CTA waits for another.
//   gqa_rows_kernel      a portion: queries normed, cache rows stored.
//   gate_rows_kernel     out = x * sigmoid(gate) * scale.
#pragma once
#include "latent_attn.cuh"

namespace llvq {

constexpr int kGqHeads = 4, kGqTile = 64, kGqThreads = 256, kGqMaxSplits = 128;

struct GqaRing {
    void* rows;  // [slots, ld] of T
    int slots, ld;
    int kd, vd;  // a head's key and value, padded; the values start at kv_heads * kd
};

struct GqaArgs {
    const float* q;       // [heads, dim]
    const float* k;       // [kv_heads, dim]
    const float* v;       // [kv_heads, vdim]
    const float* gate;    // [heads, vdim] before the sigmoid, or null
    const float* q_norm;  // [dim], as applied
    const float* k_norm;
    const long long* pos;
    float* part_ml;       // [heads, splits, 2]
    float* part_o;        // [heads, splits, vdim]
    unsigned int* arrived; // [units], zero before the first launch and after every one
    float* out;           // [heads, vdim]
    GqaRing ring;
    int heads, kv_heads, dim, vdim, window, splits;
    float scale, eps, out_scale;
};

__host__ __device__ inline int gqa_chunks(int heads, int kv_heads) { return (heads / kv_heads + kGqHeads - 1) / kGqHeads; }
inline int gqa_ctas(int heads, int kv_heads, int splits) { return kv_heads * gqa_chunks(heads, kv_heads) * splits; }
// Shared memory of one CTA: queries, quarter scores, weights, split factors, and the tile of keys and values, whose place the
// sums take afterwards. A tile has fewer than 64 positions where the rows are long.
template <typename T>
__host__ __device__ inline int gqa_key_pitch(int kd) { return kd + (kd / Vec16<T>::N % 2 ? 0 : Vec16<T>::N); }  // an odd number of vectors
template <typename T>
__host__ __device__ inline int gqa_tile(int kd, int vd) {
    int tile = kGqTile;
    while (tile > 8 && (size_t)tile * (gqa_key_pitch<T>(kd) + vd) * sizeof(T) > 96 * 1024) tile /= 2;
    return tile;
}
template <typename T>
inline size_t gqa_token_smem(int kd, int vd) {
    const size_t tile = (size_t)gqa_tile<T>(kd, vd) * (gqa_key_pitch<T>(kd) + vd) * sizeof(T), sums = (size_t)kGqHeads * kGqThreads * Vec16<T>::N * 4;
    return (tile > sums ? tile : sums) + (size_t)kGqHeads * kd * 4 + (size_t)5 * kGqHeads * kGqTile * 4 + (size_t)kGqHeads * kGqMaxSplits * 4 + 64;
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

// sigmoid, silu and gelu for results that are rounded to T: in bf16 the fast exponential and division are far inside the rounding.
template <typename T>
__device__ __forceinline__ float sigmoid_t(float x) {
    if constexpr (sizeof(T) == 2) return __fdividef(1.0f, 1.0f + __expf(-x));
    return sigmoid_f(x);
}
template <typename T>
__device__ __forceinline__ float silu_t(float x) { return x * sigmoid_t<T>(x); }

// 1 / rms of a row by one warp, the same value in every lane.
template <typename X>
__device__ __forceinline__ float warp_inv_rms(const X* x, int n, float eps) {
    float ss = 0.0f;
    for (int i = threadIdx.x & 31; i < n; i += 32) {
        const float v = to_f32(x[i]);
        ss = fmaf(v, v, ss);
    }
    return 1.0f / sqrtf(warp_sum_f(ss) / (float)n + eps);
}

// One CTA's part of the token step. `smem` holds gqa_token_smem bytes. The caller has passed the dependency wait.
template <typename T>
__device__ __forceinline__ void gqa_token(const GqaArgs& A, int cta, unsigned char* smem) {
    constexpr int VN = Vec16<T>::N;
    __shared__ float corr_s[kGqHeads], inv_s[kGqHeads];
    __shared__ int last_s;
    const int kd = A.ring.kd, vd = A.ring.vd, kvecs = kd / VN, vvecs = vd / VN, kp = gqa_key_pitch<T>(kd), tile = gqa_tile<T>(kd, vd);
    float* q_s = reinterpret_cast<float*>(smem);                                 // [4][kd]
    float* s_s = q_s + kGqHeads * kd;                                            // [quarter][4][64]
    float* p_s = s_s + 4 * kGqHeads * kGqTile;                                   // [4][64]
    float* f_s = p_s + kGqHeads * kGqTile;                                       // [4][splits]
    T* k_s = reinterpret_cast<T*>(f_s + kGqHeads * kGqMaxSplits);                // [tile][kp]
    T* v_s = k_s + (size_t)tile * kp;                                            // [tile][vd]
    float* red = reinterpret_cast<float*>(k_s);                                  // [rows][4][values], at most 4 * 256 * VN
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int unit = cta / A.splits, split = cta - unit * A.splits, chunks = gqa_chunks(A.heads, A.kv_heads);
    const int g = unit / chunks, chunk = unit - g * chunks, rep = A.heads / A.kv_heads;
    const int head0 = g * rep + chunk * kGqHeads, nh = min(kGqHeads, rep - chunk * kGqHeads);
    const long long pos = *A.pos;
    const int n = (int)min((long long)A.window, pos + 1);  // visible positions pos - n + 1 .. pos
    int per = (n + A.splits - 1) / A.splits;
    per = (per + tile - 1) / tile * tile;
    const int t0 = split * per, t1 = min(n, t0 + per);
    const bool own = t0 < n && t1 == n;  // this split holds the token itself
    const int slot_new = (int)((unsigned int)pos % (unsigned int)A.ring.slots);
    const int slot0 = slot_new - n + 1 + (slot_new < n - 1 ? A.ring.slots : 0);  // n <= slots: at most one wrap below
    T* row_new = reinterpret_cast<T*>(A.ring.rows) + (size_t)slot_new * A.ring.ld;

    // positions base .. of this split into the tile, the token's own row aside
    auto stage = [&](int base) {
        const int here = min(tile, t1 - base), per_row = kvecs + vvecs;
        int r = tid / per_row, c = tid - r * per_row;
        const int dr = kGqThreads / per_row, dc = kGqThreads - dr * per_row;
#pragma unroll 1
        while (r < here) {
            int slot = slot0 + base + r;
            if (slot >= A.ring.slots) slot -= A.ring.slots;
            const T* src = reinterpret_cast<const T*>(A.ring.rows) + (size_t)slot * A.ring.ld;
            src += c < kvecs ? (size_t)g * kd + c * VN : (size_t)A.kv_heads * kd + (size_t)g * vd + (c - kvecs) * VN;
            T* dst = c < kvecs ? k_s + (size_t)r * kp + c * VN : v_s + (size_t)r * vd + (c - kvecs) * VN;
            if (base + r != n - 1)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned int)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
            c += dc;
            r += dr;
            if (c >= per_row) c -= per_row, ++r;
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (t0 < t1) stage(t0);
    T* k_new = k_s + (size_t)(max(n - 1 - t0, 0) % tile) * kp;  // the token's own place, where this split holds it
    T* v_new = v_s + (size_t)(max(n - 1 - t0, 0) % tile) * vd;

    if (warp < nh && t0 < t1) {
        const float* q = A.q + (size_t)(head0 + warp) * A.dim;
        const float f = warp_inv_rms(q, A.dim, A.eps) * A.scale * kLog2e;
        for (int i = lane; i < kd; i += 32) q_s[warp * kd + i] = i < A.dim ? q[i] * f * A.q_norm[i] : 0.0f;
    } else if (warp < kGqHeads) {
        for (int i = lane; i < kd; i += 32) q_s[warp * kd + i] = 0.0f;
    }
    // its normed key and its value: stored once per group, and kept by every CTA whose split ends with it
    auto own_row = [&]() {
        if (warp == kGqHeads) {
            const float* k = A.k + (size_t)g * A.dim;
            const float f = warp_inv_rms(k, A.dim, A.eps);
            for (int i = lane; i < kd; i += 32) {
                const T t = from_f32<T>(i < A.dim ? k[i] * f * A.k_norm[i] : 0.0f);
                k_new[i] = t;
                if (chunk == 0) row_new[(size_t)g * kd + i] = t;
            }
        } else if (warp == kGqHeads + 1) {
            const float* v = A.v + (size_t)g * A.vdim;
            for (int i = lane; i < vd; i += 32) {
                const T t = from_f32<T>(i < A.vdim ? v[i] : 0.0f);
                v_new[i] = t;
                if (chunk == 0) row_new[(size_t)A.kv_heads * kd + (size_t)g * vd + i] = t;
            }
        }
    };
    int vl = 1;  // threads along the value vectors
    while (vl < vvecs) vl *= 2;
    const int vi = tid & (vl - 1), grp = tid / vl, grps = kGqThreads / vl;

    float m = -INFINITY, l = 0.0f;  // of head `warp`, in warps below nh
    float acc[kGqHeads][VN];
#pragma unroll
    for (int h = 0; h < kGqHeads; ++h)
#pragma unroll
        for (int j = 0; j < VN; ++j) acc[h][j] = 0.0f;
#pragma unroll 1
    for (int base = t0; base < t1; base += tile) {
        const int here = min(tile, t1 - base);
        if (own && base + here == n) own_row();
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        {  // scores: thread = (position, quarter of the key's vectors)
            const int p = tid & (kGqTile - 1), quarter = tid / kGqTile;
            float s[kGqHeads] = {0.0f, 0.0f, 0.0f, 0.0f};
            if (p < here) {
                const uint4* kr = reinterpret_cast<const uint4*>(k_s + (size_t)p * kp);
#pragma unroll 1
                for (int c = quarter; c < kvecs; c += 4) {
                    float f[VN];
                    Vec16<T>::widen(kr[c], f);
#pragma unroll
                    for (int h = 0; h < kGqHeads; ++h)
#pragma unroll
                        for (int j = 0; j < VN; j += 4) {
                            const float4 qv = *reinterpret_cast<const float4*>(q_s + h * kd + c * VN + j);
                            s[h] = fmaf(f[j], qv.x, s[h]);
                            s[h] = fmaf(f[j + 1], qv.y, s[h]);
                            s[h] = fmaf(f[j + 2], qv.z, s[h]);
                            s[h] = fmaf(f[j + 3], qv.w, s[h]);
                        }
                }
            }
#pragma unroll
            for (int h = 0; h < kGqHeads; ++h) s_s[(quarter * kGqHeads + h) * kGqTile + p] = s[h];
        }
        __syncthreads();
        if (warp < kGqHeads) {
            float s[2];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int p = lane + 32 * k;
                s[k] = -INFINITY;
                if (p < here) {
                    s[k] = 0.0f;
#pragma unroll
                    for (int quarter = 0; quarter < 4; ++quarter) s[k] += s_s[(quarter * kGqHeads + warp) * kGqTile + p];
                }
            }
            const float mn = fmaxf(m, warp_max_f(fmaxf(s[0], s[1])));  // finite: a tile holds a visible position
            const float corr = exp2f(m - mn), e0 = exp2f(s[0] - mn), e1 = exp2f(s[1] - mn);
            l = l * corr + warp_sum_f(e0 + e1);
            m = mn;
            p_s[warp * kGqTile + lane] = e0;
            p_s[warp * kGqTile + lane + 32] = e1;
            if (lane == 0) corr_s[warp] = corr;
        }
        __syncthreads();
        if (base > t0) {
#pragma unroll
            for (int h = 0; h < kGqHeads; ++h)
#pragma unroll
                for (int j = 0; j < VN; ++j) acc[h][j] *= corr_s[h];
        }
        if (vi < vvecs) {
#pragma unroll 1
            for (int p = grp; p < here; p += grps) {
                float f[VN];
                Vec16<T>::widen(reinterpret_cast<const uint4*>(v_s + (size_t)p * vd)[vi], f);
#pragma unroll
                for (int h = 0; h < kGqHeads; ++h) {
                    const float w = p_s[h * kGqTile + p];
#pragma unroll
                    for (int j = 0; j < VN; ++j) acc[h][j] = fmaf(w, f[j], acc[h][j]);
                }
            }
        }
        __syncthreads();  // the tile is read
        if (base + tile < t1) stage(base + tile);
    }
    if (warp < nh && lane == 0) {
        float* ml = A.part_ml + ((size_t)(head0 + warp) * A.splits + split) * 2;
        ml[0] = m;  // -inf for a split beyond the visible positions
        ml[1] = l;
    }
    if (t0 < t1) {
        // the position groups' sums: those of a warp by shuffles, then the warps' (or, of values wider than a warp, the groups')
        for (int o = vl; o < 32; o *= 2)
#pragma unroll
            for (int h = 0; h < kGqHeads; ++h)
#pragma unroll
                for (int j = 0; j < VN; ++j) acc[h][j] += __shfl_xor_sync(0xffffffffu, acc[h][j], o);
        const int row = vl < 32 ? warp : grp, rows = vl < 32 ? kGqThreads / 32 : grps, width = vl * VN;
        if (vl >= 32 || lane < vl) {
#pragma unroll
            for (int h = 0; h < kGqHeads; ++h)
#pragma unroll
                for (int j = 0; j < VN; j += 4)
                    *reinterpret_cast<float4*>(red + ((size_t)row * kGqHeads + h) * width + vi * VN + j) =
                        make_float4(acc[h][j], acc[h][j + 1], acc[h][j + 2], acc[h][j + 3]);
        }
        __syncthreads();
        for (int e = tid; e < nh * width; e += kGqThreads) {
            const int h = e / width, d = e - h * width;
            if (d >= A.vdim) continue;
            float o = 0.0f;
            for (int k = 0; k < rows; ++k) o += red[((size_t)k * kGqHeads + h) * width + d];
            A.part_o[((size_t)(head0 + h) * A.splits + split) * A.vdim + d] = o;
        }
    }
    // ---- the last split to arrive merges ----
    __threadfence();
    __syncthreads();
    if (tid == 0) last_s = atomicAdd(A.arrived + unit, 1u) == (unsigned int)A.splits - 1u;
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    if (tid == 0) A.arrived[unit] = 0;
    if (warp < nh) {
        const float* ml = A.part_ml + (size_t)(head0 + warp) * A.splits * 2;
        float mt = -INFINITY, lt = 0.0f;
        for (int s = lane; s < A.splits; s += 32) mt = fmaxf(mt, __ldcg(ml + 2 * s));
        mt = warp_max_f(mt);
        for (int s = lane; s < A.splits; s += 32) {
            const float ms = __ldcg(ml + 2 * s), f = ms == -INFINITY ? 0.0f : exp2f(ms - mt);
            f_s[warp * kGqMaxSplits + s] = f;
            lt = fmaf(__ldcg(ml + 2 * s + 1), f, lt);
        }
        lt = warp_sum_f(lt);
        if (lane == 0) inv_s[warp] = A.out_scale / lt;
    }
    __syncthreads();
    for (int e = tid; e < nh * A.vdim; e += kGqThreads) {
        const int h = e / A.vdim, d = e - h * A.vdim;
        const size_t at = (size_t)(head0 + h) * A.vdim + d;
        const float* po = A.part_o + (size_t)(head0 + h) * A.splits * A.vdim + d;
        float o = 0.0f;
#pragma unroll 4
        for (int s = 0; s < A.splits; ++s) {
            const float f = f_s[h * kGqMaxSplits + s];
            if (f != 0.0f) o = fmaf(__ldcg(po + (size_t)s * A.vdim), f, o);  // the sums of an empty split are not written
        }
        o *= inv_s[h];
        A.out[at] = A.gate ? o * sigmoid_f(A.gate[at]) : o;
    }
}

// ---- prompt portions ----

struct GqaRowsArgs {
    const void* q;  // rows of one product, stride ldy: [heads, dim], [kv_heads, dim], [kv_heads, vdim]
    const void* k;
    const void* v;
    void* qn;       // [rows, heads * dim] of T
    const float* q_norm;
    const float* k_norm;
    GqaRing ring;
    long long pos0;
    int ldy, heads, kv_heads, dim, vdim;
    float eps;
    int vec;        // heads and rows are whole 16-byte vectors on 16-byte boundaries
};

// out = x / rms(x) * w of n values by half a warp (lanes 0 .. 15 of it), in whole vectors.
template <typename T>
__device__ __forceinline__ void half_warp_norm(const T* x, const float* w, T* out, int n, float eps) {
    constexpr int VN = Vec16<T>::N;
    const int lane = threadIdx.x & 15;
    const unsigned int mask = 0xffffu << (threadIdx.x & 16);
    float ss = 0.0f, f[VN];
    for (int i = lane * VN; i < n; i += 16 * VN) {
        load_vec(x + i, f);
#pragma unroll
        for (int j = 0; j < VN; ++j) ss = fmaf(f[j], f[j], ss);
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
    const float r = 1.0f / sqrtf(ss / (float)n + eps);
    for (int i = lane * VN; i < n; i += 16 * VN) {
        if (n > 16 * VN) load_vec(x + i, f);  // else it is still there
#pragma unroll
        for (int j = 0; j < VN; ++j) f[j] *= r * w[i + j];
        store_vec(out + i, f);
    }
}

// grid = rows, 256 threads: a warp takes a head at a time, or each of its halves one.
template <typename T>
__global__ void __launch_bounds__(256)
gqa_rows_kernel(GqaRowsArgs A) {
    llvq_dependent_enter();
    const size_t o = (size_t)blockIdx.x * A.ldy;
    const long long pos = A.pos0 + blockIdx.x;
    T* row = reinterpret_cast<T*>(A.ring.rows) + (size_t)(pos % A.ring.slots) * A.ring.ld;
    const T* Q = reinterpret_cast<const T*>(A.q) + o;
    const T* K = reinterpret_cast<const T*>(A.k) + o;
    const T* V = reinterpret_cast<const T*>(A.v) + o;
    T* QN = reinterpret_cast<T*>(A.qn) + (size_t)blockIdx.x * A.heads * A.dim;
    T* rv = row + (size_t)A.kv_heads * A.ring.kd;
    if (A.vec) {
        constexpr int VN = Vec16<T>::N;
        const int lane = threadIdx.x & 15;
        for (int u = threadIdx.x >> 4; u < A.heads + 2 * A.kv_heads; u += 16) {
            if (u < A.heads) {
                half_warp_norm(Q + (size_t)u * A.dim, A.q_norm, QN + (size_t)u * A.dim, A.dim, A.eps);
            } else if (u < A.heads + A.kv_heads) {
                half_warp_norm(K + (size_t)(u - A.heads) * A.dim, A.k_norm, row + (size_t)(u - A.heads) * A.ring.kd, A.dim, A.eps);
            } else {
                const int g = u - A.heads - A.kv_heads;
                for (int i = lane * VN; i < A.vdim; i += 16 * VN)
                    *reinterpret_cast<uint4*>(rv + (size_t)g * A.ring.vd + i) = *reinterpret_cast<const uint4*>(V + (size_t)g * A.vdim + i);
            }
        }
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int u = warp; u < A.heads + 2 * A.kv_heads; u += 8) {
        if (u < A.heads) {
            const T* q = Q + (size_t)u * A.dim;
            const float f = warp_inv_rms(q, A.dim, A.eps);
            for (int i = lane; i < A.dim; i += 32) QN[(size_t)u * A.dim + i] = from_f32<T>(to_f32(q[i]) * f * A.q_norm[i]);
        } else if (u < A.heads + A.kv_heads) {
            const int g = u - A.heads;
            const T* k = K + (size_t)g * A.dim;
            const float f = warp_inv_rms(k, A.dim, A.eps);
            for (int i = lane; i < A.dim; i += 32) row[(size_t)g * A.ring.kd + i] = from_f32<T>(to_f32(k[i]) * f * A.k_norm[i]);
        } else {
            const int g = u - A.heads - A.kv_heads;
            for (int i = lane; i < A.vdim; i += 32) rv[(size_t)g * A.ring.vd + i] = V[(size_t)g * A.vdim + i];
        }
    }
}

// out[r, c] = x[r, c] * sigmoid(gate[r, c]) * scale; grid = (rows, ceil(n / (1024, or with vec 2048))). vec: whole 16-byte
// vectors on 16-byte boundaries.
template <typename T>
__global__ void __launch_bounds__(256)
gate_rows_kernel(const T* __restrict__ x, int ldx, const T* __restrict__ gate, int ldg, T* __restrict__ out, int ldo, int n, float scale, int vec) {
    llvq_dependent_enter();
    const size_t r = blockIdx.x;
    if (vec) {
        constexpr int VN = Vec16<T>::N, K = 8 / VN;
#pragma unroll
        for (int k = 0; k < K; ++k) {
            const int c = ((blockIdx.y * K + k) * 256 + threadIdx.x) * VN;
            if (c >= n) break;
            float f[VN], g[VN];
            load_vec(x + r * ldx + c, f);
            load_vec(gate + r * ldg + c, g);
#pragma unroll
            for (int j = 0; j < VN; ++j) f[j] *= scale * sigmoid_t<T>(g[j]);
            store_vec(out + r * ldo + c, f);
        }
        return;
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const int c = (blockIdx.y * 4 + k) * 256 + threadIdx.x;
        if (c < n) out[r * ldo + c] = from_f32<T>(to_f32(x[r * ldx + c]) * scale * sigmoid_t<T>(to_f32(gate[r * ldg + c])));
    }
}

}  // namespace llvq
