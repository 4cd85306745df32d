// y = W a (+ bias) for one token over a dense row-major matrix (bf16 or f32), the activation formed in the
// kernel's own staging, as the archive-code GEMV does:
//
//   prologue  plain   a = x
//             embed   a = scale * table[token]            (also written out: the residual stream starts here)
//             norm    t = alpha * x + delta; a = t / sqrt(mean(t^2) + eps) * w   (optionally written out)
//             glu     a = clamped gated unit of [gate | up]
//   epilogue  y = W a + bias, f32; the head variant caps the logits (cap * tanh(y / cap)), stores them and
//             keeps the best (logit, row) of the CTA for lm_head_pick_kernel.
//
// The work is one pass over W. A CTA owns a contiguous range of rows, its warps are split into row groups and
// `kslices` column slices per group; a warp takes kGvRows rows at a time with 16-byte loads. The first loads
// are issued before the dependency wait: W does not depend on the kernel before. Partial sums of the column
// slices meet in shared memory and are added in slice order, so a row's result depends on nothing but the
// matrix shape. Rows are padded with zeros to whole 16-byte vectors (ldw), the staged activation likewise.
#pragma once
#include "dense_elem.cuh"
#include "head_pick.cuh"

namespace llvq {

constexpr int kGvThreads = 256;
constexpr int kGvWarps = kGvThreads / 32;
constexpr int kGvRows = 4;

enum GemvPrologue { kGvPlain = 0, kGvEmbed = 1, kGvNorm = 2, kGvGlu = 3 };

struct DenseGemvArgs {
    const void* w;        // [n_out, ldw] of T
    const float* bias;    // [n_out] or null
    float* y;             // [n_out] f32 (head: the capped logits, or null)
    const float* x;       // plain, norm: [k]; glu: [gate k | up k]
    const float* delta;   // norm: [k] or null
    const float* norm_w;  // norm: [k], the factor as applied
    float* a_out;         // embed, norm: the staged activation is also written here by CTA 0 (or null)
    const void* table;    // embed: [table_rows, ld_table] of T
    const long long* token;
    HeadBest* best;       // head: one candidate per CTA
    int n_out, k, ldw, ld_table, table_rows;
    int kslices;          // 1, 2, 4 or 8
    float alpha, eps;     // norm
    float scale;          // embed
    float limit, gain, shift;  // glu
    float cap;            // head: 0 = no cap
};

template <typename T, int PRO, bool HEAD>
__global__ void __launch_bounds__(kGvThreads)
dense_gemv_kernel(DenseGemvArgs A) {
    constexpr int VN = Vec16<T>::N;
    extern __shared__ __align__(16) float gv_smem[];
    __shared__ float red[kGvWarps];
    __shared__ HeadBest best_s[kGvWarps];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int r0 = (int)((long long)A.n_out * blockIdx.x / gridDim.x), r1 = (int)((long long)A.n_out * (blockIdx.x + 1) / gridDim.x);
    const int groups = kGvWarps / A.kslices, group = warp / A.kslices, slice = warp % A.kslices;
    const int vecs = A.ldw / VN, v0 = slice * 32 + lane, vstep = 32 * A.kslices;
    float* a_s = gv_smem;
    float* part = gv_smem + A.ldw;  // [rows of the CTA][kslices]
    const uint4* W = reinterpret_cast<const uint4*>(A.w);

    int row = r0 + group * kGvRows;
    uint4 w[kGvRows];
    const bool first = row < r1 && v0 < vecs;
    if (first) {
#pragma unroll
        for (int i = 0; i < kGvRows; ++i) w[i] = __ldg(W + (size_t)min(row + i, r1 - 1) * vecs + v0);
    }
    llvq_dependent_enter();

    if constexpr (PRO == kGvPlain) {
        for (int i = tid; i < A.ldw; i += kGvThreads) a_s[i] = i < A.k ? A.x[i] : 0.0f;
    } else if constexpr (PRO == kGvEmbed) {
        long long t = *A.token;
        if (t < 0 || t >= A.table_rows) t = 0;  // a token outside the vocabulary reads row 0 instead of foreign memory
        const T* src = reinterpret_cast<const T*>(A.table) + (size_t)t * A.ld_table;
        for (int i = tid; i < A.ldw; i += kGvThreads) {
            const float v = i < A.k ? A.scale * to_f32(src[i]) : 0.0f;
            a_s[i] = v;
            if (blockIdx.x == 0 && A.a_out && i < A.k) A.a_out[i] = v;
        }
    } else if constexpr (PRO == kGvNorm) {
        float ss = 0.0f;
        for (int i = tid; i < A.ldw; i += kGvThreads) {
            float t = 0.0f;
            if (i < A.k) {
                t = A.alpha * A.x[i];
                if (A.delta) t += A.delta[i];
            }
            a_s[i] = t;
            ss = fmaf(t, t, ss);
        }
        const float r = 1.0f / sqrtf(block_sum_f(ss, red) / (float)A.k + A.eps);
        for (int i = tid; i < A.k; i += kGvThreads) {  // the element this thread wrote above
            const float v = a_s[i] * r * A.norm_w[i];
            a_s[i] = v;
            if (blockIdx.x == 0 && A.a_out) A.a_out[i] = v;
        }
    } else {
        for (int i = tid; i < A.ldw; i += kGvThreads)
            a_s[i] = i < A.k ? clamped_glu(A.x[i], A.x[A.k + i], A.limit, A.gain, A.shift) : 0.0f;
    }
    __syncthreads();

    bool have = first;
    for (; row < r1; row += groups * kGvRows) {
        float acc[kGvRows];
#pragma unroll
        for (int i = 0; i < kGvRows; ++i) acc[i] = 0.0f;
        for (int v = v0; v < vecs; v += vstep) {
            if (!have) {
#pragma unroll
                for (int i = 0; i < kGvRows; ++i) w[i] = __ldg(W + (size_t)min(row + i, r1 - 1) * vecs + v);
            }
            have = false;
            float a[VN];
#pragma unroll
            for (int j = 0; j < VN; j += 4) {
                const float4 q = *reinterpret_cast<const float4*>(a_s + v * VN + j);
                a[j] = q.x, a[j + 1] = q.y, a[j + 2] = q.z, a[j + 3] = q.w;
            }
#pragma unroll
            for (int i = 0; i < kGvRows; ++i) {
                float f[VN];
                Vec16<T>::widen(w[i], f);
#pragma unroll
                for (int j = 0; j < VN; ++j) acc[i] = fmaf(f[j], a[j], acc[i]);
            }
        }
        have = false;
#pragma unroll
        for (int i = 0; i < kGvRows; ++i) {
            const float s = warp_sum_f(acc[i]);
            if (lane == 0 && row + i < r1) part[(row + i - r0) * A.kslices + slice] = s;
        }
    }
    __syncthreads();
    HeadBest b{-INFINITY, 0x7fffffff};
    for (int r = r0 + tid; r < r1; r += kGvThreads) {
        float s = 0.0f;
        for (int k = 0; k < A.kslices; ++k) s += part[(r - r0) * A.kslices + k];
        if (A.bias) s += A.bias[r];
        if constexpr (HEAD) {
            if (A.cap > 0.0f) s = A.cap * tanhf(s / A.cap);
            if (head_better(s, r, b.val, b.row)) b = HeadBest{s, r};
            if (A.y) A.y[r] = s;
        } else {
            A.y[r] = s;
        }
    }
    if constexpr (HEAD) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float v = __shfl_xor_sync(0xffffffffu, b.val, o);
            const int r = __shfl_xor_sync(0xffffffffu, b.row, o);
            if (head_better(v, r, b.val, b.row)) b = HeadBest{v, r};
        }
        if (lane == 0) best_s[warp] = b;
        __syncthreads();
        if (tid == 0) {
            for (int k = 1; k < kGvWarps; ++k)
                if (head_better(best_s[k].val, best_s[k].row, b.val, b.row)) b = best_s[k];
            A.best[blockIdx.x] = b;
        }
    }
}

}  // namespace llvq
