// y = W a (+ bias) for one token over a dense row-major matrix (bf16 or f32), the activation formed in the
// kernel's own staging, as the archive-code GEMV does:
//
//   prologue  plain   a = x
//             embed   a = scale * table[token]            (also written out: the residual stream starts here)
//             norm    t = alpha * x + delta; a = t / sqrt(mean(t^2) + eps) * w   (optionally written out)
//   epilogue  y = W a + bias, f32; or, with the rows of W in pairs (gate, up), the clamped gated unit of each pair;
//             the head variant caps the logits (cap * tanh(y / cap)), stores them and keeps the best (logit, row)
//             of the CTA for lm_head_pick_kernel.
//
// The work is one pass over W. Two kernels:
//
//   dense_gemv_stream_kernel (bf16)  one CTA per SM owns a contiguous range of rows; every warp is bound to one
//       column segment, keeps the activation of that segment in registers and walks the CTA's rows, two at a time,
//       with a ring of bulk copies of its own (row segment -> shared memory, one mbarrier per slot). The ring is
//       filled, and the norm's weights are read, before the dependency wait: neither depends on the kernel before,
//       so a small matrix is on the chip by the time its activation exists. The norm's 1 / rms is one factor of the
//       whole product and is applied to the row sums, so no warp waits for another until those are added.
//   dense_gemv_kernel (f32, and rows too long for the ring)  loads straight into registers.
//
// In the second, a CTA owns a contiguous range of rows, its warps are split into row groups and
// `kslices` column slices per group; a warp takes kGvRows rows at a time with 16-byte loads. The first loads
// are issued before the dependency wait. In both, partial sums of the column slices meet in shared memory and are
// added in slice order, so a row's result depends on nothing but the matrix shape. Rows are padded with zeros to
// whole 16-byte vectors (ldw), the staged activation likewise.
#pragma once
#include "dense_elem.cuh"
#include "head_pick.cuh"
#include "mbarrier.cuh"

namespace llvq {

constexpr int kGvThreads = 256;
constexpr int kGvWarps = kGvThreads / 32;
constexpr int kGvRows = 4;

enum GemvPrologue { kGvPlain = 0, kGvEmbed = 1, kGvNorm = 2 };

struct DenseGemvArgs {
    const void* w;        // [n_out, ldw] of T
    const float* bias;    // [n_out] or null
    float* y;             // [n_out] f32 (gated unit: [n_out / 2]; head: the capped logits, or null)
    const float* x;       // plain, norm: [k]
    const float* delta;   // norm: [k] or null
    const float* norm_w;  // norm: [k], the factor as applied
    float* a_out;         // embed, norm: the staged activation is also written here by CTA 0 (or null)
    const void* table;    // embed: [table_rows, ld_table] of T
    const long long* token;
    HeadBest* best;       // head: one candidate per CTA
    int n_out, k, ldw, ld_table, table_rows;
    int glu;              // rows are (gate, up) pairs: one output per pair
    int kslices;          // 1, 2, 4 or 8
    float alpha, eps;     // norm
    float scale;          // embed
    float limit, gain, shift;  // gated unit
    float cap;            // head: 0 = no cap
    // stream kernel: column segments (1, 2, 4 or 8), vectors of a segment, ring slots of a warp
    int nseg, segv, slots;
    int vec_x;            // x, delta and norm_w may be read 16 bytes at a time
    unsigned int* err;    // bit 0: a copy did not land in time
};

// First row of a CTA's range; pairs stay together.
__device__ __forceinline__ int gemv_row(const DenseGemvArgs& A, int cta) {
    return A.glu ? 2 * (int)((long long)(A.n_out / 2) * cta / gridDim.x) : (int)((long long)A.n_out * cta / gridDim.x);
}

// y of the rows [r0, r1) of a CTA from the partial sums of their segments, times `factor`.
template <bool HEAD>
__device__ __forceinline__ void gemv_finish(const DenseGemvArgs& A, const float* part, int segments, float factor, int r0, int r1, HeadBest* best_s) {
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    auto row_sum = [&](int r) {
        float s = 0.0f;
        for (int k = 0; k < segments; ++k) s += part[(r - r0) * segments + k];
        s *= factor;
        return A.bias ? s + A.bias[r] : s;
    };
    if constexpr (!HEAD) {
        if (A.glu) {
            for (int i = r0 / 2 + tid; i < r1 / 2; i += kGvThreads)
                A.y[i] = clamped_glu(row_sum(2 * i), row_sum(2 * i + 1), A.limit, A.gain, A.shift);
        } else {
            for (int r = r0 + tid; r < r1; r += kGvThreads) A.y[r] = row_sum(r);
        }
    } else {
        HeadBest b{-INFINITY, 0x7fffffff};
        for (int r = r0 + tid; r < r1; r += kGvThreads) {
            float s = row_sum(r);
            if (A.cap > 0.0f) s = A.cap * tanhf(s / A.cap);
            if (head_better(s, r, b.val, b.row)) b = HeadBest{s, r};
            if (A.y) A.y[r] = s;
        }
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

template <typename T, int PRO, bool HEAD>
__global__ void __launch_bounds__(kGvThreads)
dense_gemv_kernel(DenseGemvArgs A) {
    constexpr int VN = Vec16<T>::N;
    extern __shared__ __align__(16) float gv_smem[];
    __shared__ float red[kGvWarps];
    __shared__ HeadBest best_s[kGvWarps];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int r0 = gemv_row(A, blockIdx.x), r1 = gemv_row(A, blockIdx.x + 1);
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
    } else {
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
    gemv_finish<HEAD>(A, part, A.kslices, 1.0f, r0, r1, best_s);
}

constexpr int kGsRingBytes = 11 * 1024;  // of a warp: two CTAs (this launch's and the next one's) fit an SM together
constexpr int kGsMaxSlots = 8;
constexpr int kGsMaxVpl = 10;            // activation vectors a lane can keep

// Eight consecutive activation values from column c on; zeros beyond k.
__device__ __forceinline__ void gs_load8(const float* p, int c, int k, int vec, float (&f)[8]) {
    if (vec && c + 8 <= k) {
        const float4 u = *reinterpret_cast<const float4*>(p + c), v = *reinterpret_cast<const float4*>(p + c + 4);
        f[0] = u.x, f[1] = u.y, f[2] = u.z, f[3] = u.w, f[4] = v.x, f[5] = v.y, f[6] = v.z, f[7] = v.w;
    } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = c + j < k ? p[c + j] : 0.0f;
    }
}

template <int VPL, int PRO, bool HEAD>
__global__ void __launch_bounds__(kGvThreads, 2)
dense_gemv_stream_kernel(DenseGemvArgs A) {
    extern __shared__ __align__(128) unsigned char gs_raw[];
    __shared__ __align__(8) unsigned long long bars[kGvWarps][kGsMaxSlots];
    __shared__ float red[kGvWarps];
    __shared__ HeadBest best_s[kGvWarps];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r0 = gemv_row(A, blockIdx.x), r1 = gemv_row(A, blockIdx.x + 1);
    const int seg = warp % A.nseg, group = warp / A.nseg, groups = kGvWarps / A.nseg;
    const int nv = min(A.segv, A.ldw / 8 - seg * A.segv);      // vectors of this warp's segment
    const int mine = (r1 - r0 - group + groups - 1) / groups;  // rows of this warp: r0 + group, + groups, ...
    const unsigned int slot_bytes = (unsigned int)A.segv * 16u, bytes = (unsigned int)nv * 16u;
    unsigned char* ring = gs_raw + (size_t)warp * A.slots * slot_bytes;
    const unsigned int ring_s = pipe_smem_addr(ring), bar0 = pipe_smem_addr(&bars[warp][0]);
    float* part = reinterpret_cast<float*>(gs_raw + (size_t)kGvWarps * A.slots * slot_bytes);  // [rows of the CTA][nseg]
    const unsigned char* src = reinterpret_cast<const unsigned char*>(A.w) + ((size_t)(r0 + group) * A.ldw + (size_t)seg * A.segv * 8) * 2;
    const size_t src_step = (size_t)groups * A.ldw * 2;
    if (lane == 0) {
        for (int i = 0; i < A.slots; ++i) mbar_init(bar0 + 8 * i, 1);
        mbar_init_fence();
        for (int i = 0; i < min(A.slots, mine); ++i) {
            pipe_expect_tx(bar0 + 8 * i, bytes);
            pipe_bulk_copy(ring_s + i * slot_bytes, src + i * src_step, bytes, bar0 + 8 * i);
        }
    }
    __syncwarp();

    // ---- the activation of this warp's segment, in registers ----
    float a[VPL][8];
    const int c_seg = seg * A.segv * 8;
    if constexpr (PRO == kGvNorm) {
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
            const int v = lane + 32 * i;
            if (v < nv) gs_load8(A.norm_w, c_seg + v * 8, A.k, A.vec_x, a[i]);
        }
    }
    llvq_dependent_enter();
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < VPL; ++i) {
        const int v = lane + 32 * i, c = c_seg + v * 8;
        if (v >= nv) continue;
        if constexpr (PRO == kGvPlain) {
            gs_load8(A.x, c, A.k, A.vec_x, a[i]);
        } else if constexpr (PRO == kGvEmbed) {
            long long t = *A.token;
            if (t < 0 || t >= A.table_rows) t = 0;
            const bf16* row = reinterpret_cast<const bf16*>(A.table) + (size_t)t * A.ld_table;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                a[i][j] = c + j < A.k ? A.scale * to_f32(row[c + j]) : 0.0f;
                if (blockIdx.x == 0 && group == 0 && A.a_out && c + j < A.k) A.a_out[c + j] = a[i][j];
            }
        } else {
            float t[8], d[8];
            gs_load8(A.x, c, A.k, A.vec_x, t);
#pragma unroll
            for (int j = 0; j < 8; ++j) d[j] = 0.0f;
            if (A.delta) gs_load8(A.delta, c, A.k, A.vec_x, d);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                t[j] = fmaf(A.alpha, t[j], d[j]);
                ss = fmaf(t[j], t[j], ss);
                a[i][j] *= t[j];
            }
        }
    }
    if constexpr (PRO == kGvNorm) {  // the first row group's warps hold every segment once
        ss = warp_sum_f(ss);
        if (lane == 0) red[warp] = ss;
    }

    // ---- the rows, two at a time ----
    bool ok = true;
    int slot = 0;
    unsigned int parity = 0;
    for (int i = 0; i < mine; i += 2) {
        const bool two = i + 1 < mine;
        const int slot1 = two ? (slot + 1 == A.slots ? 0 : slot + 1) : slot;
        const unsigned int parity1 = parity ^ (two && slot1 == 0 ? 1u : 0u);
        ok = pipe_mbar_wait(bar0 + 8 * slot, parity) && (!two || pipe_mbar_wait(bar0 + 8 * slot1, parity1));
        if (!ok) break;
        const uint4* w0 = reinterpret_cast<const uint4*>(ring + (size_t)slot * slot_bytes);
        const uint4* w1 = reinterpret_cast<const uint4*>(ring + (size_t)slot1 * slot_bytes);
        float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int k = 0; k < VPL; ++k) {
            const int v = lane + 32 * k;
            if (v < nv) {
                float f[8], g[8];
                Vec16<bf16>::widen(w0[v], f);
                Vec16<bf16>::widen(w1[v], g);
#pragma unroll
                for (int j = 0; j < 8; j += 2) {
                    acc[0] = fmaf(f[j], a[k][j], acc[0]);
                    acc[2] = fmaf(g[j], a[k][j], acc[2]);
                    acc[1] = fmaf(f[j + 1], a[k][j + 1], acc[1]);
                    acc[3] = fmaf(g[j + 1], a[k][j + 1], acc[3]);
                }
            }
        }
        __syncwarp();  // both slots are read: they take the rows `slots` further on
        if (lane == 0) {
            if (i + A.slots < mine) {
                pipe_expect_tx(bar0 + 8 * slot, bytes);
                pipe_bulk_copy(ring_s + slot * slot_bytes, src + (size_t)(i + A.slots) * src_step, bytes, bar0 + 8 * slot);
            }
            if (two && i + 1 + A.slots < mine) {
                pipe_expect_tx(bar0 + 8 * slot1, bytes);
                pipe_bulk_copy(ring_s + slot1 * slot_bytes, src + (size_t)(i + 1 + A.slots) * src_step, bytes, bar0 + 8 * slot1);
            }
        }
        // both sums in five shuffles: the half-warps take a row each
        const float s0 = acc[0] + acc[1], s1 = acc[2] + acc[3];
        float s = (lane < 16 ? s0 : s1) + __shfl_xor_sync(0xffffffffu, lane < 16 ? s1 : s0, 16);
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if ((lane & 15) == 0 && (lane == 0 || two)) part[(group + (i + (lane >> 4)) * groups) * A.nseg + seg] = s;
        slot += 2;
        if (slot >= A.slots) {
            slot -= A.slots;
            parity ^= 1u;
        }
    }
    if (!ok) {  // give the copies in flight one more bounded chance to land before the CTA's memory is given up
        for (int i = 0; i < A.slots; ++i) pipe_mbar_wait(bar0 + 8 * i, parity);
        if (lane == 0) atomicOr(A.err, 1u);
    }
    __syncthreads();
    float factor = 1.0f;
    if constexpr (PRO == kGvNorm) {
        float tot = 0.0f;
        for (int s = 0; s < A.nseg; ++s) tot += red[s];
        factor = 1.0f / sqrtf(tot / (float)A.k + A.eps);
        if (blockIdx.x == 0 && group == 0 && A.a_out) {
#pragma unroll
            for (int i = 0; i < VPL; ++i) {
                const int v = lane + 32 * i, c = c_seg + v * 8;
                if (v >= nv) continue;
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (c + j < A.k) A.a_out[c + j] = a[i][j] * factor;
            }
        }
    }
    gemv_finish<HEAD>(A, part, A.nseg, factor, r0, r1, best_s);
}

}  // namespace llvq
