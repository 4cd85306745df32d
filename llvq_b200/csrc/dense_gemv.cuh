// y = W a (+ bias) for one token over a dense row-major matrix (bf16 or f32), the activation formed in the
// kernel's own staging, as the archive-code GEMV does:
//
//   prologue  plain   a = x
//             embed   a = scale * table[token]            (also written out: the residual stream starts here)
//             norm    t = alpha * x + delta; a = t / sqrt(mean(t^2) + eps) * w   (optionally written out; with a table,
//                     t is the token's row of it and may be written out: the residual stream starts here)
//   epilogue  y = W a + bias (+ residual), f32; or, with the rows of W in pairs (gate, up), the clamped gated unit of
//             each pair;
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
//
// A launch may serve more than one matrix:
//
//   second rows    rows of another matrix over the same t with a norm weight, a result and an epilogue of their own (a
//                  layer whose two sublayers read the same stream); CTAs are dealt to the two in proportion.
//   routed         the second rows, or further columns, come from matrices of a stack that the token's row of an integer
//                  table names: rows [matrix j | row], or y = W a + sum_j W_j a_j with a = [a | a_0 | a_1 | ...].
//                  The token is read ahead of the dependency wait: a step writes it at least one ordinary launch before
//                  its first projection.
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
    float glu_scale;      // times the gated unit
    const float* residual; // [n_out] or null: added to y (may be y)
    float* t_out;         // norm: t is also written here by CTA 0 (or null)
    // second rows (norm): [rows2, ldw], or the stack's [matrices, rows_m, ldw] with rows2 = top * rows_m
    const void* w2;
    const float* norm_w2;
    float* y2;
    int rows2, glu2;
    int cta2;             // first CTA of the second rows (gridDim.x: there are none)
    // routed columns (plain): the stack [matrices, n_out, ld_r], activation of matrix j at ldw + j * ld_r
    const void* w_r;
    int k_r, ld_r;
    // the token's matrices: table row [top]; null: nothing is routed
    const int* route;
    int route_rows, top, matrices, rows_m;
    // stream kernel: column segments (1, 2, 4 or 8), vectors of a segment, ring slots of a warp
    int nseg, segv, slots;
    int seg_r;            // routed columns: segments of one matrix; those of W come first
    int vec_x;            // x, delta and norm_w may be read 16 bytes at a time
    unsigned int* err;    // bit 0: a copy did not land in time
};

// The rows of one CTA and what becomes of them. Pairs stay together.
struct GemvRows {
    const void* w;
    const float* norm_w;
    float* y;
    int r0, r1, glu;
    bool second;
};
__device__ __forceinline__ GemvRows gemv_rows(const DenseGemvArgs& A) {
    GemvRows R;
    R.second = (int)blockIdx.x >= A.cta2;
    R.w = R.second ? A.w2 : A.w;
    R.norm_w = R.second ? A.norm_w2 : A.norm_w;
    R.y = R.second ? A.y2 : A.y;
    R.glu = R.second ? A.glu2 : A.glu;
    const int n = R.second ? A.rows2 : A.n_out, unit = R.glu ? 2 : 1;
    const int cta = R.second ? (int)blockIdx.x - A.cta2 : (int)blockIdx.x, ctas = R.second ? (int)gridDim.x - A.cta2 : A.cta2;
    R.r0 = unit * (int)((long long)(n / unit) * cta / ctas);
    R.r1 = unit * (int)((long long)(n / unit) * (cta + 1) / ctas);
    return R;
}

// Matrix j of the token. A token outside the table reads row 0, a matrix outside the stack is its nearest: no foreign memory.
constexpr int kGvRouteKept = 16;  // matrices of the token a CTA keeps the numbers of
__device__ __forceinline__ int gemv_route(const DenseGemvArgs& A, int j) {
    long long t = *A.token;
    if (t < 0 || t >= A.route_rows) t = 0;
    return min(max(A.route[t * A.top + j], 0), A.matrices - 1);
}
// Fills `kept`; a barrier for the whole CTA where anything is routed.
__device__ __forceinline__ void gemv_keep_route(const DenseGemvArgs& A, int* kept) {
    if (!A.route) return;
    if (A.table) llvq_dependent_enter();  // a step's first launch: the token is not older than the launch before
    if ((int)threadIdx.x < min(A.top, kGvRouteKept)) kept[threadIdx.x] = gemv_route(A, threadIdx.x);
    __syncthreads();
}
__device__ __forceinline__ int gemv_routed(const DenseGemvArgs& A, const int* kept, int j) { return j < kGvRouteKept ? kept[j] : gemv_route(A, j); }
// Row r of a CTA's rows in its matrix or stack.
__device__ __forceinline__ size_t gemv_src_row(const DenseGemvArgs& A, const GemvRows& R, const int* kept, int r) {
    if (!R.second || !A.route) return (size_t)r;
    return (size_t)gemv_routed(A, kept, r / A.rows_m) * A.rows_m + r % A.rows_m;
}

// y of the rows of a CTA from the partial sums of their segments, times `factor`.
template <bool HEAD>
__device__ __forceinline__ void gemv_finish(const DenseGemvArgs& A, const GemvRows& R, const float* part, int segments, float factor, HeadBest* best_s) {
    const int r0 = R.r0, r1 = R.r1;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    auto row_sum = [&](int r) {
        float s = 0.0f;
        for (int k = 0; k < segments; ++k) s += part[(r - r0) * segments + k];
        s *= factor;
        return A.bias && !R.second ? s + A.bias[r] : s;
    };
    if constexpr (!HEAD) {
        if (R.glu) {
            for (int i = r0 / 2 + tid; i < r1 / 2; i += kGvThreads)
                R.y[i] = A.glu_scale * clamped_glu(row_sum(2 * i), row_sum(2 * i + 1), A.limit, A.gain, A.shift);
        } else {
            for (int r = r0 + tid; r < r1; r += kGvThreads) R.y[r] = row_sum(r) + (A.residual && !R.second ? A.residual[r] : 0.0f);
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
    __shared__ int kept[kGvRouteKept];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const GemvRows R = gemv_rows(A);
    const int r0 = R.r0, r1 = R.r1;
    const int groups = kGvWarps / A.kslices, group = warp / A.kslices, slice = warp % A.kslices;
    const int vecs_w = A.ldw / VN, vecs_r = A.w_r ? A.ld_r / VN : 0, vecs = vecs_w + A.top * vecs_r, v0 = slice * 32 + lane, vstep = 32 * A.kslices;
    float* a_s = gv_smem;
    float* part = gv_smem + vecs * VN;  // [rows of the CTA][kslices]
    const uint4* W = reinterpret_cast<const uint4*>(R.w);
    gemv_keep_route(A, kept);
    auto load = [&](int r, int v) {
        if (v < vecs_w) return __ldg(W + gemv_src_row(A, R, kept, r) * vecs_w + v);
        const int j = (v - vecs_w) / vecs_r;
        return __ldg(reinterpret_cast<const uint4*>(A.w_r) + ((size_t)gemv_routed(A, kept, j) * A.n_out + r) * vecs_r + (v - vecs_w - j * vecs_r));
    };

    int row = r0 + group * kGvRows;
    uint4 w[kGvRows];
    const bool first = row < r1 && v0 < vecs;
    if (first) {
#pragma unroll
        for (int i = 0; i < kGvRows; ++i) w[i] = load(min(row + i, r1 - 1), v0);
    }
    llvq_dependent_enter();

    if constexpr (PRO == kGvPlain) {
        for (int i = tid; i < vecs * VN; i += kGvThreads) {
            const bool in = i < A.ldw ? i < A.k : (i - A.ldw) % A.ld_r < A.k_r;
            a_s[i] = in ? A.x[i] : 0.0f;
        }
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
        const T* src = nullptr;
        if (A.table) {
            long long t = *A.token;
            if (t < 0 || t >= A.table_rows) t = 0;
            src = reinterpret_cast<const T*>(A.table) + (size_t)t * A.ld_table;
        }
        for (int i = tid; i < A.ldw; i += kGvThreads) {
            float t = 0.0f;
            if (i < A.k) {
                t = src ? A.scale * to_f32(src[i]) : A.alpha * A.x[i];
                if (A.delta) t += A.delta[i];
                if (blockIdx.x == 0 && A.t_out) A.t_out[i] = t;
            }
            a_s[i] = t;
            ss = fmaf(t, t, ss);
        }
        const float r = 1.0f / sqrtf(block_sum_f(ss, red) / (float)A.k + A.eps);
        for (int i = tid; i < A.k; i += kGvThreads) {  // the element this thread wrote above
            const float v = a_s[i] * r * R.norm_w[i];
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
                for (int i = 0; i < kGvRows; ++i) w[i] = load(min(row + i, r1 - 1), v);
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
    gemv_finish<HEAD>(A, R, part, A.kslices, 1.0f, best_s);
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
    __shared__ int kept[kGvRouteKept];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const GemvRows R = gemv_rows(A);
    const int r0 = R.r0, r1 = R.r1;
    const int seg = warp % A.nseg, group = warp / A.nseg, groups = kGvWarps / A.nseg;
    const int seg_w = A.nseg - A.seg_r * A.top;                 // segments of W itself; then those of the routed matrices
    const int part_j = seg < seg_w ? -1 : (seg - seg_w) / A.seg_r, part_s = seg < seg_w ? seg : (seg - seg_w) % A.seg_r;
    const int ld = part_j < 0 ? A.ldw : A.ld_r, c_part = part_j < 0 ? 0 : A.ldw + part_j * A.ld_r;
    const int k_end = c_part + (part_j < 0 ? A.k : A.k_r);      // activation columns of the part end here
    const int nv = min(A.segv, ld / 8 - part_s * A.segv);       // vectors of this warp's segment
    // rows of this warp: r0 + group, + groups, ... (none for the warps left over)
    const int mine = group < groups ? (r1 - r0 - group + groups - 1) / groups : 0;
    gemv_keep_route(A, kept);
    const unsigned int slot_bytes = (unsigned int)A.segv * 16u, bytes = (unsigned int)nv * 16u;
    unsigned char* ring = gs_raw + (size_t)warp * A.slots * slot_bytes;
    const unsigned int ring_s = pipe_smem_addr(ring), bar0 = pipe_smem_addr(&bars[warp][0]);
    float* part = reinterpret_cast<float*>(gs_raw + (size_t)kGvWarps * A.slots * slot_bytes);  // [rows of the CTA][nseg]
    const unsigned char* src0 = part_j < 0 ? reinterpret_cast<const unsigned char*>(R.w)
                                           : reinterpret_cast<const unsigned char*>(A.w_r) + (size_t)gemv_routed(A, kept, part_j) * A.n_out * ld * 2;
    src0 += (size_t)part_s * A.segv * 16;
    auto src = [&](int i) { return src0 + gemv_src_row(A, R, kept, r0 + group + i * groups) * ld * 2; };  // of this warp's row i
    if (lane == 0) {
        for (int i = 0; i < A.slots; ++i) mbar_init(bar0 + 8 * i, 1);
        mbar_init_fence();
        for (int i = 0; i < min(A.slots, mine); ++i) {
            pipe_expect_tx(bar0 + 8 * i, bytes);
            pipe_bulk_copy(ring_s + i * slot_bytes, src(i), bytes, bar0 + 8 * i);
        }
    }
    __syncwarp();

    // ---- the activation of this warp's segment, in registers ----
    float a[VPL][8];
    const int c_seg = c_part + part_s * A.segv * 8;
    if constexpr (PRO == kGvNorm) {
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
            const int v = lane + 32 * i;
            if (v < nv) gs_load8(R.norm_w, c_seg + v * 8, A.k, A.vec_x, a[i]);
        }
    }
    llvq_dependent_enter();
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < VPL; ++i) {
        const int v = lane + 32 * i, c = c_seg + v * 8;
        if (v >= nv) continue;
        if constexpr (PRO == kGvPlain) {
            gs_load8(A.x, c, k_end, A.vec_x, a[i]);
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
            float alpha = A.alpha;
            if (A.table) {
                long long id = *A.token;
                if (id < 0 || id >= A.table_rows) id = 0;
                Vec16<bf16>::widen(*reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(A.table) + (size_t)id * A.ld_table + c), t);
                alpha = A.scale;
            } else {
                gs_load8(A.x, c, A.k, A.vec_x, t);
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) d[j] = 0.0f;
            if (A.delta) gs_load8(A.delta, c, A.k, A.vec_x, d);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                t[j] = fmaf(alpha, t[j], d[j]);
                if (A.t_out && blockIdx.x == 0 && group == 0 && c + j < A.k) A.t_out[c + j] = t[j];
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
                pipe_bulk_copy(ring_s + slot * slot_bytes, src(i + A.slots), bytes, bar0 + 8 * slot);
            }
            if (two && i + 1 + A.slots < mine) {
                pipe_expect_tx(bar0 + 8 * slot1, bytes);
                pipe_bulk_copy(ring_s + slot1 * slot_bytes, src(i + 1 + A.slots), bytes, bar0 + 8 * slot1);
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
    gemv_finish<HEAD>(A, R, part, A.nseg, factor, best_s);
}

}  // namespace llvq
