// Latent attention of a prompt portion on the 5th-generation tensor cores (tcgen05 + TMEM), sm_100a; bf16 operands,
// f32 scores, softmax and sums. The same operator as latent_prefill.cuh with the expanded values transposed
// (vt [heads * vdim, ld_vt], positions along the row: both products then take K-major operands).
//
// A CTA serves 256 queries of one head as two tiles of 128, which share every key and value tile of 64 positions and
// take turns on the tensor cores: while one tile's softmax runs, the other's products do. Warps:
//
//   0-3, 4-7   softmax of query tile 0 / 1, thread = query row = TMEM lane: read the scores (tcgen05.ld), mask only
//              where the tile crosses an edge of the row's window, exponentials in base 2, weights as bf16 into the
//              tile's operand buffer. The sums in TMEM are rescaled only when a row's maximum has grown by more than
//              2^8 since the last time (the final division takes the difference out exactly).
//   8          one thread issues the products: S_w = Q_w K^T (N = 64) ahead of O_w += P_w V (N = vdim).
//   9-10       key tiles [unrotated of the head | rotated, shared] by cp.async, double buffered.
//   11         value tiles likewise.
//
// Tiles are 128-byte-swizzled K-major panels of 64 columns. Scores and sums live in TMEM: columns [0, 128) hold S_0 and
// S_1, then O_0 and O_1. Every wait is bounded; on a time-out a flag is raised, all roles leave their loops, TMEM is freed.
#pragma once
#include <cstddef>

#include "latent_prefill.cuh"
#include "mbarrier.cuh"

namespace llvq {

constexpr int kTcM = 128, kTcN = 64;
constexpr int kTcThreads = 12 * 32;
constexpr int kTcKeyLoaders = 64, kTcValueLoaders = 32;  // threads

struct LatentPrefillTcArgs {
    LatentPrefillArgs p;      // kv = the keys [n_k, ld_kv]
    const void* vt;           // [heads / rep * vdim, ld_vt], zero from n_k to the next multiple of 8
    int ld_vt;
    unsigned int* err;
};

__host__ __device__ inline int tc_panels(int qk) { return (qk + 63) / 64; }
__host__ __device__ inline int tc_v_rows(int vdim) { return (vdim + 15) / 16 * 16; }
inline size_t latent_prefill_tc_smem(int qk, int vdim) {
    const size_t q = 2 * (size_t)kTcM * 128 * tc_panels(qk), k = 2 * (size_t)kTcN * 128 * tc_panels(qk), v = 2 * (size_t)tc_v_rows(vdim) * 128;
    return q + k + v + 2 * (size_t)kTcM * 128 + 1024;
}

// Shared-memory matrix descriptor: K-major operand, 128-byte swizzle, 8-row groups 1024 bytes apart.
__device__ __forceinline__ unsigned long long umma_desc_k128(unsigned int addr) {
    unsigned long long d = ((unsigned long long)addr & 0x3FFFFull) >> 4;
    d |= 1ull << 16;
    d |= (1024ull >> 4) << 32;
    d |= 1ull << 46;  // descriptor version of sm_100
    d |= 2ull << 61;  // SWIZZLE_128B
    return d;
}
// Byte offset of 16-byte piece c (0..7) of row r in a panel of 128-byte rows.
__device__ __forceinline__ unsigned int tc_swz(int r, int c) { return (unsigned int)(r * 128 + ((c ^ (r & 7)) << 4)); }

__device__ __forceinline__ void tc_mma(unsigned int d, unsigned long long a, unsigned long long b, unsigned int idesc, bool accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %6, %7, %8}, p;\n\t}" ::"r"(d),
        "l"(a), "l"(b), "r"(idesc), "r"((unsigned int)accumulate), "r"(0u), "r"(0u), "r"(0u), "r"(0u)
        : "memory");
}
__device__ __forceinline__ void tc_commit(unsigned int bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void tc_arrive(unsigned int bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
// TMEM -> registers; the wait is part of the statement, so that no use of a register moves ahead of it.
__device__ __forceinline__ void tc_ld32(unsigned int (&r)[32], unsigned int addr) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, %17, %18, %19, "
        "%20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];\n\ttcgen05.wait::ld.sync.aligned;"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
          "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]),
          "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]),
          "=r"(r[31])
        : "r"(addr)
        : "memory");
}
__device__ __forceinline__ void tc_ld16(unsigned int (&r)[16], unsigned int addr) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];\n\t"
        "tcgen05.wait::ld.sync.aligned;"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
          "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(addr)
        : "memory");
}
__device__ __forceinline__ void tc_st16(unsigned int addr, const unsigned int (&r)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(addr),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]),
        "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
        : "memory");
}
__device__ __forceinline__ float tc_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

struct TcBarriers {
    unsigned long long k_full[2], k_free[2], v_full[2], v_free[2];
    unsigned long long s_ready[2], p_ready[2], o_ready[2];  // per query tile
    unsigned long long drained;
    unsigned int tmem;
};

__global__ void __launch_bounds__(kTcThreads, 1)
latent_prefill_tc_kernel(LatentPrefillTcArgs T) {
    extern __shared__ unsigned char tc_raw[];
    __shared__ TcBarriers B;
    const LatentPrefillArgs& A = T.p;
    const int qk = A.dim + A.rot_dim, panels = tc_panels(qk), ksteps = (qk + 15) / 16, vrows = tc_v_rows(A.vdim);
    const unsigned int smem0 = (pipe_smem_addr(tc_raw) + 1023u) & ~1023u;
    unsigned char* base0 = tc_raw + (smem0 - pipe_smem_addr(tc_raw));
    const unsigned int q_bytes = (unsigned int)(kTcM * 128 * panels), k_bytes = (unsigned int)(kTcN * 128 * panels), v_bytes = (unsigned int)(vrows * 128);
    const unsigned int off_k = 2 * q_bytes, off_v = off_k + 2 * k_bytes, off_p = off_v + 2 * v_bytes;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, hk = h / A.rep;
    const int q_lo = ((int)gridDim.x - 1 - (int)blockIdx.x) * 2 * kTcM;  // rows with the most keys first
    const int off = (int)(A.pos0 - A.key0);
    const bool two = q_lo + kTcM < A.n_q;
    // keys by their place in the operands: query i sees places i + off - window + 1 .. i + off
    const int last_q = min(A.n_q, q_lo + 2 * kTcM) - 1;
    const int k_end = last_q + off + 1;
    const int k_begin = max(0, q_lo + off - A.window + 1) & ~7;
    const int tiles = (k_end - k_begin + kTcN - 1) / kTcN;
    // tiles a query tile takes part in: [t_lo(w), t_hi(w))
    const int hi0 = (min(A.n_q, q_lo + kTcM) - 1 + off - k_begin) / kTcN + 1;
    const int lo1 = two ? max(0, q_lo + kTcM + off - A.window + 1 - k_begin) / kTcN : tiles;

    const unsigned int bar = pipe_smem_addr(&B);
    const unsigned int kfull = bar + offsetof(TcBarriers, k_full), kfree = bar + offsetof(TcBarriers, k_free), vfull = bar + offsetof(TcBarriers, v_full),
                       vfree = bar + offsetof(TcBarriers, v_free), sready = bar + offsetof(TcBarriers, s_ready), pready = bar + offsetof(TcBarriers, p_ready),
                       oready = bar + offsetof(TcBarriers, o_ready);
    if (tid == 0) {
        for (int i = 0; i < 2; ++i) {
            mbar_init(kfull + 8 * i, kTcKeyLoaders);
            mbar_init(vfull + 8 * i, kTcValueLoaders);
            mbar_init(kfree + 8 * i, 1);
            mbar_init(vfree + 8 * i, 1);
            mbar_init(sready + 8 * i, 1);
            mbar_init(oready + 8 * i, 1);
            mbar_init(pready + 8 * i, kTcM);
        }
        mbar_init(bar + offsetof(TcBarriers, drained), 1);
        mbar_init_fence();
    }
    if (warp == 8) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(pipe_smem_addr(&B.tmem)), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    llvq_dependent_enter();

    // ---- query tiles, rotated: rows beyond the portion and columns beyond qk are zero. Eight lanes bring the 128 bytes of
    // a row's panel, a warp four rows at a time ----
    {
        const bf16* Q = reinterpret_cast<const bf16*>(A.q) + (size_t)h * qk;
        const size_t qrow = (size_t)A.heads * qk;
        const int cn = A.dim / 8, half = A.rt.dims / 2, rows = two ? 2 * kTcM : kTcM;
        for (int p = 0; p < panels; ++p) {
            const int c = p * 8 + (lane & 7);
            if (c >= cn && 8 * c < qk) continue;  // the rotated part comes below
#pragma unroll 4
            for (int r = warp * 4 + (lane >> 3); r < rows; r += kTcThreads / 8) {
                const bool in = c < cn && q_lo + r < A.n_q;
                copy16_async(reinterpret_cast<bf16*>(base0 + (r >= kTcM ? q_bytes : 0) + p * (kTcM * 128) + tc_swz(r & (kTcM - 1), lane & 7)),
                             in ? Q + (size_t)(q_lo + r) * qrow + 8 * c : Q, in);
            }
        }
        auto at = [&](int r, int col) {
            return base0 + (r >= kTcM ? q_bytes : 0) + (col >> 6) * (kTcM * 128) + tc_swz(r & (kTcM - 1), (col & 63) >> 3) + 2 * (col & 7);
        };
        if (half % 8 == 0) {  // whole vectors of pairs
            const int hp = half / 8, per = hp + (A.rot_dim - 2 * half) / 8;
#pragma unroll 2
            for (int i = tid; i < rows * per; i += kTcThreads) {
                const int r = i / per, c = i - r * per;
                const bool in = q_lo + r < A.n_q;
                const bf16* src = Q + (size_t)(q_lo + r) * qrow + A.dim;
                const uint4 zero = make_uint4(0, 0, 0, 0);
                if (c >= hp) {
                    *reinterpret_cast<uint4*>(at(r, A.dim + half + 8 * c)) = in ? *reinterpret_cast<const uint4*>(src + half + 8 * c) : zero;
                    continue;
                }
                uint4 a = zero, b = zero;
                if (in) {
                    float u[8], v[8], x[8], y[8];
                    Vec16<bf16>::widen(*reinterpret_cast<const uint4*>(src + 8 * c), u);
                    Vec16<bf16>::widen(*reinterpret_cast<const uint4*>(src + half + 8 * c), v);
                    const size_t p = (size_t)(A.pos0 + q_lo + r) * half + 8 * c;
#pragma unroll
                    for (int j = 0; j < 8; ++j) {
                        const float cs = A.rt.cos_t[p + j], sn = A.rt.sin_t[p + j];
                        x[j] = u[j] * cs - v[j] * sn;
                        y[j] = v[j] * cs + u[j] * sn;
                    }
                    a = make_uint4(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]), pack_bf16(x[4], x[5]), pack_bf16(x[6], x[7]));
                    b = make_uint4(pack_bf16(y[0], y[1]), pack_bf16(y[2], y[3]), pack_bf16(y[4], y[5]), pack_bf16(y[6], y[7]));
                }
                *reinterpret_cast<uint4*>(at(r, A.dim + 8 * c)) = a;
                *reinterpret_cast<uint4*>(at(r, A.dim + half + 8 * c)) = b;
            }
        } else {
            const int rest = A.rot_dim - half;  // pairs, then what passes
            for (int i = tid; i < rows * rest; i += kTcThreads) {
                const int r = i / rest, c = i - r * rest;
                const bool in = q_lo + r < A.n_q;
                const bf16* src = Q + (size_t)(q_lo + r) * qrow + A.dim;
                if (c < half) {
                    float x = 0.0f, y = 0.0f;
                    if (in) {
                        const size_t p = (size_t)(A.pos0 + q_lo + r) * half + c;
                        const float cs = A.rt.cos_t[p], sn = A.rt.sin_t[p], u = to_f32(src[c]), v = to_f32(src[c + half]);
                        x = u * cs - v * sn;
                        y = v * cs + u * sn;
                    }
                    *reinterpret_cast<bf16*>(at(r, A.dim + c)) = from_f32<bf16>(x);
                    *reinterpret_cast<bf16*>(at(r, A.dim + c + half)) = from_f32<bf16>(y);
                } else {
                    *reinterpret_cast<bf16*>(at(r, A.dim + c + half)) = in ? src[c + half] : __float2bfloat16_rn(0.0f);
                }
            }
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const unsigned int tmem = B.tmem;
    const unsigned int o_col = 2 * kTcN;  // O_w at o_col + w * vrows
    bool ok = true;

    if (warp < 8) {
        // ---- softmax ----
        const int w = warp >> 2, row = tid & (kTcM - 1);
        const int t_lo = w ? lo1 : 0, t_hi = w ? (two ? tiles : lo1) : hi0;
        const unsigned int lanes = (unsigned int)((warp & 3) * 32) << 16;
        const unsigned int s_addr = tmem + lanes + w * kTcN, o_addr = tmem + lanes + o_col + w * vrows;
        unsigned char* p_row = base0 + off_p + w * (kTcM * 128);
        const int place = q_lo + w * kTcM + row + off;  // of this row's own key
        const int first_w = q_lo + w * kTcM + (warp & 3) * 32 + off;  // of the warp's rows: first_w .. first_w + 31
        const float s2 = A.scale * kLog2e;
        float m = -INFINITY, l = 0.0f;  // base-2 maximum the weights are taken against; their sum
        int n = 0;                       // tiles done
        for (int t = t_lo; t < t_hi; ++t, ++n) {
            ok = __all_sync(0xffffffffu, pipe_mbar_wait(sready + 8 * w, n & 1));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            unsigned int s[2][32];
            tc_ld32(s[0], s_addr);
            tc_ld32(s[1], s_addr + 32);
            const int base = k_begin + t * kTcN;
            if (base + kTcN - 1 > first_w || base < first_w + 31 - A.window + 1) {  // warp-uniform: the tile crosses an edge
                const int c_hi = place - base, c_lo = place - A.window + 1 - base;
#pragma unroll
                for (int j = 0; j < 64; ++j)
                    if (j > c_hi || j < c_lo) s[j >> 5][j & 31] = 0xff800000u;  // -inf
            }
            float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
            for (int j = 0; j < 32; ++j) {
                mx0 = fmaxf(mx0, __uint_as_float(s[0][j]));
                mx1 = fmaxf(mx1, __uint_as_float(s[1][j]));
            }
            const float top = fmaxf(mx0, mx1) * s2;  // scale > 0
            // the weights of the tile before are read once its product is done; the sums may then be rescaled as well
            if (n > 0) {
                ok = __all_sync(0xffffffffu, pipe_mbar_wait(oready + 8 * w, (n - 1) & 1));
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            }
            if (__any_sync(0xffffffffu, top > m + 8.0f)) {
                const float mn = fmaxf(m, top), f = m == -INFINITY ? 0.0f : tc_ex2(m - mn);
                m = mn;
                l *= f;
                if (n > 0) {
                    for (int c = 0; c < vrows; c += 16) {
                        unsigned int r[16];
                        tc_ld16(r, o_addr + c);
#pragma unroll
                        for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * f);
                        tc_st16(o_addr + c, r);
                    }
                    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
                }
            }
            const float mb = m == -INFINITY ? 0.0f : m;  // a row that has seen no key yet
            float l0 = 0.0f, l1 = 0.0f;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                unsigned int v[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int k = 8 * c + 2 * j;
                    const float e0 = tc_ex2(fmaf(__uint_as_float(s[k >> 5][k & 31]), s2, -mb));
                    const float e1 = tc_ex2(fmaf(__uint_as_float(s[k >> 5][(k & 31) + 1]), s2, -mb));
                    l0 += e0;
                    l1 += e1;
                    v[j] = pack_bf16(e0, e1);
                }
                *reinterpret_cast<uint4*>(p_row + tc_swz(row, c)) = make_uint4(v[0], v[1], v[2], v[3]);
            }
            l += l0 + l1;
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            tc_arrive(pready + 8 * w);
        }
        if (ok && n > 0) {
            ok = __all_sync(0xffffffffu, pipe_mbar_wait(oready + 8 * w, (n - 1) & 1));
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int i = q_lo + w * kTcM + row;
            float f = 1.0f, den = l;
            if (A.sink) {
                const float sk2 = A.sink[h] * kLog2e, mt = fmaxf(m, sk2);
                f = exp2f(m - mt);
                den = l * f + exp2f(sk2 - mt);
            }
            f /= den;
            bf16* dst = reinterpret_cast<bf16*>(A.out) + (size_t)i * A.heads * A.vdim + (size_t)h * A.vdim;
            for (int c = 0; ok && c < vrows; c += 16) {
                unsigned int r[16];
                __syncwarp();
                tc_ld16(r, o_addr + c);
#pragma unroll
                for (int k = 0; k < 16; k += 8) {
                    unsigned int v[4];
#pragma unroll
                    for (int j = 0; j < 4; ++j) v[j] = pack_bf16(__uint_as_float(r[k + 2 * j]) * f, __uint_as_float(r[k + 2 * j + 1]) * f);
                    if (i < A.n_q && c + k < A.vdim) *reinterpret_cast<uint4*>(dst + c + k) = make_uint4(v[0], v[1], v[2], v[3]);
                }
            }
        }
    } else if (warp == 8) {
        // ---- products ----
        if (lane == 0) {
            const unsigned int s_desc = (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned int)(kTcN >> 3) << 17) | ((unsigned int)(kTcM >> 4) << 24);
            const unsigned int o_desc = (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned int)(vrows >> 3) << 17) | ((unsigned int)(kTcM >> 4) << 24);
            auto active = [&](int w, int t) { return w ? (t >= lo1 && t < tiles) : (t < hi0); };
            auto scores = [&](int w, int t) {
                for (int k = 0; k < ksteps; ++k) {
                    const unsigned int p = (unsigned int)k >> 2;
                    tc_mma(tmem + w * kTcN, umma_desc_k128(smem0 + w * q_bytes + p * (kTcM * 128)) + 2ull * (k & 3),
                           umma_desc_k128(smem0 + off_k + (t & 1) * k_bytes + p * (kTcN * 128)) + 2ull * (k & 3), s_desc, k > 0);
                }
                tc_commit(sready + 8 * w);
            };
            int done[2] = {0, 0};  // tiles whose weights have been consumed, per query tile
            ok = pipe_mbar_wait(kfull, 0);
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (ok) {
                for (int w = 0; w < 2; ++w)
                    if (active(w, 0)) scores(w, 0);
                tc_commit(kfree);
            }
            for (int t = 0; ok && t < tiles; ++t) {
                const bool more = t + 1 < tiles;
                bool have_k = false, have_v = false;
                for (int w = 0; ok && w < 2; ++w) {
                    const bool now = active(w, t), next = more && active(w, t + 1);
                    if (now) ok = pipe_mbar_wait(pready + 8 * w, done[w] & 1);
                    if (ok && next) {
                        if (!have_k) ok = pipe_mbar_wait(kfull + 8 * ((t + 1) & 1), ((t + 1) >> 1) & 1);
                        have_k = true;
                    }
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    if (ok && next) scores(w, t + 1);
                    if (ok && now) {
                        if (!have_v) ok = pipe_mbar_wait(vfull + 8 * (t & 1), (t >> 1) & 1);
                        have_v = true;
                        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                        if (!ok) break;
                        for (int k = 0; k < kTcN / 16; ++k)
                            tc_mma(tmem + o_col + w * vrows, umma_desc_k128(smem0 + off_p + w * (kTcM * 128)) + 2ull * k,
                                   umma_desc_k128(smem0 + off_v + (t & 1) * v_bytes) + 2ull * k, o_desc, done[w] > 0 || k > 0);
                        tc_commit(oready + 8 * w);
                        ++done[w];
                    }
                }
                if (ok && more) tc_commit(kfree + 8 * ((t + 1) & 1));
                if (ok) tc_commit(vfree + 8 * (t & 1));
            }
            // nothing of this CTA's products is in flight when its memory is given up, on a time-out either
            const unsigned int drained = bar + offsetof(TcBarriers, drained);
            tc_commit(drained);
            ok = pipe_mbar_wait(drained) && ok;
        }
    } else {
        // ---- key and value tiles ----
        const bf16* K = reinterpret_cast<const bf16*>(A.kv);
        const bf16* KR = reinterpret_cast<const bf16*>(A.kr);
        const bf16* VT = reinterpret_cast<const bf16*>(T.vt);
        const bool keys = warp < 11;
        const unsigned int full = keys ? kfull : vfull, free_ = keys ? kfree : vfree;
        const int cn = A.dim / 8, cq = qk / 8, sub = lane >> 3, c8 = lane & 7;  // a warp brings 128 bytes of four rows at a time
        for (int t = 0; t < tiles; ++t) {
            if (t >= 2) ok = pipe_mbar_wait(free_ + 8 * (t & 1), ((t >> 1) - 1) & 1);
            if (!ok) break;
            const int base = k_begin + t * kTcN;
            if (keys) {
                const int r0 = (warp - 9) * 32 + sub, n_in = k_end - base - r0;  // rows r0, r0 + 4, ...: row 4 i is there for 4 i < n_in
                for (int p = 0; p < panels; ++p) {
                    const int c = p * 8 + c8;
                    if (c >= 2 * ksteps) continue;
                    const bool own = c < cn, in_c = c < cq;
                    const size_t step = 4 * (size_t)(own ? A.ld_kv : A.ld_kr);
                    const bf16* src = own ? K + (size_t)(base + r0) * A.ld_kv + (size_t)hk * A.k_head + 8 * c : KR + (size_t)(base + r0) * A.ld_kr + 8 * (c - cn);
                    unsigned char* dst = base0 + off_k + (t & 1) * k_bytes + p * (kTcN * 128) + r0 * 128;
                    const int even = (c8 ^ (r0 & 7)) << 4, odd = (c8 ^ ((r0 + 4) & 7)) << 4;
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        const bool in = in_c && 4 * i < n_in;
                        copy16_async(reinterpret_cast<bf16*>(dst + i * 512 + (i & 1 ? odd : even)), in ? src + i * step : K, in);
                    }
                }
            } else {
                const int j = base + 8 * c8;
                const bool in_j = j < A.n_k;
                const size_t step = 4 * (size_t)T.ld_vt;
                const bf16* src = VT + ((size_t)hk * A.vdim + sub) * T.ld_vt + j;
                unsigned char* dst = base0 + off_v + (t & 1) * v_bytes + sub * 128;
                const int even = (c8 ^ sub) << 4, odd = (c8 ^ (sub + 4)) << 4;
#pragma unroll 4
                for (int i = 0; i < vrows / 4; ++i) {
                    const bool in = in_j && 4 * i + sub < A.vdim;
                    copy16_async(reinterpret_cast<bf16*>(dst + i * 512 + (i & 1 ? odd : even)), in ? src + i * step : VT, in);
                }
            }
            asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            tc_arrive(full + 8 * (t & 1));
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
    }
    if (!ok) atomicOr(T.err, 1u);
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 8) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
}

}  // namespace llvq
