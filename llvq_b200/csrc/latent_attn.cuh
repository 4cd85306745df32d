// Latent attention, the token step. A layer caches per position one row [latent c | rotated key part] that all
// heads share (T elements, row stride ld: whole 16-byte vectors, zero beyond kv_rank + rot_dim). The row of
// position p sits in slot p % slots of the layer's ring, so a windowed layer keeps only what its window (and a
// prompt portion) can still see. The token step never expands keys or values:
//
//   latent_query_kernel   per head: the unrotated query is carried into the latent space (q W_uk), the rotated
//                         part is turned to its position: one f32 row [ld] per head that meets the cache rows
//                         directly. One extra CTA norms the token's own latent, rotates its key part and
//                         stores the row into the ring.
//   latent_decode_mma_kernel  bf16: grid (groups of 16 heads, splits); every split of the visible positions in tiles
//                         of 64 rows staged once in shared memory, the heads are the rows of the tensor-core tiles:
//                         scores with warp = 8 positions, sums of latents with warp = 16-dimension pieces.
//   latent_decode_kernel  f32 (and latents too wide for the other): groups of 8 heads, tiles of 32 rows; warp = head
//                         and lane = position for the scores and the online softmax, thread = latent dimensions
//                         for the sums.
//   latent_value_kernel   per head: merges the splits, adds the sink to the denominator (a learned score with no
//                         key and no value), and expands the sum of latents by W_uv.
//
// Softmax runs in base 2 in f32; the position is read from device memory, so a captured graph replays.
#pragma once
#include "dense_elem.cuh"
#include "warp_mma.cuh"

namespace llvq {

constexpr float kLog2e = 1.4426950408889634f;

struct RotaryTable {
    const float* cos_t;  // [positions, dims / 2]
    const float* sin_t;
    int dims;            // rotated dimensions of the rotated part: i is paired with i + dims / 2, the rest pass
};

// Where position p of a cached layer lives.
struct LatentRing {
    void* rows;  // [slots, ld] of T
    int slots, ld;
};

// One token's cache row from its down projection y = [kv_rank latent | rot_dim rotated part]: the latent is RMS
// normed, the rest is turned to `pos`. A whole CTA calls it; `red` holds a float per warp.
template <typename T, typename Y>
__device__ __forceinline__ void store_latent_row(const Y* y, const float* norm_w, float eps, int kv_rank, int rot_dim,
                                                 RotaryTable rt, long long pos, LatentRing ring, float* red) {
    T* dst = reinterpret_cast<T*>(ring.rows) + (size_t)(pos % ring.slots) * ring.ld;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) {
        const float v = to_f32(y[i]);
        ss = fmaf(v, v, ss);
    }
    const float r = 1.0f / sqrtf(block_sum_f(ss, red) / (float)kv_rank + eps);
    for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) dst[i] = from_f32<T>(to_f32(y[i]) * r * norm_w[i]);
    const int half = rt.dims / 2;
    for (int i = threadIdx.x; i < rot_dim; i += blockDim.x) {
        if (i < half) {
            const float c = rt.cos_t[pos * half + i], s = rt.sin_t[pos * half + i];
            const float u = to_f32(y[kv_rank + i]), v = to_f32(y[kv_rank + half + i]);
            dst[kv_rank + i] = from_f32<T>(u * c - v * s);
            dst[kv_rank + half + i] = from_f32<T>(v * c + u * s);
        } else if (i >= rt.dims) {
            dst[kv_rank + i] = from_f32<T>(to_f32(y[kv_rank + i]));
        }
    }
}

struct LatentQueryArgs {
    const float* q;       // [heads, dim + rot_dim]
    const void* uk;       // [heads * dim, ldk] of T
    void* qlat;           // [heads, ring.ld] of Q: latent part, rotated part, zeros
    const float* y_kv;    // [kv_rank + rot_dim] of this token, or null (the layer reads another layer's ring)
    const float* kv_norm; // [kv_rank]
    const long long* pos;
    LatentRing ring;
    RotaryTable rt;
    int heads, dim, rot_dim, kv_rank, ldk;
    float eps;
};

// grid = (heads + (y_kv ? 1 : 0), column slices), 256 threads: 32 lanes of one 16-byte vector each, 8 groups over d.
// Q: f32, or bf16 where the tensor cores read it. The first rows of W_uk are on their way before the dependency wait.
template <typename T, typename Q>
__global__ void __launch_bounds__(256)
latent_query_kernel(LatentQueryArgs A) {
    constexpr int VN = Vec16<T>::N;
    __shared__ float red[8];
    __shared__ float sum_s[8][32][VN + 1];
    const int h = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int vecs = A.ldk / VN, v = blockIdx.y * 32 + lane;
    const uint4* W = reinterpret_cast<const uint4*>(A.uk) + (size_t)h * A.dim * vecs + v;
    constexpr int kAhead = 8;
    uint4 ahead[kAhead];
    if (h < A.heads && v < vecs) {
#pragma unroll
        for (int i = 0; i < kAhead; ++i) ahead[i] = __ldg(W + (size_t)min(warp + 8 * i, A.dim - 1) * vecs);
    }
    llvq_dependent_enter();
    const long long pos = *A.pos;
    if (h == A.heads) {
        if (blockIdx.y == 0) store_latent_row<T>(A.y_kv, A.kv_norm, A.eps, A.kv_rank, A.rot_dim, A.rt, pos, A.ring, red);
        return;
    }
    const float* q = A.q + (size_t)h * (A.dim + A.rot_dim);
    float acc[VN];
#pragma unroll
    for (int j = 0; j < VN; ++j) acc[j] = 0.0f;
    if (v < vecs) {
        auto add = [&](const uint4& w, float qd) {
            float f[VN];
            Vec16<T>::widen(w, f);
#pragma unroll
            for (int j = 0; j < VN; ++j) acc[j] = fmaf(qd, f[j], acc[j]);
        };
#pragma unroll
        for (int i = 0; i < kAhead; ++i)
            if (warp + 8 * i < A.dim) add(ahead[i], q[warp + 8 * i]);
#pragma unroll 4
        for (int d = warp + 8 * kAhead; d < A.dim; d += 8) add(__ldg(W + (size_t)d * vecs), q[d]);
    }
#pragma unroll
    for (int j = 0; j < VN; ++j) sum_s[warp][lane][j] = acc[j];
    __syncthreads();
    Q* out = reinterpret_cast<Q*>(A.qlat) + (size_t)h * A.ring.ld;
    for (int e = threadIdx.x; e < 32 * VN; e += 256) {
        const int r = blockIdx.y * 32 * VN + e;
        if (r >= A.kv_rank) break;
        float s = 0.0f;
#pragma unroll
        for (int k = 0; k < 8; ++k) s += sum_s[k][e / VN][e % VN];
        out[r] = from_f32<Q>(s);
    }
    if (blockIdx.y == 0) {
        const int half = A.rt.dims / 2;
        for (int i = threadIdx.x; i < A.rot_dim; i += 256) {
            if (i < half) {
                const float c = A.rt.cos_t[pos * half + i], s = A.rt.sin_t[pos * half + i];
                const float a = q[A.dim + i], b = q[A.dim + half + i];
                out[A.kv_rank + i] = from_f32<Q>(a * c - b * s);
                out[A.kv_rank + half + i] = from_f32<Q>(b * c + a * s);
            } else if (i >= A.rt.dims) {
                out[A.kv_rank + i] = from_f32<Q>(q[A.dim + i]);
            }
        }
        for (int i = A.kv_rank + A.rot_dim + threadIdx.x; i < A.ring.ld; i += 256) out[i] = from_f32<Q>(0.0f);
    }
}

constexpr int kLdHeads = 8;   // heads per CTA = warps
constexpr int kLdTile = 32;   // positions per tile = lanes

struct LatentDecodeArgs {
    const void* qlat;   // [heads, ring.ld] of f32 (bf16 for the tensor-core kernel)
    const long long* pos;
    float* part_ml;     // [heads, splits, 2]: base-2 maximum, sum
    float* part_o;      // [heads, splits, kv_rank]
    LatentRing ring;
    int heads, kv_rank;
    int window;         // visible positions including the token itself
    float scale;
};

// Shared memory of one CTA: cache tile, queries, sums, weights.
template <typename T>
inline size_t latent_decode_smem(int ld, int kv_rank) {
    const int pitch = ld + 16 / (int)sizeof(T) * ((ld * (int)sizeof(T) / 16) % 2 ? 0 : 1);
    return (size_t)kLdTile * pitch * sizeof(T) + (size_t)kLdHeads * ld * 4 + (size_t)(kv_rank + 1) * kLdHeads * 4 +
           (size_t)kLdTile * kLdHeads * 4 + kLdHeads * 4 + 64;
}

template <typename T>
__global__ void __launch_bounds__(256)
latent_decode_kernel(LatentDecodeArgs A) {
    constexpr int VN = Vec16<T>::N;
    extern __shared__ __align__(16) unsigned char ld_raw[];
    const int ld = A.ring.ld, vecs = ld / VN;
    const int pitch = ld + ((vecs & 1) ? 0 : VN);  // an odd number of 16-byte vectors: rows fall into different banks
    T* tile = reinterpret_cast<T*>(ld_raw);                              // [32][pitch]
    float* qs = reinterpret_cast<float*>(tile + (size_t)kLdTile * pitch);  // [8][ld]
    float* p_s = qs + kLdHeads * ld;                                       // [32][8]
    float* corr_s = p_s + kLdTile * kLdHeads;                              // [8]
    float* o_s = corr_s + kLdHeads;                                        // [kv_rank][8]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int head0 = blockIdx.x * kLdHeads, split = blockIdx.y, splits = gridDim.y;
    llvq_dependent_enter();
    const long long pos = *A.pos;
    const int n = (int)min((long long)A.window, pos + 1);  // visible positions pos - n + 1 .. pos
    int per = (n + splits - 1) / splits;
    per = (per + kLdTile - 1) / kLdTile * kLdTile;
    const int t0 = split * per, t1 = min(n, t0 + per);
    const int slot0 = (int)((pos - n + 1) % A.ring.slots);  // n <= slots: at most one wrap below
    const float qscale = A.scale * kLog2e;
    for (int i = tid; i < kLdHeads * ld; i += 256) {
        const int h = head0 + i / ld;
        qs[i] = h < A.heads ? reinterpret_cast<const float*>(A.qlat)[(size_t)h * ld + i % ld] * qscale : 0.0f;
    }
    for (int i = tid; i < A.kv_rank * kLdHeads; i += 256) o_s[i] = 0.0f;
    float m = -INFINITY, l = 0.0f;  // of this warp's head
    const uint4* rows = reinterpret_cast<const uint4*>(A.ring.rows);
    for (int base = t0; base < t1; base += kLdTile) {
        const int here = min(kLdTile, t1 - base);
        __syncthreads();  // the tile and the weights of the step before are read
        for (int i = tid; i < here * vecs; i += 256) {
            const int r = i / vecs, c = i - r * vecs;
            int slot = slot0 + base + r;
            if (slot >= A.ring.slots) slot -= A.ring.slots;
            const unsigned int dst = (unsigned int)__cvta_generic_to_shared(tile + (size_t)r * pitch + c * VN);
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(rows + (size_t)slot * vecs + c) : "memory");
        }
        asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        // scores: warp = head, lane = position
        float s = -INFINITY;
        if (lane < here) {
            const uint4* kr = reinterpret_cast<const uint4*>(tile + (size_t)lane * pitch);
            const float* q = qs + warp * ld;
            float a0 = 0.0f, a1 = 0.0f;
#pragma unroll 2
            for (int c = 0; c < vecs; ++c) {
                float f[VN];
                Vec16<T>::widen(kr[c], f);
#pragma unroll
                for (int j = 0; j < VN; j += 4) {
                    const float4 qv = *reinterpret_cast<const float4*>(q + c * VN + j);
                    a0 = fmaf(f[j], qv.x, a0);
                    a1 = fmaf(f[j + 1], qv.y, a1);
                    a0 = fmaf(f[j + 2], qv.z, a0);
                    a1 = fmaf(f[j + 3], qv.w, a1);
                }
            }
            s = a0 + a1;
        }
        const float m_new = fmaxf(m, warp_max_f(s));  // finite: a tile holds a visible position
        const float corr = exp2f(m - m_new), p = exp2f(s - m_new);
        l = l * corr + warp_sum_f(p);
        m = m_new;
        p_s[lane * kLdHeads + warp] = p;
        if (lane == 0) corr_s[warp] = corr;
        __syncthreads();
        // sums of latents: thread = dimensions d, d + 256, ..., all 8 heads
        for (int d = tid; d < A.kv_rank; d += 256) {
            float acc[kLdHeads];
#pragma unroll
            for (int h = 0; h < kLdHeads; ++h) acc[h] = o_s[d * kLdHeads + h] * corr_s[h];
#pragma unroll 4
            for (int k = 0; k < here; ++k) {
                const float c = to_f32(tile[(size_t)k * pitch + d]);
                const float4 pa = *reinterpret_cast<const float4*>(p_s + k * kLdHeads);
                const float4 pb = *reinterpret_cast<const float4*>(p_s + k * kLdHeads + 4);
                acc[0] = fmaf(pa.x, c, acc[0]), acc[1] = fmaf(pa.y, c, acc[1]);
                acc[2] = fmaf(pa.z, c, acc[2]), acc[3] = fmaf(pa.w, c, acc[3]);
                acc[4] = fmaf(pb.x, c, acc[4]), acc[5] = fmaf(pb.y, c, acc[5]);
                acc[6] = fmaf(pb.z, c, acc[6]), acc[7] = fmaf(pb.w, c, acc[7]);
            }
#pragma unroll
            for (int h = 0; h < kLdHeads; ++h) o_s[d * kLdHeads + h] = acc[h];
        }
    }
    if (head0 + warp < A.heads && lane == 0) {
        float* ml = A.part_ml + ((size_t)(head0 + warp) * splits + split) * 2;
        ml[0] = m;  // -inf for a split beyond the visible positions
        ml[1] = l;
    }
    __syncthreads();
    if (t0 < t1) {
        for (int i = tid; i < A.kv_rank * kLdHeads; i += 256) {
            const int h = i / A.kv_rank, d = i - h * A.kv_rank;
            if (head0 + h < A.heads) A.part_o[((size_t)(head0 + h) * splits + split) * A.kv_rank + d] = o_s[d * kLdHeads + h];
        }
    }
}

constexpr int kLmHeads = 16;  // rows of a tensor-core tile
constexpr int kLmKeys = 64;   // positions per tile, 8 per warp
constexpr int kLmPPitch = kLmKeys + 8;

// Row pitch of the staged queries and cache rows: whole pairs of 16-wide steps (zeros beyond ld), an odd number of
// 16-byte vectors.
__host__ __device__ inline int lm_pitch(int ld) { return (ld + 31) / 32 * 32 + 8; }
inline size_t latent_decode_mma_smem(int ld) {
    return (size_t)(kLmHeads + kLmKeys) * lm_pitch(ld) * sizeof(bf16) + kLmHeads * kLmPPitch * sizeof(bf16) + 2 * 8 * kLmHeads * sizeof(float);
}

// CH: 16-dimension pieces of the latent per warp (kv_rank <= 128 CH).
template <int CH>
__global__ void __launch_bounds__(256)
latent_decode_mma_kernel(LatentDecodeArgs A) {
    extern __shared__ __align__(16) unsigned char lm_raw[];
    const int ld = A.ring.ld, vecs = ld / 8, pitch = lm_pitch(ld), kpad = pitch - 8;
    bf16* sq = reinterpret_cast<bf16*>(lm_raw);           // [16][pitch]
    bf16* sk = sq + kLmHeads * pitch;                     // [64][pitch]
    bf16* sp = sk + kLmKeys * pitch;                      // [16][72] softmax weights
    float* red_m = reinterpret_cast<float*>(sp + kLmHeads * kLmPPitch);  // [8][16]
    float* red_l = red_m + 8 * kLmHeads;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int head0 = blockIdx.x * kLmHeads, split = blockIdx.y, splits = gridDim.y;
    const int pad_v = (kpad - ld) / 8;  // zero vectors behind a row
    for (int i = tid; i < (kLmHeads + kLmKeys) * pad_v; i += 256)
        *reinterpret_cast<uint4*>(sq + (size_t)(i / pad_v) * pitch + ld + 8 * (i % pad_v)) = make_uint4(0, 0, 0, 0);
    llvq_dependent_enter();
    const long long pos = *A.pos;
    const int n = (int)min((long long)A.window, pos + 1);  // visible positions pos - n + 1 .. pos
    int per = (n + splits - 1) / splits;
    per = (per + kLmKeys - 1) / kLmKeys * kLmKeys;
    const int t0 = split * per, t1 = min(n, t0 + per);
    const int slot0 = (int)((pos - n + 1) % A.ring.slots);  // n <= slots: at most one wrap below
    const bf16* rows = reinterpret_cast<const bf16*>(A.ring.rows);
    const bf16* qlat = reinterpret_cast<const bf16*>(A.qlat);
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};  // of heads g and g + 8, the same in every warp
    float o[CH][2][4];
#pragma unroll
    for (int c = 0; c < CH; ++c)
#pragma unroll
        for (int k = 0; k < 2; ++k)
#pragma unroll
            for (int j = 0; j < 4; ++j) o[c][k][j] = 0.0f;
    if (t0 < t1) {
        for (int r = warp; r < kLmHeads; r += 8) {
            const bool in = head0 + r < A.heads;
            for (int c = lane; c < vecs; c += 32) copy16_async(sq + r * pitch + 8 * c, in ? qlat + (size_t)(head0 + r) * ld + 8 * c : qlat, in);
        }
    }
    const float s2 = A.scale * kLog2e;
    for (int base = t0; base < t1; base += kLmKeys) {
        const int here = min(kLmKeys, t1 - base);
#pragma unroll 4
        for (int r = warp; r < kLmKeys; r += 8) {  // rows beyond the split are zero
            int slot = slot0 + base + r;
            if (slot >= A.ring.slots) slot -= A.ring.slots;
            const bool in = r < here;
            const bf16* src = in ? rows + (size_t)slot * ld : rows;
            for (int c = lane; c < vecs; c += 32) copy16_async(sk + r * pitch + 8 * c, src + 8 * c, in);
        }
        asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        // ---- scores of this warp's 8 positions against 16 heads ----
        float s[2][4];
#pragma unroll
        for (int j = 0; j < 4; ++j) s[0][j] = s[1][j] = 0.0f;
#pragma unroll 3
        for (int k = 0; k < kpad; k += 32) {
            unsigned int b[4], a0[4], a1[4];
            ldmatrix4(b, sk + (warp * 8 + (lane & 7)) * pitch + k + (lane >> 3) * 8);
            ldmatrix4(a0, sq + (lane & 15) * pitch + k + (lane >> 4) * 8);
            ldmatrix4(a1, sq + (lane & 15) * pitch + k + 16 + (lane >> 4) * 8);
            mma_bf16(s[0], a0, b[0], b[1]);
            mma_bf16(s[1], a1, b[2], b[3]);
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float v = warp * 8 + 2 * t + (j & 1) < here ? (s[0][j] + s[1][j]) * s2 : -INFINITY;
            s[0][j] = v;
            mx[j >> 1] = fmaxf(mx[j >> 1], v);
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            if (t == 0) red_m[warp * kLmHeads + g + 8 * r] = mx[r];
        }
        __syncthreads();
        float corr[2], sum[2] = {0.0f, 0.0f};
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float mn = m[r];
#pragma unroll
            for (int w = 0; w < 8; ++w) mn = fmaxf(mn, red_m[w * kLmHeads + g + 8 * r]);  // finite: a tile holds a visible position
            corr[r] = exp2f(m[r] - mn);
            m[r] = mn;
        }
        float p[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            p[j] = exp2f(s[0][j] - m[j >> 1]);
            sum[j >> 1] += p[j];
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
            sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
            if (t == 0) red_l[warp * kLmHeads + g + 8 * r] = sum[r];
            *reinterpret_cast<unsigned int*>(sp + (g + 8 * r) * kLmPPitch + warp * 8 + 2 * t) = pack_bf16(p[2 * r], p[2 * r + 1]);
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            l[r] *= corr[r];
#pragma unroll
            for (int w = 0; w < 8; ++w) l[r] += red_l[w * kLmHeads + g + 8 * r];
        }
        // ---- sums of latents: this warp's 16-dimension pieces ----
        unsigned int a[4][4];
#pragma unroll
        for (int k = 0; k < 4; ++k) ldmatrix4(a[k], sp + (lane & 15) * kLmPPitch + k * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const int d0 = (warp + 8 * c) * 16;
            if (d0 >= A.kv_rank) break;
#pragma unroll
            for (int k = 0; k < 2; ++k)
#pragma unroll
                for (int j = 0; j < 4; ++j) o[c][k][j] *= corr[j >> 1];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                unsigned int b[4];
                ldmatrix4_trans(b, sk + (k * 16 + (lane & 15)) * pitch + d0 + (lane >> 4) * 8);
                mma_bf16(o[c][0], a[k], b[0], b[1]);
                mma_bf16(o[c][1], a[k], b[2], b[3]);
            }
        }
        __syncthreads();  // the tile and the weights are read
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int head = head0 + g + 8 * r;
        if (head >= A.heads) continue;
        const size_t at = (size_t)head * splits + split;
        if (warp == 0 && t == 0) {
            A.part_ml[2 * at] = m[r];  // -inf for a split beyond the visible positions
            A.part_ml[2 * at + 1] = l[r];
        }
        if (t0 >= t1) continue;
#pragma unroll
        for (int c = 0; c < CH; ++c)
#pragma unroll
            for (int k = 0; k < 2; ++k)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int d = (warp + 8 * c) * 16 + k * 8 + 2 * t + j;
                    if (d < A.kv_rank) A.part_o[at * A.kv_rank + d] = o[c][k][2 * r + j];
                }
    }
}

struct LatentValueArgs {
    const float* part_ml;
    const float* part_o;
    const float* sink;  // [heads] or null
    const void* uv;     // [heads * vdim, ldk] of T
    float* ctx;         // [heads, vdim]
    int heads, vdim, kv_rank, ldk, splits;
};

constexpr int kLvRows = 32;  // value rows per CTA, 4 per warp

// grid = (heads, ceil(vdim / 32)), 256 threads. Dynamic shared memory: ldk + splits floats.
template <typename T>
__global__ void __launch_bounds__(256)
latent_value_kernel(LatentValueArgs A) {
    constexpr int VN = Vec16<T>::N;
    extern __shared__ __align__(16) float lv_smem[];
    __shared__ float red[8];
    float* o_s = lv_smem;           // [ldk]
    float* f_s = lv_smem + A.ldk;   // [splits]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x;
    const int vecs = A.ldk / VN;
    const uint4* W = reinterpret_cast<const uint4*>(A.uv) + (size_t)h * A.vdim * vecs;
    const int row0 = blockIdx.y * kLvRows + warp * 4;
    uint4 w[4];  // the first vectors of W_uv are on their way before the dependency wait
    if (row0 < A.vdim && lane < vecs) {
#pragma unroll
        for (int i = 0; i < 4; ++i) w[i] = __ldg(W + (size_t)min(row0 + i, A.vdim - 1) * vecs + lane);
    }
    llvq_dependent_enter();
    const float* ml = A.part_ml + (size_t)h * A.splits * 2;
    float m = A.sink ? A.sink[h] * kLog2e : -INFINITY;
    for (int s = lane; s < A.splits; s += 32) m = fmaxf(m, ml[2 * s]);
    m = warp_max_f(m);
    float l = 0.0f;
    for (int s = tid; s < A.splits; s += 256) {
        const float f = ml[2 * s] == -INFINITY ? 0.0f : exp2f(ml[2 * s] - m);
        f_s[s] = f;
        l = fmaf(ml[2 * s + 1], f, l);
    }
    l = block_sum_f(l, red);  // also publishes f_s
    if (A.sink) l += exp2f(A.sink[h] * kLog2e - m);
    const float inv = 1.0f / l;
    const float* po = A.part_o + (size_t)h * A.splits * A.kv_rank;
    for (int d = tid; d < A.ldk; d += 256) {
        float o = 0.0f;
        if (d < A.kv_rank) {
#pragma unroll 8
            for (int s = 0; s < A.splits; ++s) {
                const float f = f_s[s], v = po[(size_t)s * A.kv_rank + d];
                if (f != 0.0f) o = fmaf(v, f, o);  // the sums of an empty split are not written
            }
        }
        o_s[d] = o * inv;
    }
    __syncthreads();
    float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    if (row0 < A.vdim) {
        for (int v = lane; v < vecs; v += 32) {
            if (v != lane) {
#pragma unroll
                for (int i = 0; i < 4; ++i) w[i] = __ldg(W + (size_t)min(row0 + i, A.vdim - 1) * vecs + v);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                float f[VN];
                Vec16<T>::widen(w[i], f);
#pragma unroll
                for (int j = 0; j < VN; ++j) acc[i] = fmaf(f[j], o_s[v * VN + j], acc[i]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float s = warp_sum_f(acc[i]);
        if (lane == 0 && row0 + i < A.vdim) A.ctx[(size_t)h * A.vdim + row0 + i] = s;
    }
}

}  // namespace llvq
