// Gated delta rule: per head a state S [dim, vdim] in f32,
//
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//
// with unit vectors k and q / sqrt(dim) from short convolutions and a silu, beta = sigmoid(b),
// g = exp(-exp(A_log) softplus(a + dt_bias)). Both read-outs are taken from the state before the token,
// S^T k and S^T q, so that one reduction over dim serves them: o = g S^T q + (k q) u. Stores follow
// linear_recurrence.cuh (decays less one, convolution inputs by position, the state in two halves by the position's parity);
// a head's state is [dim, vp] with vp the value size in whole vectors of four, zero beyond vdim.
//
//   delta_token_kernel  a CTA takes 32 value columns of a head; the head's last CTA to arrive norms and gates its
//                       output: no CTA waits for another.
//   delta_prep_kernel   a portion's convolutions, and the scalars of every four tokens.
//   delta_scan_kernel   the recurrence of a portion: a CTA keeps 32 columns of a head's state in registers, LANES lanes
//                       per four columns, and walks the tokens; keys and queries come in double-buffered tiles.
//   head_gate_rows_kernel  per head: o / rms(o) * w * silu(gate).
#pragma once
#include "linear_recurrence.cuh"

namespace llvq {

constexpr int kDtCols = 32, kDtThreads = 256, kDtKeep = 8;  // columns of a CTA; row groups of 32 rows kept in registers

struct DeltaArgs {
    const float* x;       // [2 kv_heads * dim + heads * vdim] inputs of the convolutions: q, k, v
    const float* gate;    // [heads, vdim]
    const float* b;       // [heads]
    const float* a;       // [heads]
    const float* conv_w;  // [channels, taps]
    const float* decay;   // [heads]: exp(A_log)
    const float* dt_bias; // [heads]
    const float* norm;    // [vdim]
    const long long* pos;
    float* conv;          // [taps, channels]
    float* state;         // [2, heads, dim, vp]
    float* o;             // scratch [heads, vp]
    unsigned int* arrived; // [heads], zero before the first launch and after every one
    float* out;           // [heads, vdim]
    int heads, kv_heads, dim, vdim, vp, taps;
    float eps;
};

constexpr float kUnitEps = 1e-6f;

inline size_t delta_token_smem(int dim) { return (size_t)2 * dim * sizeof(float); }

// grid = (ceil(vp / 32), heads).
__global__ void __launch_bounds__(kDtThreads)
delta_token_kernel(DeltaArgs A) {
    extern __shared__ __align__(16) float dt_smem[];
    __shared__ float red[8], red3[8][3], col_s[8][2][kDtCols], u_s[kDtCols];
    __shared__ int last_s;
    float* q_s = dt_smem;
    float* k_s = dt_smem + A.dim;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, g = h / (A.heads / A.kv_heads), c0 = blockIdx.x * kDtCols;
    const int j4 = (tid & 7) * 4, rg = tid >> 3;  // this thread's four columns, its rows rg, rg + 32, ...
    const bool in = c0 + j4 < A.vp;
    const int channels = 2 * A.kv_heads * A.dim + A.heads * A.vdim;
    llvq_dependent_enter();
    const long long pos = *A.pos;
    const size_t half = (size_t)A.heads * A.dim * A.vp, base = (size_t)h * A.dim * A.vp + c0 + j4;
    const float* S = A.state + (pos & 1) * half + base;
    float* Sn = A.state + ((pos + 1) & 1) * half + base;
    auto load = [&](int i) { return pos > 0 && in && i < A.dim ? *reinterpret_cast<const float4*>(S + (size_t)i * A.vp) : make_float4(0.0f, 0.0f, 0.0f, 0.0f); };
    float4 keep[kDtKeep];
#pragma unroll
    for (int k = 0; k < kDtKeep; ++k) keep[k] = load(rg + 32 * k);

    // ---- the token's query, key and value ----
    const int conv_row = (int)((unsigned int)pos % (unsigned int)A.taps), j = c0 + tid, cv = 2 * A.kv_heads * A.dim + h * A.vdim + j;
    const bool own_col = tid < kDtCols && j < A.vdim;
    float xv = 0.0f, v = 0.0f;
    if (own_col) {
        xv = A.x[cv];
        v = silu_f(conv_token(A.conv_w + (size_t)cv * A.taps, A.taps, A.conv, channels, cv, pos, conv_row, xv));
        A.conv[(size_t)conv_row * channels + cv] = xv;
    }
    const bool owner = blockIdx.x == 0 && h == g * (A.heads / A.kv_heads);  // stores the inputs of the shared q and k
    float qq = 0.0f, kk = 0.0f, kq = 0.0f;
    for (int i = tid; i < A.dim; i += kDtThreads) {
        const int cq = g * A.dim + i, ck = (A.kv_heads + g) * A.dim + i;
        const float xq = A.x[cq], xk = A.x[ck];
        const float q = silu_f(conv_token(A.conv_w + (size_t)cq * A.taps, A.taps, A.conv, channels, cq, pos, conv_row, xq));
        const float k = silu_f(conv_token(A.conv_w + (size_t)ck * A.taps, A.taps, A.conv, channels, ck, pos, conv_row, xk));
        if (owner) {
            A.conv[(size_t)conv_row * channels + cq] = xq;
            A.conv[(size_t)conv_row * channels + ck] = xk;
        }
        q_s[i] = q;
        k_s[i] = k;
        qq = fmaf(q, q, qq), kk = fmaf(k, k, kk), kq = fmaf(k, q, kq);
    }
    qq = warp_sum_f(qq), kk = warp_sum_f(kk), kq = warp_sum_f(kq);
    if (lane == 0) red3[warp][0] = qq, red3[warp][1] = kk, red3[warp][2] = kq;
    __syncthreads();  // q_s and k_s are there as well
    qq = kk = kq = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) qq += red3[w][0], kk += red3[w][1], kq += red3[w][2];
    const float fq = 1.0f / sqrtf(qq + kUnitEps) / sqrtf((float)A.dim), fk = 1.0f / sqrtf(kk + kUnitEps);
    const float dec = expm1f(-A.decay[h] * softplus_f(A.a[h] + A.dt_bias[h]));  // g - 1

    // ---- both read-outs of the state before the token ----
    float4 sk = make_float4(0.0f, 0.0f, 0.0f, 0.0f), sq = sk;
    auto read = [&](const float4& s, int i) {
        const float k = k_s[i], q = q_s[i];
        sk.x = fmaf(s.x, k, sk.x), sk.y = fmaf(s.y, k, sk.y), sk.z = fmaf(s.z, k, sk.z), sk.w = fmaf(s.w, k, sk.w);
        sq.x = fmaf(s.x, q, sq.x), sq.y = fmaf(s.y, q, sq.y), sq.z = fmaf(s.z, q, sq.z), sq.w = fmaf(s.w, q, sq.w);
    };
#pragma unroll
    for (int k = 0; k < kDtKeep; ++k)
        if (rg + 32 * k < A.dim) read(keep[k], rg + 32 * k);
    for (int i = rg + 32 * kDtKeep; i < A.dim; i += 32) read(load(i), i);
    float v8[8] = {sk.x, sk.y, sk.z, sk.w, sq.x, sq.y, sq.z, sq.w};
#pragma unroll
    for (int e = 0; e < 8; ++e) {  // lanes 8 apart hold the same columns
        v8[e] += __shfl_xor_sync(0xffffffffu, v8[e], 8);
        v8[e] += __shfl_xor_sync(0xffffffffu, v8[e], 16);
        if (lane < 8) col_s[warp][e >> 2][j4 + (e & 3)] = v8[e];
    }
    __syncthreads();
    if (tid < kDtCols && j < A.vp) {
        float tk = 0.0f, tq = 0.0f;
#pragma unroll
        for (int w = 0; w < 8; ++w) tk += col_s[w][0][tid], tq += col_s[w][1][tid];
        const float u = own_col ? sigmoid_f(A.b[h]) * (v - fk * carry(dec, tk, 0.0f)) : 0.0f;
        u_s[tid] = u * fk;  // the key is scaled where it is used
        A.o[(size_t)h * A.vp + j] = fq * (carry(dec, tq, 0.0f) + kq * fk * u);
    }
    __syncthreads();
    const float4 u = *reinterpret_cast<const float4*>(u_s + j4);
    auto write = [&](const float4& s, int i) {
        const float k = k_s[i];
        *reinterpret_cast<float4*>(Sn + (size_t)i * A.vp) =
            make_float4(carry(dec, s.x, k * u.x), carry(dec, s.y, k * u.y), carry(dec, s.z, k * u.z), carry(dec, s.w, k * u.w));
    };
    if (in) {
#pragma unroll
        for (int k = 0; k < kDtKeep; ++k)
            if (rg + 32 * k < A.dim) write(keep[k], rg + 32 * k);
        for (int i = rg + 32 * kDtKeep; i < A.dim; i += 32) write(load(i), i);
    }
    // ---- the head's last CTA norms and gates ----
    __threadfence();
    __syncthreads();
    if (tid == 0) last_s = atomicAdd(A.arrived + h, 1u) == gridDim.x - 1u;
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    if (tid == 0) A.arrived[h] = 0;
    const float* o = A.o + (size_t)h * A.vp;
    float ss = 0.0f;
    for (int j = tid; j < A.vdim; j += kDtThreads) {
        const float t = __ldcg(o + j);
        ss = fmaf(t, t, ss);
    }
    const float r = 1.0f / sqrtf(block_sum_f(ss, red) / (float)A.vdim + A.eps);
    for (int j = tid; j < A.vdim; j += kDtThreads) A.out[(size_t)h * A.vdim + j] = __ldcg(o + j) * r * A.norm[j] * silu_f(A.gate[(size_t)h * A.vdim + j]);
}

// ---- prompt portions ----
//
// Tokens go four at a time. With G_i the decay from the group's start through token i, R_im = G_i / G_m (k_m k_i) and
// P_im = G_i / G_m (k_m q_i), the four steps from a state S are
//
//   u_i = beta_i (v_i - G_i S^T k_i - sum_{m<i} R_im u_m),  o_i = G_i S^T q_i + sum_{m<=i} P_im u_m,
//   S <- G_3 S + sum_i (G_3 / G_i) k_i u_i^T:
//
// one reduction over dim and one update of the state for four tokens. Keys and queries stay as the convolution left them;
// their scales to unit vectors go with the group's scalars.

constexpr int kDeltaGroup = 4;
constexpr int kDeltaScalars = 40;  // beta[4], G - 1 [4], key scales [4], query scales [4], G_3 / G_i key scale [4], R [6], P [10]

// Lanes of a column and rows of a lane (in fours) of the scan; dims beyond 1024 are not served.
__host__ __device__ inline int delta_lanes(int dim) { return dim <= 256 ? 16 : 32; }
__host__ __device__ inline int delta_fours(int dim) { return (dim + 4 * delta_lanes(dim) - 1) / (4 * delta_lanes(dim)); }
// Row length of the keys and queries of a portion: what the lanes of a column hold, zeros beyond dim.
__host__ __device__ inline int delta_padded(int dim) { return delta_fours(dim) * 4 * delta_lanes(dim); }
__host__ __device__ inline int delta_tile(int dim) { return dim <= 128 ? 32 : dim <= 256 ? 16 : 4; }  // tokens of a staged tile
__host__ __device__ inline int delta_groups(int n) { return (n + kDeltaGroup - 1) / kDeltaGroup; }

struct DeltaPrepArgs {
    const void* x;   // rows of one product, stride ldx: [q | k | v] channels
    const float* ba; // [n, 2 heads]: b, then a
    const float* conv_w;
    const float* conv;
    const float* decay;
    const float* dt_bias;
    float* qk;       // [groups * 4, kv_heads, 2, dp]: key, query
    float* v;        // [n, heads, vdim]
    float* sc;       // [groups, heads, 40]
    long long pos0;
    int n, ldx, heads, kv_heads, dim, vdim, taps, dp;
};

// silu of the convolution of channel c at places t0 .. t0 + 3.
template <typename T>
__device__ __forceinline__ void delta_conv4(const DeltaPrepArgs& A, int channels, int t0, int c, float (&out)[kDeltaGroup]) {
    const T* X = reinterpret_cast<const T*>(A.x);
    if (A.taps == 4) {
        const float4 w = *reinterpret_cast<const float4*>(A.conv_w + (size_t)c * 4);
        float in[kDeltaGroup + 3];
        if (t0 >= 3 && t0 + kDeltaGroup <= A.n) {
            const T* p = X + (size_t)(t0 - 3) * A.ldx + c;
#pragma unroll
            for (int k = 0; k < kDeltaGroup + 3; ++k) in[k] = to_f32(p[(size_t)k * A.ldx]);
        } else {
#pragma unroll
            for (int k = 0; k < kDeltaGroup + 3; ++k) in[k] = conv_input(X, A.ldx, 0.0f, A.conv, channels, 4, A.pos0, min(t0 + k - 3, A.n - 1), c);
        }
#pragma unroll
        for (int i = 0; i < kDeltaGroup; ++i) out[i] = silu_t<T>(fmaf(w.x, in[i], fmaf(w.y, in[i + 1], fmaf(w.z, in[i + 2], w.w * in[i + 3]))));
        return;
    }
    const float* w = A.conv_w + (size_t)c * A.taps;
#pragma unroll
    for (int i = 0; i < kDeltaGroup; ++i) {
        float u = 0.0f;
        for (int k = 0; k < A.taps; ++k) u = fmaf(w[A.taps - 1 - k], conv_input(X, A.ldx, 0.0f, A.conv, channels, A.taps, A.pos0, min(t0 + i - k, A.n - 1), c), u);
        out[i] = silu_t<T>(u);
    }
}

// The same for channels c .. c + CH - 1 (CH = 4: taps 4, dims, offsets and rows in fours, T vectors of four aligned).
template <typename T, int CH>
__device__ __forceinline__ void delta_conv(const DeltaPrepArgs& A, int channels, int t0, int c, float (&out)[CH][kDeltaGroup]) {
    if constexpr (CH == 1) {
        delta_conv4<T>(A, channels, t0, c, out[0]);
    } else {
        if (t0 < 3 || t0 + kDeltaGroup > A.n) {
#pragma unroll
            for (int j = 0; j < CH; ++j) delta_conv4<T>(A, channels, t0, c + j, out[j]);
            return;
        }
        const T* p = reinterpret_cast<const T*>(A.x) + (size_t)(t0 - 3) * A.ldx + c;
        float4 in[kDeltaGroup + 3];
#pragma unroll
        for (int k = 0; k < kDeltaGroup + 3; ++k) in[k] = load4(p + (size_t)k * A.ldx);
#pragma unroll
        for (int j = 0; j < CH; ++j) {
            const float4 w = *reinterpret_cast<const float4*>(A.conv_w + (size_t)(c + j) * 4);
            auto at = [&](int k) { return j == 0 ? in[k].x : j == 1 ? in[k].y : j == 2 ? in[k].z : in[k].w; };
#pragma unroll
            for (int i = 0; i < kDeltaGroup; ++i) out[j][i] = silu_t<T>(fmaf(w.x, at(i), fmaf(w.y, at(i + 1), fmaf(w.z, at(i + 2), w.w * at(i + 3)))));
        }
    }
}

// grid = groups, 256 threads: a warp takes a key head at a time, then all share the values. A thread takes CH channels.
template <typename T, int CH>
__global__ void __launch_bounds__(256)
delta_prep_kernel(DeltaPrepArgs A) {
    llvq_dependent_enter();
    constexpr int G = kDeltaGroup;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t0 = blockIdx.x * G, here = min(G, A.n - t0);
    const int channels = 2 * A.kv_heads * A.dim + A.heads * A.vdim, rep = A.heads / A.kv_heads;
    for (int g = warp; g < A.kv_heads; g += 8) {
        float kk[G][G], kq[G][G], qq[G];  // [i][m], m <= i
#pragma unroll
        for (int i = 0; i < G; ++i) {
            qq[i] = 0.0f;
#pragma unroll
            for (int m = 0; m <= i; ++m) kk[i][m] = kq[i][m] = 0.0f;
        }
        for (int e = lane * CH; e < A.dp; e += 32 * CH) {
            float q[CH][G], k[CH][G];
            if (e < A.dim) {
                delta_conv<T, CH>(A, channels, t0, g * A.dim + e, q);
                delta_conv<T, CH>(A, channels, t0, (A.kv_heads + g) * A.dim + e, k);
            }
#pragma unroll
            for (int i = 0; i < G; ++i) {
#pragma unroll
                for (int j = 0; j < CH; ++j)
                    if (i >= here || e >= A.dim) q[j][i] = k[j][i] = 0.0f;
                float* dst = A.qk + ((size_t)(t0 + i) * A.kv_heads + g) * 2 * A.dp + e;
                if constexpr (CH == 4) {
                    *reinterpret_cast<float4*>(dst) = make_float4(k[0][i], k[1][i], k[2][i], k[3][i]);
                    *reinterpret_cast<float4*>(dst + A.dp) = make_float4(q[0][i], q[1][i], q[2][i], q[3][i]);
                } else {
                    dst[0] = k[0][i];
                    dst[A.dp] = q[0][i];
                }
#pragma unroll
                for (int j = 0; j < CH; ++j) {
                    qq[i] = fmaf(q[j][i], q[j][i], qq[i]);
#pragma unroll
                    for (int m = 0; m <= i; ++m) {
                        kk[i][m] = fmaf(k[j][m], k[j][i], kk[i][m]);
                        kq[i][m] = fmaf(k[j][m], q[j][i], kq[i][m]);
                    }
                }
            }
        }
        float fk[G], fq[G];
        const float root = 1.0f / sqrtf((float)A.dim);
#pragma unroll
        for (int i = 0; i < G; ++i) {
#pragma unroll
            for (int m = 0; m <= i; ++m) {
                kk[i][m] = warp_sum_f(kk[i][m]);
                kq[i][m] = warp_sum_f(kq[i][m]);
            }
            fk[i] = 1.0f / sqrtf(kk[i][i] + kUnitEps);
            fq[i] = root / sqrtf(warp_sum_f(qq[i]) + kUnitEps);
        }
        for (int r = lane; r < rep; r += 32) {
            const int h = g * rep + r;
            float sc[kDeltaScalars], lg[G];
#pragma unroll
            for (int i = 0; i < kDeltaScalars; ++i) sc[i] = 0.0f;
            float sum = 0.0f;
#pragma unroll
            for (int i = 0; i < G; ++i) {
                const float* ba = A.ba + (size_t)min(t0 + i, A.n - 1) * 2 * A.heads;
                lg[i] = i < here ? -A.decay[h] * softplus_f(ba[A.heads + h] + A.dt_bias[h]) : 0.0f;
                sum += lg[i];
                sc[i] = i < here ? sigmoid_f(ba[h]) : 0.0f;
                sc[4 + i] = expm1f(sum);
                sc[8 + i] = fk[i];
                sc[12 + i] = fq[i];
            }
#pragma unroll
            for (int m = 0; m < G; ++m) {
                float from = 0.0f;  // log of the decay from token m on
#pragma unroll
                for (int i = m; i < G; ++i) {
                    if (i > m) from += lg[i];
                    const float f = i > m ? expf(from) : 1.0f;
                    sc[26 + i * (i + 1) / 2 + m] = f * kq[i][m] * fk[m] * fq[i];
                    if (i > m) sc[20 + i * (i - 1) / 2 + m] = f * kk[i][m] * fk[m] * fk[i];
                    if (i == G - 1) sc[16 + m] = f * fk[m];
                }
            }
            float4* dst = reinterpret_cast<float4*>(A.sc + ((size_t)blockIdx.x * A.heads + h) * kDeltaScalars);
#pragma unroll
            for (int i = 0; i < kDeltaScalars / 4; ++i) dst[i] = make_float4(sc[4 * i], sc[4 * i + 1], sc[4 * i + 2], sc[4 * i + 3]);
        }
    }
    for (int c = threadIdx.x * CH; c < A.heads * A.vdim; c += 256 * CH) {
        float v[CH][G];
        delta_conv<T, CH>(A, channels, t0, 2 * A.kv_heads * A.dim + c, v);
#pragma unroll
        for (int i = 0; i < G; ++i) {
            if (i >= here) break;
            float* dst = A.v + (size_t)(t0 + i) * A.heads * A.vdim + c;
            if constexpr (CH == 4)
                *reinterpret_cast<float4*>(dst) = make_float4(v[0][i], v[1][i], v[2][i], v[3][i]);
            else
                dst[0] = v[0][i];
        }
    }
}

struct DeltaScanArgs {
    const float* qk;
    const float* v;
    const float* sc;
    float* state;  // [2, heads, dim, vp]
    float* o;      // [n, heads, vdim]
    long long pos0;
    int n, heads, kv_heads, dim, vdim, vp;
};

inline size_t delta_scan_smem(int dim) {  // two tiles of keys, queries, values and scalars; one of outputs
    return (size_t)delta_tile(dim) * (2 * (2 * delta_padded(dim) + kDtCols + kDeltaScalars / kDeltaGroup) + kDtCols) * sizeof(float);
}

// Two f32 at a time.
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// grid = (ceil(vdim / 32), heads), 32 / NC * LANES threads: lane l of a group of NC (4 or 2) columns holds rows
// 4 (l + LANES m) .. + 3, m < FOURS, of each. A lane numbers its columns by its own highest bits (number c is column
// c ^ mine), so that the exchanges below always send the upper numbers, and number 0 is the column whose sums end up in
// this lane.
template <int LANES, int FOURS, int NC>
__global__ void __launch_bounds__(kDtCols / NC * LANES)
delta_scan_kernel(DeltaScanArgs A) {
    constexpr int kThreads = kDtCols / NC * LANES, dp = 4 * LANES * FOURS, G = kDeltaGroup;
    extern __shared__ __align__(16) float ds_smem[];
    const int TT = delta_tile(A.dim), tid = threadIdx.x, l = tid % LANES, cg = tid / LANES;
    const int h = blockIdx.y, g = h / (A.heads / A.kv_heads), c0 = blockIdx.x * kDtCols, cols = min(kDtCols, A.vdim - c0);
    float* qk_s = ds_smem;                                  // [2][TT][2 dp]
    float* sc_s = qk_s + 2 * TT * 2 * dp;                   // [2][TT / 4][40]
    float* v_s = sc_s + 2 * (TT / G) * kDeltaScalars;       // [2][TT][32]
    float* o_s = v_s + 2 * TT * kDtCols;                    // [TT][32]
    llvq_dependent_enter();
    auto copy16 = [](float* dst, const float* src) {
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned int)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
    };
    const int whole = delta_groups(A.n) * G;  // rows of qk
    auto stage = [&](int t0, int buf) {
        const int here = min(TT, whole - t0);
        constexpr int per = 2 * dp / 4;
        for (int i = tid; i < here * per; i += kThreads) {
            const int t = i / per, c = i - t * per;
            copy16(qk_s + (size_t)(buf * TT + t) * 2 * dp + 4 * c, A.qk + ((size_t)(t0 + t) * A.kv_heads + g) * 2 * dp + 4 * c);
        }
        constexpr int ps = kDeltaScalars / 4;
        for (int i = tid; i < here / G * ps; i += kThreads) {
            const int t = i / ps, c = i - t * ps;
            copy16(sc_s + (size_t)(buf * (TT / G) + t) * kDeltaScalars + 4 * c, A.sc + ((size_t)(t0 / G + t) * A.heads + h) * kDeltaScalars + 4 * c);
        }
        for (int i = tid; i < here * kDtCols; i += kThreads) {
            const int t = i / kDtCols, c = i - t * kDtCols;
            float* dst = v_s + buf * TT * kDtCols + i;
            if (c < cols && t0 + t < A.n)
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned int)__cvta_generic_to_shared(dst)),
                             "l"(A.v + ((size_t)(t0 + t) * A.heads + h) * A.vdim + c0 + c)
                             : "memory");
            else
                *dst = 0.0f;
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    const int mine = l / (LANES / NC);
    f32x2 S[NC][FOURS][2];
    const size_t half = (size_t)A.heads * A.dim * A.vp, base = (size_t)h * A.dim * A.vp + c0 + cg * NC;
    const bool in = c0 + cg * NC < A.vp;  // vp is a multiple of four
    const float* S0 = A.state + (A.pos0 & 1) * half + base;
#pragma unroll
    for (int m = 0; m < FOURS; ++m) {
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            float e[4];
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                const int i = 4 * (l + LANES * m) + r;
                e[r] = A.pos0 > 0 && in && i < A.dim ? S0[(size_t)i * A.vp + (c ^ mine)] : 0.0f;
            }
            S[c][m][0] = pack2(e[0], e[1]);
            S[c][m][1] = pack2(e[2], e[3]);
        }
    }
    for (int t0 = 0, buf = 0; t0 < A.n; t0 += TT, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the tile is staged, the outputs before are stored and the other buffer is read
        if (t0 + TT < A.n) stage(t0 + TT, buf ^ 1);
        const int here = min(TT, whole - t0);
        for (int t = 0; t < here; t += G) {
            const float* kr = qk_s + (size_t)(buf * TT + t) * 2 * dp + 4 * l;
            float sc[36];
#pragma unroll
            for (int i = 0; i < 9; ++i) {
                const float4 q = *reinterpret_cast<const float4*>(sc_s + (size_t)(buf * (TT / G) + t / G) * kDeltaScalars + 4 * i);
                sc[4 * i] = q.x, sc[4 * i + 1] = q.y, sc[4 * i + 2] = q.z, sc[4 * i + 3] = q.w;
            }
            f32x2 k[G][FOURS][2];
            float val[NC][2 * G];
#pragma unroll
            for (int i = 0; i < G; ++i) {
                f32x2 ak[NC], aq[NC];
#pragma unroll
                for (int m = 0; m < FOURS; ++m) {
                    const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(kr + (size_t)i * 2 * dp + 4 * LANES * m);
                    const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(kr + (size_t)i * 2 * dp + dp + 4 * LANES * m);
                    k[i][m][0] = kk.x, k[i][m][1] = kk.y;
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        ak[c] = m ? fma2(S[c][m][0], kk.x, ak[c]) : mul2(S[c][m][0], kk.x);
                        aq[c] = m ? fma2(S[c][m][0], qq.x, aq[c]) : mul2(S[c][m][0], qq.x);
                        ak[c] = fma2(S[c][m][1], kk.y, ak[c]);
                        aq[c] = fma2(S[c][m][1], qq.y, aq[c]);
                    }
                }
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float2 a = unpack2(ak[c]), b = unpack2(aq[c]);
                    val[c][i] = a.x + a.y;
                    val[c][G + i] = b.x + b.y;
                }
            }
            // the sums over dim: exchanges leave a column to a lane, the rest adds up among the lanes that share it
            float s[2 * G];
            if constexpr (NC == 4) {
                float two[2][2 * G];
#pragma unroll
                for (int e = 0; e < 2 * G; ++e)
#pragma unroll
                    for (int c = 0; c < 2; ++c) two[c][e] = val[c][e] + __shfl_xor_sync(0xffffffffu, val[2 + c][e], LANES / 2);
#pragma unroll
                for (int e = 0; e < 2 * G; ++e) s[e] = two[0][e] + __shfl_xor_sync(0xffffffffu, two[1][e], LANES / 4);
            } else {
#pragma unroll
                for (int e = 0; e < 2 * G; ++e) s[e] = val[0][e] + __shfl_xor_sync(0xffffffffu, val[1][e], LANES / 2);
            }
#pragma unroll
            for (int o = LANES / (2 * NC); o > 0; o >>= 1)
#pragma unroll
                for (int e = 0; e < 2 * G; ++e) s[e] += __shfl_xor_sync(0xffffffffu, s[e], o);
            float u[G], w[NC][G], out = 0.0f;
#pragma unroll
            for (int i = 0; i < G; ++i) {
                const float tk = s[i] * sc[8 + i], tq = s[G + i] * sc[12 + i];
                float x = v_s[(buf * TT + t + i) * kDtCols + cg * NC + mine] - carry(sc[4 + i], tk, 0.0f);
                float y = carry(sc[4 + i], tq, 0.0f);
#pragma unroll
                for (int m = 0; m < i; ++m) {
                    x = fmaf(-sc[20 + i * (i - 1) / 2 + m], u[m], x);
                    y = fmaf(sc[26 + i * (i + 1) / 2 + m], u[m], y);
                }
                u[i] = sc[i] * x;
                y = fmaf(sc[26 + i * (i + 1) / 2 + i], u[i], y);
                if ((l & 3) == i) out = y;
            }
            if (l % (LANES / NC) < G) o_s[(t + (l & 3)) * kDtCols + cg * NC + mine] = out;
#pragma unroll
            for (int i = 0; i < G; ++i) {
                w[0][i] = u[i] * sc[16 + i];
                w[1][i] = __shfl_xor_sync(0xffffffffu, w[0][i], LANES / NC);
                if constexpr (NC == 4) {
                    w[2][i] = __shfl_xor_sync(0xffffffffu, w[0][i], LANES / 2);
                    w[3][i] = __shfl_xor_sync(0xffffffffu, w[1][i], LANES / 2);
                }
            }
            const f32x2 g2 = pack2(sc[7], sc[7]);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
#pragma unroll
                for (int m = 0; m < FOURS; ++m)
#pragma unroll
                    for (int p = 0; p < 2; ++p) S[c][m][p] = fma2(g2, S[c][m][p], S[c][m][p]);
#pragma unroll
                for (int i = 0; i < G; ++i) {
                    const f32x2 w2 = pack2(w[c][i], w[c][i]);
#pragma unroll
                    for (int m = 0; m < FOURS; ++m)
#pragma unroll
                        for (int p = 0; p < 2; ++p) S[c][m][p] = fma2(k[i][m][p], w2, S[c][m][p]);
                }
            }
        }
        __syncthreads();
        for (int i = tid; i < min(TT, A.n - t0) * kDtCols; i += kThreads) {
            const int t = i / kDtCols, c = i - t * kDtCols;
            if (c < cols) A.o[((size_t)(t0 + t) * A.heads + h) * A.vdim + c0 + c] = o_s[i];
        }
    }
    if (!in) return;
    float* Sn = A.state + ((A.pos0 + A.n) & 1) * half + base;
#pragma unroll
    for (int m = 0; m < FOURS; ++m)
#pragma unroll
        for (int p = 0; p < 2; ++p)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const float2 a = unpack2(S[c][m][p]);
                const int i = 4 * (l + LANES * m) + 2 * p;
                if (i < A.dim) Sn[(size_t)i * A.vp + (c ^ mine)] = a.x;
                if (i + 1 < A.dim) Sn[(size_t)(i + 1) * A.vp + (c ^ mine)] = a.y;
            }
}

// out[t, h, :] = o / sqrt(mean(o^2) + eps) * w * silu(gate); grid = rows, 256 threads: a warp takes a head at a time, or (vec:
// whole vectors of 8 on 16-byte boundaries, vdim <= 256) each of its halves one.
template <typename T>
__global__ void __launch_bounds__(256)
head_gate_rows_kernel(const float* __restrict__ o, const float* __restrict__ w, const T* __restrict__ gate, int ldg, T* __restrict__ out, int ldo,
                      int heads, int vdim, float eps, int vec) {
    llvq_dependent_enter();
    const size_t t = blockIdx.x;
    if (vec) {
        const int lane = threadIdx.x & 15;
        const unsigned int mask = 0xffffu << (threadIdx.x & 16);
        for (int h = threadIdx.x >> 4; h < heads; h += 16) {
            const float* src = o + (t * heads + h) * vdim;
            float f[2][8], g[2][8], ss = 0.0f;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int i = (lane + 16 * k) * 8;
                if (i >= vdim) break;
                float4 a = *reinterpret_cast<const float4*>(src + i), b = *reinterpret_cast<const float4*>(src + i + 4);
                f[k][0] = a.x, f[k][1] = a.y, f[k][2] = a.z, f[k][3] = a.w, f[k][4] = b.x, f[k][5] = b.y, f[k][6] = b.z, f[k][7] = b.w;
#pragma unroll
                for (int j = 0; j < 8; ++j) g[k][j] = 0.0f, ss = fmaf(f[k][j], f[k][j], ss);
                const T* gp = gate + t * ldg + (size_t)h * vdim + i;
#pragma unroll
                for (int e = 0; e < 8; e += Vec16<T>::N) {
                    float v[Vec16<T>::N];
                    load_vec(gp + e, v);
#pragma unroll
                    for (int j = 0; j < Vec16<T>::N; ++j) g[k][e + j] = v[j];
                }
            }
#pragma unroll
            for (int s = 8; s > 0; s >>= 1) ss += __shfl_xor_sync(mask, ss, s);
            const float r = 1.0f / sqrtf(ss / (float)vdim + eps);
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int i = (lane + 16 * k) * 8;
                if (i >= vdim) break;
#pragma unroll
                for (int e = 0; e < 8; e += Vec16<T>::N) {
                    float v[Vec16<T>::N];
#pragma unroll
                    for (int j = 0; j < Vec16<T>::N; ++j) v[j] = f[k][e + j] * r * w[i + e + j] * silu_t<T>(g[k][e + j]);
                    store_vec(out + t * ldo + (size_t)h * vdim + i + e, v);
                }
            }
        }
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int h = warp; h < heads; h += 8) {
        const float* src = o + (t * heads + h) * vdim;
        const float f = warp_inv_rms(src, vdim, eps);
        for (int i = lane; i < vdim; i += 32)
            out[t * ldo + (size_t)h * vdim + i] = from_f32<T>(src[i] * f * w[i] * silu_t<T>(to_f32(gate[t * ldg + (size_t)h * vdim + i])));
    }
}

}  // namespace llvq
