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
//   delta_prep_kernel   a portion's convolutions, unit vectors, k q, decays and step sizes.
//   delta_scan_kernel   the recurrence of a portion: a CTA keeps 32 columns of a head's state in registers, LANES lanes
//                       per column, and walks the tokens; keys and queries come in double-buffered tiles.
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
    __shared__ float red[8], col_s[8][2][kDtCols], u_s[kDtCols];
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
    const bool owner = blockIdx.x == 0 && h == g * (A.heads / A.kv_heads);  // stores the inputs of the shared q and k
    float qq = 0.0f, kk = 0.0f, kq = 0.0f;
    for (int i = tid; i < A.dim; i += kDtThreads) {
        const int cq = g * A.dim + i, ck = (A.kv_heads + g) * A.dim + i;
        const float xq = A.x[cq], xk = A.x[ck];
        const float q = silu_f(conv_token(A.conv_w + (size_t)cq * A.taps, A.taps, A.conv, channels, cq, pos, xq));
        const float k = silu_f(conv_token(A.conv_w + (size_t)ck * A.taps, A.taps, A.conv, channels, ck, pos, xk));
        if (owner) {
            A.conv[(size_t)(pos % A.taps) * channels + cq] = xq;
            A.conv[(size_t)(pos % A.taps) * channels + ck] = xk;
        }
        q_s[i] = q;
        k_s[i] = k;
        qq = fmaf(q, q, qq), kk = fmaf(k, k, kk), kq = fmaf(k, q, kq);
    }
    qq = block_sum_f(qq, red);  // also publishes q_s and k_s
    kk = block_sum_f(kk, red);
    kq = block_sum_f(kq, red);
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
    if (tid < kDtCols && c0 + tid < A.vp) {
        const int j = c0 + tid;
        float tk = 0.0f, tq = 0.0f;
#pragma unroll
        for (int w = 0; w < 8; ++w) tk += col_s[w][0][tid], tq += col_s[w][1][tid];
        float u = 0.0f;
        if (j < A.vdim) {
            const int cv = 2 * A.kv_heads * A.dim + h * A.vdim + j;
            const float xv = A.x[cv];
            const float v = silu_f(conv_token(A.conv_w + (size_t)cv * A.taps, A.taps, A.conv, channels, cv, pos, xv));
            A.conv[(size_t)(pos % A.taps) * channels + cv] = xv;
            u = sigmoid_f(A.b[h]) * (v - fk * carry(dec, tk, 0.0f));
        }
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

// Lanes of a column and rows of a lane (in fours) of the scan; dims beyond 1024 are not served.
__host__ __device__ inline int delta_lanes(int dim) { return dim <= 256 ? 8 : 32; }
__host__ __device__ inline int delta_fours(int dim) { return (dim + 4 * delta_lanes(dim) - 1) / (4 * delta_lanes(dim)); }
// Row length of the unit vectors of a portion: what the lanes of a column hold, zeros beyond dim.
__host__ __device__ inline int delta_padded(int dim) { return delta_fours(dim) * 4 * delta_lanes(dim); }
__host__ __device__ inline int delta_tile(int dim) { return dim <= 128 ? 32 : dim <= 256 ? 16 : 4; }  // tokens of a staged tile

struct DeltaPrepArgs {
    const void* x;   // rows of one product, stride ldx: [q | k | v] channels
    const float* ba; // [n, 2 heads]: b, then a
    const float* conv_w;
    const float* conv;
    const float* decay;
    const float* dt_bias;
    float* qk;       // [n, kv_heads, 2, dp]: unit key, unit query / sqrt(dim)
    float* v;        // [n, heads, vdim]
    float* sc;       // [n, heads, 4]: g - 1, beta, k q, 0
    long long pos0;
    int ldx, heads, kv_heads, dim, vdim, taps, dp;
};

// grid = n, 256 threads. Dynamic shared memory: kv_heads floats.
template <typename T>
__global__ void __launch_bounds__(256)
delta_prep_kernel(DeltaPrepArgs A) {
    extern __shared__ float kq_s[];
    llvq_dependent_enter();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x;
    const int channels = 2 * A.kv_heads * A.dim + A.heads * A.vdim;
    const T* X = reinterpret_cast<const T*>(A.x);
    auto conv = [&](int c) {
        const float* w = A.conv_w + (size_t)c * A.taps;
        float u = 0.0f;
        for (int k = 0; k < A.taps; ++k) u = fmaf(w[A.taps - 1 - k], conv_input(X, A.ldx, 0.0f, A.conv, channels, A.taps, A.pos0, t - k, c), u);
        return silu_f(u);
    };
    for (int g = warp; g < A.kv_heads; g += 8) {
        float* kd = A.qk + ((size_t)t * A.kv_heads + g) * 2 * A.dp;
        float* qd = kd + A.dp;
        float qq = 0.0f, kk = 0.0f, kq = 0.0f;
        for (int i = lane; i < A.dp; i += 32) {
            float q = 0.0f, k = 0.0f;
            if (i < A.dim) q = conv(g * A.dim + i), k = conv((A.kv_heads + g) * A.dim + i);
            kd[i] = k;
            qd[i] = q;
            qq = fmaf(q, q, qq), kk = fmaf(k, k, kk), kq = fmaf(k, q, kq);
        }
        const float fq = 1.0f / sqrtf(warp_sum_f(qq) + kUnitEps) / sqrtf((float)A.dim), fk = 1.0f / sqrtf(warp_sum_f(kk) + kUnitEps);
        kq = warp_sum_f(kq) * fq * fk;
        for (int i = lane; i < A.dp; i += 32) kd[i] *= fk, qd[i] *= fq;  // what this lane wrote
        if (lane == 0) kq_s[g] = kq;
    }
    for (int c = threadIdx.x; c < A.heads * A.vdim; c += 256) A.v[(size_t)t * A.heads * A.vdim + c] = conv(2 * A.kv_heads * A.dim + c);
    __syncthreads();
    const int rep = A.heads / A.kv_heads;
    for (int h = threadIdx.x; h < A.heads; h += 256) {
        const float* ba = A.ba + (size_t)t * 2 * A.heads;
        reinterpret_cast<float4*>(A.sc)[(size_t)t * A.heads + h] =
            make_float4(expm1f(-A.decay[h] * softplus_f(ba[A.heads + h] + A.dt_bias[h])), sigmoid_f(ba[h]), kq_s[h / rep], 0.0f);
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
    return (size_t)delta_tile(dim) * (2 * (2 * delta_padded(dim) + kDtCols + 4) + kDtCols) * sizeof(float);
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

// grid = (ceil(vdim / 32), heads), 32 * LANES threads: lane l of a column holds rows 4 (l + LANES m) .. + 3, m < FOURS.
template <int LANES, int FOURS>
__global__ void __launch_bounds__(kDtCols * LANES)
delta_scan_kernel(DeltaScanArgs A) {
    constexpr int kThreads = kDtCols * LANES, dp = 4 * LANES * FOURS;
    extern __shared__ __align__(16) float ds_smem[];
    const int TT = delta_tile(A.dim), tid = threadIdx.x, l = tid % LANES, col = tid / LANES;
    const int h = blockIdx.y, g = h / (A.heads / A.kv_heads), j = blockIdx.x * kDtCols + col;
    float* qk_s = ds_smem;                          // [2][TT][2 dp]
    float* sc_s = qk_s + 2 * TT * 2 * dp;           // [2][TT][4]
    float* v_s = sc_s + 2 * TT * 4;                 // [2][TT][32]
    float* o_s = v_s + 2 * TT * kDtCols;            // [TT][32]
    llvq_dependent_enter();
    auto copy16 = [](float* dst, const float* src) {
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned int)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
    };
    const int c0 = blockIdx.x * kDtCols, cols = min(kDtCols, A.vdim - c0);
    auto stage = [&](int t0, int buf) {
        const int here = min(TT, A.n - t0);
        constexpr int per = 2 * dp / 4;
        for (int i = tid; i < here * per; i += kThreads) {
            const int t = i / per, c = i - t * per;
            copy16(qk_s + (size_t)(buf * TT + t) * 2 * dp + 4 * c, A.qk + ((size_t)(t0 + t) * A.kv_heads + g) * 2 * dp + 4 * c);
        }
        for (int t = tid; t < here; t += kThreads) copy16(sc_s + (buf * TT + t) * 4, A.sc + ((size_t)(t0 + t) * A.heads + h) * 4);
        for (int i = tid; i < here * kDtCols; i += kThreads) {
            const int t = i / kDtCols, c = i - t * kDtCols;
            if (c < cols)
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned int)__cvta_generic_to_shared(v_s + buf * TT * kDtCols + i)),
                             "l"(A.v + ((size_t)(t0 + t) * A.heads + h) * A.vdim + c0 + c)
                             : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    f32x2 S[FOURS][2];
    const size_t half = (size_t)A.heads * A.dim * A.vp, base = (size_t)h * A.dim * A.vp + j;
    const float* S0 = A.state + (A.pos0 & 1) * half + base;
#pragma unroll
    for (int m = 0; m < FOURS; ++m) {
        float e[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int i = 4 * (l + LANES * m) + r;
            e[r] = A.pos0 > 0 && i < A.dim && j < A.vdim ? S0[(size_t)i * A.vp] : 0.0f;
        }
        S[m][0] = pack2(e[0], e[1]);
        S[m][1] = pack2(e[2], e[3]);
    }
    for (int t0 = 0, buf = 0; t0 < A.n; t0 += TT, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the tile is staged, the outputs before are stored and the other buffer is read
        if (t0 + TT < A.n) stage(t0 + TT, buf ^ 1);
        const int here = min(TT, A.n - t0);
        for (int t = 0; t < here; ++t) {
            const float* kr = qk_s + (size_t)(buf * TT + t) * 2 * dp + 4 * l;
            const float4 sc = *reinterpret_cast<const float4*>(sc_s + (buf * TT + t) * 4);
            const float v = v_s[(buf * TT + t) * kDtCols + col];
            f32x2 k[FOURS][2], sk[2] = {0ull, 0ull}, sq[2] = {0ull, 0ull};
#pragma unroll
            for (int m = 0; m < FOURS; ++m) {
                const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(kr + 4 * LANES * m), qq = *reinterpret_cast<const ulonglong2*>(kr + dp + 4 * LANES * m);
                k[m][0] = kk.x, k[m][1] = kk.y;
                sk[0] = fma2(S[m][0], kk.x, sk[0]);
                sk[1] = fma2(S[m][1], kk.y, sk[1]);
                sq[0] = fma2(S[m][0], qq.x, sq[0]);
                sq[1] = fma2(S[m][1], qq.y, sq[1]);
            }
            const float2 k0 = unpack2(sk[0]), k1 = unpack2(sk[1]), q0 = unpack2(sq[0]), q1 = unpack2(sq[1]);
            float tk = (k0.x + k0.y) + (k1.x + k1.y), tq = (q0.x + q0.y) + (q1.x + q1.y);
#pragma unroll
            for (int o = LANES / 2; o > 0; o >>= 1) {
                tk += __shfl_xor_sync(0xffffffffu, tk, o);
                tq += __shfl_xor_sync(0xffffffffu, tq, o);
            }
            const float u = sc.y * (v - carry(sc.x, tk, 0.0f));
            const f32x2 g2 = pack2(sc.x, sc.x), u2 = pack2(u, u);
#pragma unroll
            for (int m = 0; m < FOURS; ++m) {
                S[m][0] = fma2(k[m][0], u2, fma2(g2, S[m][0], S[m][0]));
                S[m][1] = fma2(k[m][1], u2, fma2(g2, S[m][1], S[m][1]));
            }
            if (l == 0) o_s[t * kDtCols + col] = fmaf(sc.z, u, carry(sc.x, tq, 0.0f));
        }
        __syncthreads();
        for (int i = tid; i < here * kDtCols; i += kThreads) {
            const int t = i / kDtCols, c = i - t * kDtCols;
            if (c < cols) A.o[((size_t)(t0 + t) * A.heads + h) * A.vdim + c0 + c] = o_s[i];
        }
    }
    if (j >= A.vdim) return;
    float* Sn = A.state + ((A.pos0 + A.n) & 1) * half + base;
#pragma unroll
    for (int m = 0; m < FOURS; ++m) {
        const float2 a = unpack2(S[m][0]), b = unpack2(S[m][1]);
        const float e[4] = {a.x, a.y, b.x, b.y};
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int i = 4 * (l + LANES * m) + r;
            if (i < A.dim) Sn[(size_t)i * A.vp] = e[r];
        }
    }
}

// out[t, h, :] = o / sqrt(mean(o^2) + eps) * w * silu(gate); grid = rows, 256 threads: a warp takes a head at a time.
template <typename T>
__global__ void __launch_bounds__(256)
head_gate_rows_kernel(const float* __restrict__ o, const float* __restrict__ w, const T* __restrict__ gate, int ldg, T* __restrict__ out, int ldo,
                      int heads, int vdim, float eps) {
    llvq_dependent_enter();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const size_t t = blockIdx.x;
    for (int h = warp; h < heads; h += 8) {
        const float* src = o + (t * heads + h) * vdim;
        const float f = warp_inv_rms(src, vdim, eps);
        for (int i = lane; i < vdim; i += 32)
            out[t * ldo + (size_t)h * vdim + i] = from_f32<T>(src[i] * f * w[i] * silu_f(to_f32(gate[t * ldg + (size_t)h * vdim + i])));
    }
}

}  // namespace llvq
