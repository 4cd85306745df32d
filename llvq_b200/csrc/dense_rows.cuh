// Row kernels of a prompt portion on the dense-weight path: one CTA per token, f32 arithmetic, T activations.
//
//   embed_rows_kernel   x = scale * table[token], and its T copy for the first projections
//   postnorm_rows_kernel  t = alpha * x + y (+ bias); x = t / sqrt(mean(t^2) + eps) * w, and its T copy
//   latent_rows_kernel  the down projections of a latent-attention layer: the query latent normed into cq, the
//                       token's cache row normed, rotated and stored into the ring
//   add_norms_rows_kernel  x += y (+ the token's rows of a routed product); two norms of the sum for two sublayers
//   route_rows_kernel   a portion's rows sorted by the expert their tokens name
//   glu_rows_kernel     clamped gated unit of (gate, up) pairs with their biases
//   softcap_kernel      logits <- cap * tanh(logits / cap)
#pragma once
#include "latent_attn.cuh"

namespace llvq {

constexpr int kRowThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kRowThreads)
embed_rows_kernel(const T* __restrict__ table, int ld, int table_rows, const long long* __restrict__ tokens, float scale,
                  float* __restrict__ x, T* __restrict__ xt, int n) {
    llvq_dependent_enter();
    long long t = tokens[blockIdx.x];
    if (t < 0 || t >= table_rows) t = 0;
    const T* src = table + (size_t)t * ld;
    const size_t o = (size_t)blockIdx.x * n;
    for (int i = threadIdx.x; i < n; i += kRowThreads) {
        const float v = scale * to_f32(src[i]);
        x[o + i] = v;
        if (xt) xt[o + i] = from_f32<T>(v);
    }
}

// Dynamic shared memory: n floats. out may be x: a CTA has read its row before it writes; y may be null (alpha = 1: a
// plain norm). vec: n % 4 == 0 and every row on a 16-byte boundary.
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
postnorm_rows_kernel(const float* x, const T* __restrict__ y, const float* __restrict__ bias, const float* __restrict__ w,
                     float alpha, float eps, T* __restrict__ xt, float* out, int n, int vec) {
    extern __shared__ __align__(16) float row_s[];
    __shared__ float red[kRowThreads / 32];
    llvq_dependent_enter();
    const size_t o = (size_t)blockIdx.x * n;
    float ss = 0.0f;
    if (vec) {
        for (int i = 4 * threadIdx.x; i < n; i += 4 * kRowThreads) {
            float4 t = load4(x + o + i);
            t.x *= alpha, t.y *= alpha, t.z *= alpha, t.w *= alpha;
            if (y) {
                const float4 d = load4(y + o + i);
                const float4 b = bias ? load4(bias + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                t.x += d.x + b.x, t.y += d.y + b.y, t.z += d.z + b.z, t.w += d.w + b.w;
            }
            *reinterpret_cast<float4*>(row_s + i) = t;
            ss = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, fmaf(t.w, t.w, ss))));
        }
    } else {
        for (int i = threadIdx.x; i < n; i += kRowThreads) {
            float t = alpha * x[o + i];
            if (y) t += to_f32(y[o + i]) + (bias ? bias[i] : 0.0f);
            row_s[i] = t;
            ss = fmaf(t, t, ss);
        }
    }
    const float r = 1.0f / sqrtf(block_sum_f(ss, red) / (float)n + eps);
    if (vec) {
        for (int i = 4 * threadIdx.x; i < n; i += 4 * kRowThreads) {
            float4 t = *reinterpret_cast<const float4*>(row_s + i);
            const float4 f = load4(w + i);
            t.x *= r * f.x, t.y *= r * f.y, t.z *= r * f.z, t.w *= r * f.w;
            if (out) store4(out + o + i, t);
            if (xt) store4(xt + o + i, t);
        }
    } else {
        for (int i = threadIdx.x; i < n; i += kRowThreads) {
            const float v = row_s[i] * r * w[i];
            if (out) out[o + i] = v;
            if (xt) xt[o + i] = from_f32<T>(v);
        }
    }
}

struct AddNormsArgs {
    float* x;            // [rows, n], the residual stream
    const void* y;       // [rows, n] of T, or null
    const void* routed;  // [rows * top, n] of T, or null: row t takes places[t * top ..]
    const int* places;
    const float* w1;     // norm weights as applied, or null: no such norm
    const float* w2;
    void* h1;            // [rows, n] of T
    void* h2;
    int n, top, vec;
    float eps;
};

// Dynamic shared memory: n floats. vec: n % 4 == 0 and every row on a 16-byte boundary.
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
add_norms_rows_kernel(AddNormsArgs A) {
    extern __shared__ __align__(16) float row_s[];
    __shared__ float red[kRowThreads / 32];
    llvq_dependent_enter();
    const size_t o = (size_t)blockIdx.x * A.n;
    const T* Y = reinterpret_cast<const T*>(A.y);
    const T* P = reinterpret_cast<const T*>(A.routed);
    const int* place = A.places + (size_t)blockIdx.x * A.top;
    const bool change = Y || P;
    float ss = 0.0f;
    if (A.vec) {
        for (int i = 4 * threadIdx.x; i < A.n; i += 4 * kRowThreads) {
            float4 t = load4(A.x + o + i);
            if (Y) {
                const float4 d = load4(Y + o + i);
                t.x += d.x, t.y += d.y, t.z += d.z, t.w += d.w;
            }
            if (P) {
                float4 d = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                for (int j = 0; j < A.top; ++j) {
                    const float4 e = load4(P + (size_t)place[j] * A.n + i);
                    d.x += e.x, d.y += e.y, d.z += e.z, d.w += e.w;
                }
                t.x += d.x, t.y += d.y, t.z += d.z, t.w += d.w;
            }
            if (change) store4(A.x + o + i, t);
            *reinterpret_cast<float4*>(row_s + i) = t;
            ss = fmaf(t.x, t.x, fmaf(t.y, t.y, fmaf(t.z, t.z, fmaf(t.w, t.w, ss))));
        }
    } else {
        for (int i = threadIdx.x; i < A.n; i += kRowThreads) {
            float t = A.x[o + i];
            if (Y) t += to_f32(Y[o + i]);
            if (P) {
                float d = 0.0f;
                for (int j = 0; j < A.top; ++j) d += to_f32(P[(size_t)place[j] * A.n + i]);
                t += d;
            }
            if (change) A.x[o + i] = t;
            row_s[i] = t;
            ss = fmaf(t, t, ss);
        }
    }
    if (!A.w1 && !A.w2) return;
    const float r = 1.0f / sqrtf(block_sum_f(ss, red) / (float)A.n + A.eps);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const float* w = k ? A.w2 : A.w1;
        T* h = reinterpret_cast<T*>(k ? A.h2 : A.h1);
        if (!w) continue;
        if (A.vec) {
            for (int i = 4 * threadIdx.x; i < A.n; i += 4 * kRowThreads) {
                float4 t = *reinterpret_cast<const float4*>(row_s + i);
                const float4 f = load4(w + i);
                t.x *= r * f.x, t.y *= r * f.y, t.z *= r * f.z, t.w *= r * f.w;
                store4(h + o + i, t);
            }
        } else {
            for (int i = threadIdx.x; i < A.n; i += kRowThreads) h[o + i] = from_f32<T>(row_s[i] * r * w[i]);
        }
    }
}

constexpr int kRouteThreads = 1024;

// One CTA. Counts, ends, then a warp per expert walks all choices in order and hands out the expert's places. Dynamic shared
// memory: experts + 1 ints.
__global__ void __launch_bounds__(kRouteThreads)
route_rows_kernel(const int* __restrict__ table, int table_rows, int top, int experts, const long long* __restrict__ tokens, int rows,
                  int* __restrict__ source, int* places, int* __restrict__ ends) {
    extern __shared__ int start_s[];
    llvq_dependent_enter();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = rows * top;
    for (int e = tid; e <= experts; e += kRouteThreads) start_s[e] = 0;
    __syncthreads();
    for (int i = tid; i < n; i += kRouteThreads) {
        const int r = i / top;
        long long t = tokens[r];
        if (t < 0 || t >= table_rows) t = 0;
        const int e = min(max(table[t * top + (i - r * top)], 0), experts - 1);
        places[i] = e;  // the expert for now
        atomicAdd(start_s + e + 1, 1);
    }
    __syncthreads();
    if (warp == 0) {
        int sum = 0;
        for (int lo = 0; lo < experts; lo += 32) {
            int c = lo + lane < experts ? start_s[lo + lane + 1] : 0;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, c, o);
                if (lane >= o) c += v;
            }
            if (lo + lane < experts) ends[lo + lane] = start_s[lo + lane + 1] = sum + c;
            sum += __shfl_sync(0xffffffffu, c, 31);
        }
    }
    __syncthreads();
    for (int e = warp; e < experts; e += kRouteThreads / 32) {
        int at = start_s[e];
        const int end = start_s[e + 1];
        for (int lo = 0; lo < n && at < end; lo += 32) {
            const int i = lo + lane;
            const bool mine = i < n && places[i] == e;
            const unsigned int votes = __ballot_sync(0xffffffffu, mine);
            if (mine) source[at + __popc(votes & ((1u << lane) - 1u))] = i;
            at += __popc(votes);
        }
    }
    __syncthreads();
    for (int p = tid; p < n; p += kRouteThreads) {
        const int i = source[p];
        places[i] = p;
        source[p] = i / top;
    }
}

// y: [rows, q_rank + kv_rank + rot_dim] (q_rank only when the layer reads another layer's ring: ring.rows null).
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
latent_rows_kernel(const T* __restrict__ y, int ldy, int q_rank, const float* __restrict__ q_norm, T* __restrict__ cq,
                   const float* __restrict__ kv_norm, int kv_rank, int rot_dim, RotaryTable rt, long long pos0, LatentRing ring,
                   float eps) {
    __shared__ float red[kRowThreads / 32];
    llvq_dependent_enter();
    const T* row = y + (size_t)blockIdx.x * ldy;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < q_rank; i += kRowThreads) {
        const float v = to_f32(row[i]);
        ss = fmaf(v, v, ss);
    }
    const float r = 1.0f / sqrtf(block_sum_f(ss, red) / (float)q_rank + eps);
    for (int i = threadIdx.x; i < q_rank; i += kRowThreads) cq[(size_t)blockIdx.x * q_rank + i] = from_f32<T>(to_f32(row[i]) * r * q_norm[i]);
    if (ring.rows) store_latent_row<T>(row + q_rank, kv_norm, eps, kv_rank, rot_dim, rt, pos0 + blockIdx.x, ring, red);
}

// gu: [rows, n, 2] (gate, up) pairs, bias: [n, 2] or null; the unit times `scale` into rows of stride ldo. grid = (rows, ceil(n / (8 threads))); a thread takes four
// neighbouring outputs at a time where the row allows 16-byte loads (vec).
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
glu_rows_kernel(const T* __restrict__ gu, const float* __restrict__ bias, T* __restrict__ out, int ldo, int n, float limit, float gain, float shift,
                float scale, int vec) {
    llvq_dependent_enter();
    const T* g = gu + (size_t)blockIdx.x * 2 * n;
    T* o = out + (size_t)blockIdx.x * ldo;
    const int lo = blockIdx.y * 8 * kRowThreads, hi = min(n, lo + 8 * kRowThreads);
    if (vec) {  // n % 4 == 0, rows on 16-byte boundaries
        constexpr int LV = 8 * sizeof(T) / 16;  // 16-byte loads of four pairs
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int i = lo + 4 * (threadIdx.x + k * kRowThreads);
            if (i >= hi) break;
            float f[8], b[8];
#pragma unroll
            for (int j = 0; j < LV; ++j) {
                float t[Vec16<T>::N];
                Vec16<T>::widen(__ldg(reinterpret_cast<const uint4*>(g + 2 * i) + j), t);
#pragma unroll
                for (int e = 0; e < Vec16<T>::N; ++e) f[j * Vec16<T>::N + e] = t[e];
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) b[j] = 0.0f;
            if (bias) {
                const float4 u = __ldg(reinterpret_cast<const float4*>(bias + 2 * i)), v = __ldg(reinterpret_cast<const float4*>(bias + 2 * i) + 1);
                b[0] = u.x, b[1] = u.y, b[2] = u.z, b[3] = u.w, b[4] = v.x, b[5] = v.y, b[6] = v.z, b[7] = v.w;
            }
            __align__(16) T r[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) r[j] = from_f32<T>(scale * clamped_glu(f[2 * j] + b[2 * j], f[2 * j + 1] + b[2 * j + 1], limit, gain, shift));
            if constexpr (sizeof(T) == 2)
                *reinterpret_cast<uint2*>(o + i) = *reinterpret_cast<const uint2*>(r);
            else
                *reinterpret_cast<uint4*>(o + i) = *reinterpret_cast<const uint4*>(r);
        }
        return;
    }
    for (int i = lo + threadIdx.x; i < hi; i += kRowThreads) {
        const float bg = bias ? bias[2 * i] : 0.0f, bu = bias ? bias[2 * i + 1] : 0.0f;
        o[i] = from_f32<T>(scale * clamped_glu(to_f32(g[2 * i]) + bg, to_f32(g[2 * i + 1]) + bu, limit, gain, shift));
    }
}

__global__ void __launch_bounds__(kRowThreads)
softcap_kernel(float* __restrict__ y, size_t n, float cap) {
    llvq_dependent_enter();
    for (size_t i = (size_t)blockIdx.x * kRowThreads + threadIdx.x; i < n; i += (size_t)gridDim.x * kRowThreads) y[i] = cap * tanhf(y[i] / cap);
}

}  // namespace llvq
