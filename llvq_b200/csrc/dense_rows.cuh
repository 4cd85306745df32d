// Row kernels of a prompt portion on the dense-weight path: one CTA per token, f32 arithmetic, T activations.
//
//   embed_rows_kernel   x = scale * table[token], and its T copy for the first projections
//   postnorm_rows_kernel  t = alpha * x + y (+ bias); x = t / sqrt(mean(t^2) + eps) * w, and its T copy
//   latent_rows_kernel  the down projections of a latent-attention layer: the query latent normed into cq, the
//                       token's cache row normed, rotated and stored into the ring
//   glu_rows_kernel     clamped gated unit of [gate | up] with their biases
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

// Dynamic shared memory: n floats. out may be x: a CTA has read its row before it writes; y may be null (alpha = 1: a plain norm).
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
postnorm_rows_kernel(const float* x, const T* __restrict__ y, const float* __restrict__ bias, const float* __restrict__ w,
                     float alpha, float eps, T* __restrict__ xt, float* out, int n) {
    extern __shared__ __align__(16) float row_s[];
    __shared__ float red[kRowThreads / 32];
    llvq_dependent_enter();
    const size_t o = (size_t)blockIdx.x * n;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < n; i += kRowThreads) {
        float t = alpha * x[o + i];
        if (y) t += to_f32(y[o + i]) + (bias ? bias[i] : 0.0f);
        row_s[i] = t;
        ss = fmaf(t, t, ss);
    }
    const float r = 1.0f / sqrtf(block_sum_f(ss, red) / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += kRowThreads) {
        const float v = row_s[i] * r * w[i];
        if (out) out[o + i] = v;
        if (xt) xt[o + i] = from_f32<T>(v);
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

template <typename T>
__global__ void __launch_bounds__(kRowThreads)
glu_rows_kernel(const T* __restrict__ gu, const float* __restrict__ bias, T* __restrict__ out, int n, float limit, float gain, float shift) {
    llvq_dependent_enter();
    const T* g = gu + (size_t)blockIdx.x * 2 * n;
    for (int i = threadIdx.x + blockIdx.y * kRowThreads; i < n; i += kRowThreads * gridDim.y) {
        const float bg = bias ? bias[i] : 0.0f, bu = bias ? bias[n + i] : 0.0f;
        out[(size_t)blockIdx.x * n + i] = from_f32<T>(clamped_glu(to_f32(g[i]) + bg, to_f32(g[n + i]) + bu, limit, gain, shift));
    }
}

__global__ void __launch_bounds__(kRowThreads)
softcap_kernel(float* __restrict__ y, size_t n, float cap) {
    llvq_dependent_enter();
    for (size_t i = (size_t)blockIdx.x * kRowThreads + threadIdx.x; i < n; i += (size_t)gridDim.x * kRowThreads) y[i] = cap * tanhf(y[i] / cap);
}

}  // namespace llvq
