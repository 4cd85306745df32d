// Short causal convolutions over time and the real-gated linear recurrence behind one (per channel):
//
//   u = conv(x) + bias;  r = sigmoid(Ra u + ra), i = sigmoid(Ri u + ri)  (block-diagonal matrices)
//   log a = -c r softplus(lam);  S <- a S + sqrt(1 - a^2) i u;  out = S gelu(y) * scale
//
// What a sequence carries from token to token lives in two kinds of store, both addressed by position, so that a step
// that is run again at its position changes nothing and no CTA reads what another writes:
//
//   convolution inputs   f32 [taps, channels]: the input of position p in row p % taps. A step reads the rows of the
//                        taps - 1 positions before it and writes its own.
//   recurrent state      f32 [2, ...]: the state before position p in half p % 2; a step reads that half and writes the
//                        other. Position 0 reads zeros whatever is stored, as convolutions do ahead of the first token.
//
//   lru_token            the token step: a CTA takes 32 channels of a block: the block's u, two rows of the gate matrix
//                        per channel, the recurrence, the gate branch.
//   conv_rows_kernel     u of a prompt portion; conv_keep_kernel then stores the inputs the next step reads.
//   lru_scan_kernel      the recurrence of a portion, one pass: a CTA owns 16 channels, a thread 8 tokens at a time in
//                        registers; their products and sums meet in shared memory, 256 tokens a turn.
#pragma once
#include "gqa_attn.cuh"

namespace llvq {

__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

constexpr float kLruDecay = 8.0f;  // c
constexpr int kLruRows = 32;       // channels of a CTA

// Convolution of one channel at position `pos`, whose input's row in the ring of `taps` rows is `row`; x is the token's own
// input.
__device__ __forceinline__ float conv_token(const float* w, int taps, const float* ring, int channels, int ch, long long pos, int row, float x) {
    if (taps == 4 && pos >= 3) {
        const int r1 = (row + 3) & 3, r2 = (row + 2) & 3, r3 = (row + 1) & 3;
        const float x1 = ring[(size_t)r1 * channels + ch], x2 = ring[(size_t)r2 * channels + ch], x3 = ring[(size_t)r3 * channels + ch];
        return fmaf(w[0], x3, fmaf(w[1], x2, fmaf(w[2], x1, w[3] * x)));
    }
    float u = w[taps - 1] * x;
    for (int k = 1; k < taps; ++k) {
        const int r = row - k + (row < k ? taps : 0);
        if (pos >= k) u = fmaf(w[taps - 1 - k], ring[(size_t)r * channels + ch], u);
    }
    return u;
}

struct LruArgs {
    const float* x;       // [width] input of the convolution
    const float* y;       // [width] gate branch before its activation
    const float* conv_w;  // [width, taps]
    const float* conv_b;  // [width]
    const void* w;        // [blocks, 2 n, ldw] of T: the rows of Ra, then those of Ri
    const float* b;       // [blocks, 2 n]
    const float* lam;     // [width]: softplus of the stored value
    const long long* pos;
    float* conv;          // [taps, width]
    float* state;         // [2, width]
    float* out;           // [width]
    int blocks, n, taps, ldw;
    float out_scale;
};

__host__ __device__ inline int lru_tiles(int n) { return (n + kLruRows - 1) / kLruRows; }

// Decays are kept as d = a - 1: a state is carried by s + (d s + x), which loses nothing where a rounds to a value near
// one and a sequence is long. 1 - a^2 = -d (2 + d).
__device__ __forceinline__ float lru_decay(float r, float lam) { return expm1f(-kLruDecay * r * lam); }
__device__ __forceinline__ float lru_input(float d, float i, float u) { return sqrtf(-d * (2.0f + d)) * i * u; }
__device__ __forceinline__ float carry(float d, float s, float x) { return s + fmaf(d, s, x); }

// One CTA's part; `smem` holds ldw floats. Calls the dependency wait itself, behind its first loads of the matrices.
template <typename T>
__device__ __forceinline__ void lru_token(const LruArgs& A, int cta, float* u_s) {
    constexpr int VN = Vec16<T>::N;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int tiles = lru_tiles(A.n), blk = cta / tiles, c0 = (cta - blk * tiles) * kLruRows + warp * 4;  // this warp's first channel of the block
    const int vecs = A.ldw / VN, width = A.blocks * A.n;
    const uint4* W = reinterpret_cast<const uint4*>(A.w) + (size_t)blk * 2 * A.n * vecs;
    auto row = [&](int k) { return W + (size_t)((k >> 2) * A.n + min(c0 + (k & 3), A.n - 1)) * vecs; };  // k: 4 rows of Ra, 4 of Ri
    uint4 ahead[8];
    if (c0 < A.n && lane < vecs) {
#pragma unroll
        for (int k = 0; k < 8; ++k) ahead[k] = __ldg(row(k) + lane);
    }
    llvq_dependent_enter();
    const long long pos = *A.pos;
    const int conv_row = (int)((unsigned int)pos % (unsigned int)A.taps);
    for (int c = tid; c < A.ldw; c += 256) {
        const int ch = blk * A.n + c;
        u_s[c] = c < A.n ? A.conv_b[ch] + conv_token(A.conv_w + (size_t)ch * A.taps, A.taps, A.conv, width, ch, pos, conv_row, A.x[ch]) : 0.0f;
    }
    __syncthreads();
    if (c0 >= A.n) return;
    float acc[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) acc[k] = 0.0f;
    for (int v = lane; v < vecs; v += 32) {
        if (v != lane) {
#pragma unroll
            for (int k = 0; k < 8; ++k) ahead[k] = __ldg(row(k) + v);
        }
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            float f[VN];
            Vec16<T>::widen(ahead[k], f);
#pragma unroll
            for (int j = 0; j < VN; ++j) acc[k] = fmaf(f[j], u_s[v * VN + j], acc[k]);
        }
    }
    float zr = 0.0f, zi = 0.0f;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
        const float s = warp_sum_f(acc[k]);
        if (lane == (k & 3)) (k < 4 ? zr : zi) = s;
    }
    const int c = c0 + lane, ch = blk * A.n + c;
    if (lane < 4 && c < A.n) {
        const float r = sigmoid_f(zr + A.b[(size_t)blk * 2 * A.n + c]), i = sigmoid_f(zi + A.b[(size_t)blk * 2 * A.n + A.n + c]);
        const float s = pos > 0 ? A.state[(size_t)(pos & 1) * width + ch] : 0.0f;
        const float d = lru_decay(r, A.lam[ch]), t = carry(d, s, lru_input(d, i, u_s[c]));
        A.state[(size_t)((pos + 1) & 1) * width + ch] = t;
        A.conv[(size_t)conv_row * width + ch] = A.x[ch];
        A.out[ch] = t * gelu_tanh_f(A.y[ch]) * A.out_scale;
    }
}

// Attention and recurrence that read the same token, side by side in one launch: the first `attn_ctas` CTAs are the attention's.
template <typename T>
__global__ void __launch_bounds__(256)
mixer_token_kernel(GqaArgs A, int attn_ctas, LruArgs R) {
    extern __shared__ __align__(16) unsigned char mt_smem[];
    if ((int)blockIdx.x < attn_ctas) {
        llvq_dependent_enter();
        gqa_token<T>(A, blockIdx.x, mt_smem);
    } else {
        lru_token<T>(R, blockIdx.x - attn_ctas, reinterpret_cast<float*>(mt_smem));
    }
}

// ---- prompt portions ----

// Input of channel c at place t of a portion that starts at pos0 (t may be negative), as f32; xb: the channel's input bias.
template <typename T>
__device__ __forceinline__ float conv_input(const T* x, int ldx, float xb, const float* ring, int channels, int taps, long long pos0, int t, int c) {
    if (t >= 0) return to_f32(x[(size_t)t * ldx + c]) + xb;
    const long long p = pos0 + t;
    return p >= 0 ? ring[(size_t)(p % taps) * channels + c] : 0.0f;
}

constexpr int kConvRun = 16;  // tokens of a thread

// grid = (ceil(channels / 256), ceil(n / 16)): a thread slides along 16 tokens of one channel.
template <typename T>
__global__ void __launch_bounds__(256)
conv_rows_kernel(const T* __restrict__ x, int ldx, const float* __restrict__ x_bias, const float* __restrict__ w, const float* __restrict__ bias, const float* __restrict__ ring,
                 T* __restrict__ out, int channels, int taps, long long pos0, int n) {
    llvq_dependent_enter();
    const int c = blockIdx.x * 256 + threadIdx.x, t0 = blockIdx.y * kConvRun, t1 = min(n, t0 + kConvRun);
    if (c >= channels) return;
    const float b = bias ? bias[c] : 0.0f, xb = x_bias ? x_bias[c] : 0.0f;
    const float* wc = w + (size_t)c * taps;
    if (taps == 4) {
        const float w0 = wc[0], w1 = wc[1], w2 = wc[2], w3 = wc[3];
        float x3 = conv_input(x, ldx, xb, ring, channels, 4, pos0, t0 - 3, c), x2 = conv_input(x, ldx, xb, ring, channels, 4, pos0, t0 - 2, c),
              x1 = conv_input(x, ldx, xb, ring, channels, 4, pos0, t0 - 1, c);
        float in[kConvRun];
#pragma unroll
        for (int k = 0; k < kConvRun; ++k) in[k] = t0 + k < t1 ? to_f32(x[(size_t)(t0 + k) * ldx + c]) + xb : 0.0f;
#pragma unroll
        for (int k = 0; k < kConvRun; ++k) {
            if (t0 + k < t1) out[(size_t)(t0 + k) * channels + c] = from_f32<T>(fmaf(w0, x3, fmaf(w1, x2, fmaf(w2, x1, fmaf(w3, in[k], b)))));
            x3 = x2, x2 = x1, x1 = in[k];
        }
        return;
    }
    for (int t = t0; t < t1; ++t) {
        float u = b;
        for (int k = 0; k < taps; ++k) u = fmaf(wc[taps - 1 - k], conv_input(x, ldx, xb, ring, channels, taps, pos0, t - k, c), u);
        out[(size_t)t * channels + c] = from_f32<T>(u);
    }
}

// The last taps inputs of the portion into the ring. Runs behind the kernels that read it.
template <typename T>
__global__ void __launch_bounds__(256)
conv_keep_kernel(const T* __restrict__ x, int ldx, const float* __restrict__ x_bias, float* __restrict__ ring, int channels, int taps, long long pos0, int n) {
    llvq_dependent_enter();
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c >= channels) return;
    for (int t = max(0, n - taps); t < n; ++t) ring[(size_t)((pos0 + t) % taps) * channels + c] = to_f32(x[(size_t)t * ldx + c]) + (x_bias ? x_bias[c] : 0.0f);
}

struct LruScanArgs {
    const void* u;       // [n_tok, width] of T
    const float* z;      // [blocks, n_tok, 2 n]: Ra u, then Ri u, without their biases
    const float* b;      // [blocks, 2 n]
    const float* lam;    // [width]: softplus of the stored value
    const void* y;       // [n_tok, ldy] of T
    const float* y_bias; // [width]
    float* state;        // [2, width]
    void* out;           // [n_tok, ldo] of T
    long long pos0;
    int n_tok, blocks, n, ldy, ldo;
    float out_scale;
};

constexpr int kScanTok = 8, kScanWarps = 16, kScanCh = 16, kScanTurn = 2 * kScanTok * kScanWarps;

template <typename T>
__device__ __forceinline__ float gelu_tanh_t(float z) {
    if constexpr (sizeof(T) == 2) return z * sigmoid_t<T>(1.5957691216057308f * (z + 0.044715f * z * z * z));
    return gelu_tanh_f(z);
}

// grid = ceil(width / 16), 512 threads: a warp's halves take 16 channels over 8 tokens each, a turn is 256 tokens.
template <typename T>
__global__ void __launch_bounds__(kScanWarps * 32, 2)
lru_scan_kernel(LruScanArgs A) {
    __shared__ float2 part_s[2][kScanWarps][kScanCh];  // decay product and sum of a warp's 16 tokens; two turns' worth
    llvq_dependent_enter();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, width = A.blocks * A.n, lc = lane & (kScanCh - 1), upper = lane / kScanCh;
    const int ch = blockIdx.x * kScanCh + lc, cc = min(ch, width - 1), blk = cc / A.n, c = cc - blk * A.n;
    const float br = A.b[(size_t)blk * 2 * A.n + c], bi = A.b[(size_t)blk * 2 * A.n + A.n + c], lam = A.lam[cc], yb = A.y_bias[cc];
    const float* z = A.z + (size_t)blk * A.n_tok * 2 * A.n + c;
    const T* U = reinterpret_cast<const T*>(A.u) + cc;
    const T* Y = reinterpret_cast<const T*>(A.y) + cc;
    T* O = reinterpret_cast<T*>(A.out) + cc;
    float state = A.pos0 > 0 ? A.state[(size_t)(A.pos0 & 1) * width + cc] : 0.0f;  // before the turn, the same in every thread of a channel
    for (int t0 = 0, turn = 0; t0 < A.n_tok; t0 += kScanTurn, ++turn) {
        const int tw = t0 + (2 * warp + upper) * kScanTok;
        float a[kScanTok], x[kScanTok], u[kScanTok], y[kScanTok];
#pragma unroll
        for (int k = 0; k < kScanTok; ++k) {
            const int t = min(tw + k, A.n_tok - 1);
            a[k] = z[(size_t)t * 2 * A.n];
            x[k] = z[(size_t)t * 2 * A.n + A.n];
            u[k] = to_f32(U[(size_t)t * width]);
            y[k] = to_f32(Y[(size_t)t * A.ldy]);
        }
        float prod = 1.0f, sum = 0.0f;  // a[] holds decays less one from here on
#pragma unroll
        for (int k = 0; k < kScanTok; ++k) {
            const bool in = tw + k < A.n_tok;
            a[k] = in ? lru_decay(sigmoid_f(a[k] + br), lam) : 0.0f;
            x[k] = in ? lru_input(a[k], sigmoid_t<T>(x[k] + bi), u[k]) : 0.0f;
            y[k] = gelu_tanh_t<T>(y[k] + yb) * A.out_scale;
            prod = carry(a[k], prod, 0.0f);
            sum = carry(a[k], sum, x[k]);
        }
        // the lower half's tokens come first
        const float lp = __shfl_sync(0xffffffffu, prod, lc), ls = __shfl_sync(0xffffffffu, sum, lc);
        if (upper) part_s[turn & 1][warp][lc] = make_float2(prod * lp, fmaf(prod, ls, sum));
        __syncthreads();
        float s = state, all = state;
#pragma unroll
        for (int w = 0; w < kScanWarps; ++w) {
            const float2 p = part_s[turn & 1][w][lc];
            all = fmaf(p.x, all, p.y);
            if (w + 1 == warp) s = all;
        }
        state = all;
        if (upper) s = fmaf(lp, s, ls);
#pragma unroll
        for (int k = 0; k < kScanTok; ++k) {
            s = carry(a[k], s, x[k]);
            if (tw + k < A.n_tok && ch < width) O[(size_t)(tw + k) * A.ldo] = from_f32<T>(s * y[k]);
        }
    }
    if (warp == 0 && !upper && ch < width) A.state[(size_t)((A.pos0 + A.n_tok) & 1) * width + ch] = state;
}

}  // namespace llvq
