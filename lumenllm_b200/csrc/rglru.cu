// Kernels of a real-gated linear recurrent unit (a recurrence with one state number a channel):
//   r_t = sigmoid(zr_t + br), i_t = sigmoid(zi_t + bi), log a_t = lam_c r_t (lam_c < 0, a number a channel),
//   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,   o_t = S_t gelu_tanh(zy_t + by).
// zr and zi come from block-diagonal products of u, zy from a projection; each arrives as the partial
// sums of a split product, [S, rows, width] float32, added in rising order where it is read. All
// arithmetic is float32, 1 - a^2 as -expm1(2 log a), which is exact where a is near 1.
//   - block_product: the block-diagonal product in true 32-bit (the 32-bit path, and blocks whose rows
//     the tensor-core product cannot address),
//   - rglru_step: a thread a (sequence, channel) walks the step's few tokens,
//   - rglru_fold and rglru_run: prompts, in chunks side by side (below).
#include "common.cuh"

__device__ __forceinline__ float rg_parts(const float* p, int S, size_t stride) {
    float x = p[0];
    for (int s = 1; s < S; ++s) x += p[(size_t)s * stride];
    return x;
}
__device__ __forceinline__ float rg_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float rg_gelu(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// ---------------------------------------------------------------- block-diagonal product, 32-bit
// out[n, g rows + j] = sum_k x[n, g K + k] w[g rows + j, k] for blocks g < G, j < rows, k < K: x float32
// [N, G K], w [G rows, K] float32 or bfloat16. A block of 256 threads makes a 64 x 64 piece of one g.
#define BP_T 64
#define BP_K 16
template <typename TW>
__global__ void __launch_bounds__(256)
block_product_kernel(const float* __restrict__ x, const TW* __restrict__ w, float* __restrict__ out, int N, int G, int rows,
                     int K) {
    pdl_trigger();
    pdl_wait();
    __shared__ float xs[BP_K][BP_T + 4], ws[BP_K][BP_T + 4];
    const int n0 = blockIdx.x * BP_T, j0 = blockIdx.y * BP_T, g = blockIdx.z, tid = threadIdx.x;
    const int ty = tid >> 4, tx = tid & 15;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += BP_K) {
        for (int i = tid; i < BP_T * BP_K; i += 256) {
            const int r = i / BP_K, k = i - r * BP_K;
            const bool kin = k0 + k < K;
            xs[k][r] = (kin && n0 + r < N) ? x[(size_t)(n0 + r) * G * K + (size_t)g * K + k0 + k] : 0.0f;
            ws[k][r] = (kin && j0 + r < rows) ? to_f32(w[((size_t)g * rows + j0 + r) * K + k0 + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BP_K; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = xs[k][4 * ty + i]; b[i] = ws[k][4 * tx + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + 4 * ty + i, jj = j0 + 4 * tx + j;
            if (n < N && jj < rows) out[(size_t)n * G * rows + (size_t)g * rows + jj] = acc[i][j];
        }
}

LUMEN_API int lumen_block_product(const float* x, const void* w, int w_is_bf16, float* out, int N, int G, int rows, int K,
                                  cudaStream_t stream) {
    if (N <= 0) return 0;
    if (G <= 0 || rows <= 0 || K <= 0) return LUMEN_ERR_BAD_ARGUMENT;
    dim3 grid((N + BP_T - 1) / BP_T, (rows + BP_T - 1) / BP_T, G);
    if (grid.y > 65535 || grid.z > 65535) return LUMEN_ERR_UNSUPPORTED;
    if (w_is_bf16)
        lumen_launch(block_product_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, x, (const __nv_bfloat16*)w, out, N, G,
                     rows, K);
    else
        lumen_launch(block_product_kernel<float>, grid, dim3(256), 0, stream, x, (const float*)w, out, N, G, rows, K);
    LUMEN_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------- the recurrence
struct RgArgs {
    const float* u;           // [N, C]
    const float* z;           // gate sums [zS][N][zW]: channel c = block g, place j: zr at g pitch + j, zi at g pitch + bs + j
    int zS;
    size_t z_stride;
    int zW, pitch, bs;
    const float* br;
    const float* bi;          // [C]
    const float* lam;         // [C]: log a = lam r
    const float* y;           // projection sums [yS][N][yW], columns y0 + c
    int yS;
    size_t y_stride;
    int yW, y0;
    const float* by;          // [C]
    float* state;             // row seq_slot[b], slot_stride floats apart: [C]
    size_t slot_stride;
    const int* cu_q;
    const int* seq_slot;
    int C;
};

// decay and input of one token from its raw sums
__device__ __forceinline__ void rg_gates(float zr, float zi, float lam, float u, float& a, float& x) {
    const float la = lam * rg_sigmoid(zr);
    a = expf(la);
    x = sqrtf(-expm1f(2.0f * la)) * rg_sigmoid(zi) * u;
}

template <typename TO>
__global__ void __launch_bounds__(128)
rglru_step_kernel(const RgArgs p, TO* __restrict__ out) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
    if (c >= p.C) return;
    const int t0 = p.cu_q[b], t1 = p.cu_q[b + 1];
    if (t1 <= t0) return;
    const int g = c / p.bs, zc = g * p.pitch + c - g * p.bs;
    float* st = p.state + (size_t)p.seq_slot[b] * p.slot_stride + c;
    const float br = p.br[c], bi = p.bi[c], lam = p.lam[c], by = p.by[c];
    float s = *st;
    for (int t = t0; t < t1; ++t) {
        const float* z = p.z + (size_t)t * p.zW + zc;
        const float zr = rg_parts(z, p.zS, p.z_stride) + br, zi = rg_parts(z + p.bs, p.zS, p.z_stride) + bi;
        const float zy = rg_parts(p.y + (size_t)t * p.yW + p.y0 + c, p.yS, p.y_stride) + by;
        float a, x;
        rg_gates(zr, zi, lam, p.u[(size_t)t * p.C + c], a, x);
        s = fmaf(a, s, x);
        out[(size_t)t * p.C + c] = from_f32<TO>(s * rg_gelu(zy));
    }
    *st = s;
}

// Prompts, in chunks of RG_CHUNK tokens of a sequence. First kernel: a thread a (chunk, channel) makes its
// tokens' decays and inputs (they go over the gates' first partial sums, which nobody else reads: decay in
// zr's place, input in zi's) and folds them into one pair: S_out = A S_in + X. A sequence's first chunk folds
// the state in (A 0). Second kernel: a thread a (chunk, channel) folds the pairs of the chunks before its
// own, which gives the state its tokens start from, and runs them; a sequence's last chunk leaves the state.
#define RG_CHUNK 64
#define RG_RUN 8               // tokens whose loads go out together
struct RgChunks {
    float* pairs;              // [chunks][3][C]: A, X and, for a sequence's first chunk, the state before it
    float* z;                  // the gates' sums, to be written over
    int n_seqs;
};
__device__ __forceinline__ bool rg_chunk(const int* cu_q, int n_seqs, int z, int& b, int& i, int& t0, int& t1, bool& last) {
    i = z;
    for (b = 0; b < n_seqs; ++b) {
        const int first = cu_q[b], q = cu_q[b + 1] - first, nc = (q + RG_CHUNK - 1) / RG_CHUNK;
        if (i < nc) {
            t0 = first + i * RG_CHUNK;
            t1 = min(t0 + RG_CHUNK, first + q);
            last = i == nc - 1;
            return true;
        }
        i -= nc;
    }
    return false;
}

__global__ void __launch_bounds__(128)
rglru_fold_kernel(const RgArgs p, const RgChunks ch) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * 128 + threadIdx.x;
    int b, i, t0, t1;
    bool last;
    if (c >= p.C || !rg_chunk(p.cu_q, ch.n_seqs, blockIdx.y, b, i, t0, t1, last)) return;
    const int g = c / p.bs, zc = g * p.pitch + c - g * p.bs;
    const float br = p.br[c], bi = p.bi[c], lam = p.lam[c];
    float* pair = ch.pairs + (size_t)blockIdx.y * 3 * p.C + c;
    float A = 1.0f, X = 0.0f;
    if (i == 0) {
        A = 0.0f;
        X = p.state[(size_t)p.seq_slot[b] * p.slot_stride + c];
        pair[2 * p.C] = X;
    }
    for (int r0 = t0; r0 < t1; r0 += RG_RUN) {
        float zr[RG_RUN], zi[RG_RUN], u[RG_RUN];
#pragma unroll
        for (int l = 0; l < RG_RUN; ++l)
            if (r0 + l < t1) {
                const float* z = p.z + (size_t)(r0 + l) * p.zW + zc;
                zr[l] = z[0];
                zi[l] = z[p.bs];
                for (int k = 1; k < p.zS; ++k) { zr[l] += z[k * p.z_stride]; zi[l] += z[k * p.z_stride + p.bs]; }
                u[l] = p.u[(size_t)(r0 + l) * p.C + c];
            }
#pragma unroll
        for (int l = 0; l < RG_RUN; ++l)
            if (r0 + l < t1) {
                float a, x;
                rg_gates(zr[l] + br, zi[l] + bi, lam, u[l], a, x);
                float* z = ch.z + (size_t)(r0 + l) * p.zW + zc;
                z[0] = a;
                z[p.bs] = x;
                A *= a;
                X = fmaf(a, X, x);
            }
    }
    pair[0] = A;
    pair[p.C] = X;
}

template <typename TO>
__global__ void __launch_bounds__(128)
rglru_run_kernel(const RgArgs p, const RgChunks ch, TO* __restrict__ out) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * 128 + threadIdx.x;
    int b, i, t0, t1;
    bool last;
    if (c >= p.C || !rg_chunk(p.cu_q, ch.n_seqs, blockIdx.y, b, i, t0, t1, last)) return;
    const int g = c / p.bs, zc = g * p.pitch + c - g * p.bs;
    const float by = p.by[c];
    const float* pair = ch.pairs + (size_t)(blockIdx.y - i) * 3 * p.C + c;
    float s = i == 0 ? pair[2 * p.C] : 0.0f;
    for (int k0 = 0; k0 < i; k0 += RG_RUN) {               // the first pair brings the state along
        float A[RG_RUN], X[RG_RUN];
#pragma unroll
        for (int k = 0; k < RG_RUN; ++k)
            if (k0 + k < i) {
                A[k] = pair[(size_t)(k0 + k) * 3 * p.C];
                X[k] = pair[(size_t)(k0 + k) * 3 * p.C + p.C];
            }
#pragma unroll
        for (int k = 0; k < RG_RUN; ++k)
            if (k0 + k < i) s = fmaf(A[k], s, X[k]);
    }
    for (int r0 = t0; r0 < t1; r0 += RG_RUN) {
        float a[RG_RUN], x[RG_RUN], y[RG_RUN];
#pragma unroll
        for (int l = 0; l < RG_RUN; ++l)
            if (r0 + l < t1) {
                const float* z = ch.z + (size_t)(r0 + l) * p.zW + zc;
                a[l] = z[0];
                x[l] = z[p.bs];
                const float* yy = p.y + (size_t)(r0 + l) * p.yW + p.y0 + c;
                y[l] = yy[0];
                for (int k = 1; k < p.yS; ++k) y[l] += yy[k * p.y_stride];
            }
#pragma unroll
        for (int l = 0; l < RG_RUN; ++l)
            if (r0 + l < t1) {
                s = fmaf(a[l], s, x[l]);
                out[(size_t)(r0 + l) * p.C + c] = from_f32<TO>(s * rg_gelu(y[l] + by));
            }
    }
    if (last) p.state[(size_t)p.seq_slot[b] * p.slot_stride + c] = s;      // nobody reads it in this kernel
}
// A step of n_seqs sequences and N tokens. z [zS, N, zW] (prompts overwrite its first part) with zW >= (C / bs) pitch, pitch >= 2 bs; y
// [yS, N, yW]; state rows updated in place; out [N, C].
#define RG_SCAN_TOKENS 8        // tokens a sequence on average from which a step is worked on in chunks
// Chunks of such a step (the scratch `pairs` then holds 3 C numbers for each); 0: no scratch is needed.
LUMEN_API int lumen_rglru_chunks(int N, int n_seqs) {
    return n_seqs > 0 && (long long)N >= (long long)RG_SCAN_TOKENS * n_seqs ? N / RG_CHUNK + n_seqs : 0;
}
LUMEN_API int lumen_rglru(const float* u, float* z, int zS, long long z_stride, int zW, int pitch, int bs,
                          const float* br, const float* bi, const float* lam, const float* y, int yS, long long y_stride,
                          int yW, int y0, const float* by, float* state, long long slot_stride, const int* cu_q,
                          const int* seq_slot, int n_seqs, void* out, int out_is_bf16, int N, int C, float* pairs,
                          cudaStream_t stream) {
    if (N <= 0 || n_seqs <= 0) return 0;
    if (C <= 0 || bs <= 0 || C % bs || pitch < 2 * bs || zW < C / bs * pitch || zS < 1 || yS < 1 || y0 < 0 || y0 + C > yW)
        return LUMEN_ERR_BAD_ARGUMENT;
    if (n_seqs > 65535) return LUMEN_ERR_UNSUPPORTED;
    const RgArgs p = {u, z, zS, (size_t)z_stride, zW, pitch, bs, br, bi, lam, y, yS, (size_t)y_stride, yW, y0, by,
                      state, (size_t)slot_stride, cu_q, seq_slot, C};
    const int chunks = lumen_rglru_chunks(N, n_seqs);
    if (chunks) {
        if (!pairs || chunks > 65535) return LUMEN_ERR_BAD_ARGUMENT;
        const RgChunks ch = {pairs, z, n_seqs};
        dim3 grid((C + 127) / 128, chunks);
        lumen_launch(rglru_fold_kernel, grid, dim3(128), 0, stream, p, ch);
        LUMEN_LAUNCH_CHECK();
        if (out_is_bf16)
            lumen_launch(rglru_run_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p, ch, (__nv_bfloat16*)out);
        else
            lumen_launch(rglru_run_kernel<float>, grid, dim3(128), 0, stream, p, ch, (float*)out);
    } else {
        dim3 grid((C + 127) / 128, n_seqs);
        if (out_is_bf16) lumen_launch(rglru_step_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p, (__nv_bfloat16*)out);
        else lumen_launch(rglru_step_kernel<float>, grid, dim3(128), 0, stream, p, (float*)out);
    }
    LUMEN_LAUNCH_CHECK();
    return 0;
}
