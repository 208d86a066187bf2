// Kernels of a real-gated linear recurrent unit (a recurrence with one state number a channel):
//   r_t = sigmoid(zr_t + br), i_t = sigmoid(zi_t + bi), log a_t = lam_c r_t (lam_c < 0, a number a channel),
//   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,   o_t = S_t gelu_tanh(zy_t + by).
// zr and zi come from block-diagonal products of u, zy from a projection; each arrives as the partial
// sums of a split product, [S, rows, width] float32, added in rising order where it is read. All
// arithmetic is float32, 1 - a^2 as -expm1(2 log a), which is exact where a is near 1.
//   - block_product: the block-diagonal product in true 32-bit (the 32-bit path, and blocks whose rows
//     the tensor-core product cannot address),
//   - rglru_step: a thread a (sequence, channel) walks the step's few tokens,
//   - rglru_scan: prompts. A block takes a sequence and 32 channels (a warp's lanes) and works on
//     RG_WARPS x RG_LEN tokens at a time, RG_LEN a warp: a warp folds its tokens into one pair (the
//     product of its a, its state from zero), the pairs meet in shared memory, every warp finds the state
//     its tokens start from by folding the pairs before its own onto the state the tile starts from, and
//     then runs its tokens from registers. The next tile's values are on their way meanwhile.
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

#define RG_WARPS 16
#define RG_LEN 4
#define RG_TILE (RG_WARPS * RG_LEN)
template <typename TO>
__global__ void __launch_bounds__(32 * RG_WARPS)
rglru_scan_kernel(const RgArgs p, TO* __restrict__ out) {
    pdl_trigger();
    pdl_wait();
    __shared__ float sa[2][RG_WARPS][32], sx[2][RG_WARPS][32];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c_raw = blockIdx.x * 32 + lane, b = blockIdx.y;
    const bool live = c_raw < p.C;
    const int c = live ? c_raw : p.C - 1;             // lanes beyond the last channel repeat it and write nothing
    const int t0 = p.cu_q[b], t1 = p.cu_q[b + 1];
    if (t1 <= t0) return;
    const int g = c / p.bs, zc = g * p.pitch + c - g * p.bs;
    float* st = p.state + (size_t)p.seq_slot[b] * p.slot_stride + c;
    const float br = p.br[c], bi = p.bi[c], lam = p.lam[c], by = p.by[c];
    float s = *st;                                    // the state the tile starts from, the same in every warp
    float u[RG_LEN], zr[RG_LEN], zi[RG_LEN], zy[RG_LEN];
    auto fetch = [&](int tile0) {
#pragma unroll
        for (int l = 0; l < RG_LEN; ++l) {
            const int t = tile0 + warp * RG_LEN + l;
            if (t < t1) {
                const float* z = p.z + (size_t)t * p.zW + zc;
                u[l] = p.u[(size_t)t * p.C + c];
                zr[l] = z[0];
                zi[l] = z[p.bs];
                zy[l] = p.y[(size_t)t * p.yW + p.y0 + c];
                for (int k = 1; k < p.zS; ++k) { zr[l] += z[k * p.z_stride]; zi[l] += z[k * p.z_stride + p.bs]; }
                for (int k = 1; k < p.yS; ++k) zy[l] += p.y[k * p.y_stride + (size_t)t * p.yW + p.y0 + c];
            }
        }
    };
    fetch(t0);
    int which = 0;
    for (int tile0 = t0; tile0 < t1; tile0 += RG_TILE, which ^= 1) {
        const int mine = tile0 + warp * RG_LEN;
        float a[RG_LEN], x[RG_LEN], y[RG_LEN];
        float A = 1.0f, X = 0.0f;                     // this warp's tokens folded: S_out = A S_in + X
#pragma unroll
        for (int l = 0; l < RG_LEN; ++l) {
            a[l] = 1.0f, x[l] = 0.0f, y[l] = 0.0f;    // a place behind the last token changes nothing
            if (mine + l < t1) {
                rg_gates(zr[l] + br, zi[l] + bi, lam, u[l], a[l], x[l]);
                y[l] = rg_gelu(zy[l] + by);
            }
            A *= a[l];
            X = fmaf(a[l], X, x[l]);
        }
        sa[which][warp][lane] = A;
        sx[which][warp][lane] = X;
        if (tile0 + RG_TILE < t1) fetch(tile0 + RG_TILE);
        __syncthreads();         // two sets in turn: the set written next was read before this barrier
        float in = s;
#pragma unroll
        for (int w = 0; w < RG_WARPS; ++w) {
            if (w == warp) in = s;
            s = fmaf(sa[which][w][lane], s, sx[which][w][lane]);
        }
#pragma unroll
        for (int l = 0; l < RG_LEN; ++l) {
            in = fmaf(a[l], in, x[l]);
            if (live && mine + l < t1) out[(size_t)(mine + l) * p.C + c] = from_f32<TO>(in * y[l]);
        }
    }
    if (live && warp == 0) *st = s;
}

// A step of n_seqs sequences and N tokens. z [zS, N, zW] with zW >= (C / bs) pitch, pitch >= 2 bs; y
// [yS, N, yW]; state rows updated in place; out [N, C].
#define RG_SCAN_TOKENS 8        // tokens a sequence on average from which the tiled scan takes the step
LUMEN_API int lumen_rglru(const float* u, const float* z, int zS, long long z_stride, int zW, int pitch, int bs,
                          const float* br, const float* bi, const float* lam, const float* y, int yS, long long y_stride,
                          int yW, int y0, const float* by, float* state, long long slot_stride, const int* cu_q,
                          const int* seq_slot, int n_seqs, void* out, int out_is_bf16, int N, int C, cudaStream_t stream) {
    if (N <= 0 || n_seqs <= 0) return 0;
    if (C <= 0 || bs <= 0 || C % bs || pitch < 2 * bs || zW < C / bs * pitch || zS < 1 || yS < 1 || y0 < 0 || y0 + C > yW)
        return LUMEN_ERR_BAD_ARGUMENT;
    if (n_seqs > 65535) return LUMEN_ERR_UNSUPPORTED;
    const RgArgs p = {u, z, zS, (size_t)z_stride, zW, pitch, bs, br, bi, lam, y, yS, (size_t)y_stride, yW, y0, by,
                      state, (size_t)slot_stride, cu_q, seq_slot, C};
    if ((long long)N >= (long long)RG_SCAN_TOKENS * n_seqs) {
        dim3 grid((C + 31) / 32, n_seqs);
        if (out_is_bf16)
            lumen_launch(rglru_scan_kernel<__nv_bfloat16>, grid, dim3(32 * RG_WARPS), 0, stream, p, (__nv_bfloat16*)out);
        else
            lumen_launch(rglru_scan_kernel<float>, grid, dim3(32 * RG_WARPS), 0, stream, p, (float*)out);
    } else {
        dim3 grid((C + 127) / 128, n_seqs);
        if (out_is_bf16) lumen_launch(rglru_step_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p, (__nv_bfloat16*)out);
        else lumen_launch(rglru_step_kernel<float>, grid, dim3(128), 0, stream, p, (float*)out);
    }
    LUMEN_LAUNCH_CHECK();
    return 0;
}
