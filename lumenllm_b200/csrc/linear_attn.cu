// Linear attention with decay: a recurrence over time with a matrix state per head,
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T  (S is d x dv),   o_t = o_scale S_t^T q_t,
// the token's own write seen by its own read; the decay is one fixed number a head (a_t = decay_h), or
// (CH) comes with every token, one number a (head, key channel), as float32 rows alpha [N, H d]. q, k (H
// heads of d) and v (H heads of dv) are columns of a projection that arrives as the S partial sums of a
// split product, [S, N, W] float32, added in rising order where a value is read; with `act` 1 each value
// goes through SiLU first. State, decay, sums and outputs are float32 whatever the run's type.
//
// With `bonus` float32 [N, H] (PRE, with decays that come with the tokens) a token reads the state BEFORE its
// own write and adds its own value with a weight of its own, o_t = o_scale (S_(t-1)^T q_t) + bonus_t v_t:
// what a bonus u for the current token comes to, bonus_t = sum_j q_j u_j k_j (made by low_rank_decay_kernel's
// second kind of blocks, once for all the columns that share it).
//
// A block takes one sequence, one head and a few columns of the state and walks the sequence's
// tokens of this step in order, the state in registers: a warp's lanes are PARTS parts x 32 / PARTS
// columns, part p holding rows p JPT .. p JPT + JPT of its column (d <= PARTS JPT; rows beyond d
// are zeros and stay zeros). The tokens' q, k and v come through shared memory in runs of LA_RUN
// tokens, staged by the whole block; the lanes of a part read the same q and k words, so a 16-byte
// shared load serves them in one go. An output is the sum of its column's parts, a few shuffles. Every
// number depends on its own sequence only, up to rounding whatever the step's division into tokens.
//
// Two ways in. Steps of few tokens a sequence (decoding) read the projection's partial sums and apply
// the activation while they stage a run. Prompts first go through linear_attn_prep_kernel, which adds
// the partial sums and applies the activation ONCE for all blocks of a head (they share q and k) into
// a dense float32 buffer (a projection that is one sum and has no activation to apply is read as it is);
// the walk then fetches run r + 1 with 16-byte asynchronous copies into a
// second set of shared rows while it walks run r, and a lane holds several columns (below).
//
// Long prompts of few sequences are walked in chunks of LA_CHUNK tokens side by side, because one walk
// would leave most of the device idle: a fold of every chunk (its state from zero, without outputs), a
// small kernel that carries the states from chunk to chunk (start_(i+1) = prod(a of chunk i) start_i +
// fold_i), and the walk of every chunk from its own start. Half the work more, in as many blocks as there
// are chunks. A chunk is a run of a sequence's tokens of this step, so a token's result still depends on
// its own sequence alone, up to rounding.
//
// The sums of a token run two rows a lane and instruction (fma.rn.f32x2, the packed form of fma.rn.f32).
#include "common.cuh"

#define LA_RUN 16
#define LA_FIXED 0       // MODE of a walk: a fixed decay a head,
#define LA_CHANNEL 1     // a decay a token and key channel,
#define LA_BONUS 2       // the same, the state read before the token's write and a bonus for its own value
#define LA_GROUP 8
#define LA_THREADS 128

__device__ __forceinline__ float la_parts_sum(const float* p, int S, size_t stride) {
    float x = p[0];
    for (int s0 = 1; s0 < S; s0 += 4) {           // four loads in flight, added in rising order
        float q[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) q[j] = s0 + j < S ? p[(size_t)(s0 + j) * stride] : 0.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (s0 + j < S) x += q[j];
    }
    return x;
}
__device__ __forceinline__ float la_act(float x, int act) { return act ? x / (1.0f + expf(-x)) : x; }

// dense[n, c] = act(sum of the partial sums of u[n, c0 + c]) for the Wd columns of q, k and v.
__global__ void __launch_bounds__(256)
linear_attn_prep_kernel(const float* __restrict__ u, int S, size_t split_stride, int W, int q_col, int k_col, int v_col,
                        int Hd, int Hdv, int act, float* __restrict__ dense, long long total) {
    // No early trigger here: the walk that follows has fewer blocks than there are SMs and must find the
    // SMs empty, so that its blocks are spread one an SM; started under this kernel's blocks they are
    // packed several an SM wherever room is, and the walk takes twice as long (858 against 460 us for a
    // prompt of 2,048 tokens at 16 heads of 128 x 128).
    pdl_wait();
    const int Wd = 2 * Hd + Hdv;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long n = i / Wd;
        const int c = (int)(i - n * Wd);
        const int src = c < Hd ? q_col + c : (c < 2 * Hd ? k_col + c - Hd : v_col + c - 2 * Hd);
        dense[i] = la_act(la_parts_sum(u + n * W + src, S, split_stride), act);
    }
}

__device__ __forceinline__ void la_cp16(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 f2_pack(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void f2_unpack(f32x2 v, float& lo, float& hi) {
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ f32x2 f2_mul(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ f32x2 f2_fma(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

#define LA_CHUNK 128
// Chunk z of the step: its sequence b, its number i in the sequence and its tokens; false: there are fewer.
__device__ __forceinline__ bool la_chunk(const int* cu_q, int n_seqs, int z, int& b, int& i, int& t0, int& t1, bool& last) {
    i = z;
    for (b = 0; b < n_seqs; ++b) {
        const int first = cu_q[b], q = cu_q[b + 1] - first, nc = (q + LA_CHUNK - 1) / LA_CHUNK;
        if (i < nc) {
            t0 = first + i * LA_CHUNK;
            t1 = min(t0 + LA_CHUNK, first + q);
            last = i == nc - 1;
            return true;
        }
        i -= nc;
    }
    return false;
}

// Steps of few tokens a sequence: PARTS lanes share a column (d <= PARTS JPT), a warp holds CW = 32 / PARTS
// columns, a block 4 CW; the block stages the tokens' q, k and v (and, CH, decays) itself.
template <int JPT, int PARTS, int MODE>
__global__ void __launch_bounds__(LA_THREADS)
linear_attn_kernel(const float* __restrict__ u, int S, size_t split_stride, int W, int q_col, int k_col, int v_col,
                   int act, const float* __restrict__ decay, float* __restrict__ state, size_t slot_stride,
                   const int* __restrict__ cu_q, const int* __restrict__ seq_slot, float* __restrict__ out, int H, int d,
                   int dv, const float* __restrict__ alpha, const float* __restrict__ bonus, float o_scale) {
    constexpr bool CH = MODE != LA_FIXED, PRE = MODE == LA_BONUS;
    constexpr int CW = 32 / PARTS, COLS = 4 * CW;   // columns a warp and a block
    constexpr int SEG = JPT + (JPT == 4 ? 0 : 4), DR = PARTS * SEG;  // a part's segment and a token's row of q (or k)
    constexpr int ROWS = CH ? 3 : 2;
    // q [LA_RUN][DR], k [LA_RUN][DR], (decays [LA_RUN][DR],) v [LA_RUN][COLS]
    extern __shared__ __align__(16) float sm[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int part = lane / CW, e_local = lane % CW;
    const int e0 = blockIdx.x * COLS, h = blockIdx.y, b = blockIdx.z;
    const int e = e0 + warp * CW + e_local;
    const float a = CH ? 0.0f : decay[h];
    pdl_trigger();
    pdl_wait();
    const int t0 = cu_q[b], t1 = cu_q[b + 1];
    if (t1 <= t0) return;
    float* Sg = state + (size_t)seq_slot[b] * slot_stride + (size_t)h * d * dv;
    f32x2 st[JPT / 2];
#pragma unroll
    for (int i = 0; i < JPT; i += 2) {
        const int j = part * JPT + i;
        st[i / 2] = f2_pack((j < d && e < dv) ? Sg[(size_t)j * dv + e] : 0.0f,
                            (j + 1 < d && e < dv) ? Sg[(size_t)(j + 1) * dv + e] : 0.0f);
    }
    const f32x2 aa = f2_pack(a, a);
    // one token: the state moves on; what comes back is this part's share of the column's output
    auto token = [&](const float* qs, const float* ks, const float* vs, int t) -> float {
        const f32x2 v = f2_pack(vs[t * COLS], vs[t * COLS]);
        const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(qs + t * DR);
        const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(ks + t * DR);
        const ulonglong2* a4 = reinterpret_cast<const ulonglong2*>(ks + LA_RUN * DR + t * DR);   // CH only: behind k's rows
        f32x2 o01 = f2_pack(0.0f, 0.0f), o23 = o01;
#pragma unroll
        for (int i = 0; i < JPT / 4; ++i) {
            const ulonglong2 k = k4[i];
            ulonglong2 g = make_ulonglong2(aa, aa);
            if (CH) g = a4[i];
            const ulonglong2 q = q4[i];
            if (PRE) {
                o01 = f2_fma(st[2 * i], q.x, o01);
                o23 = f2_fma(st[2 * i + 1], q.y, o23);
            }
            st[2 * i] = f2_fma(g.x, st[2 * i], f2_mul(k.x, v));
            st[2 * i + 1] = f2_fma(g.y, st[2 * i + 1], f2_mul(k.y, v));
            if (!PRE) {
                o01 = f2_fma(st[2 * i], q.x, o01);
                o23 = f2_fma(st[2 * i + 1], q.y, o23);
            }
        }
        float o0, o1, o2, o3;
        f2_unpack(o01, o0, o1);
        f2_unpack(o23, o2, o3);
        return (o0 + o1) + (o2 + o3);
    };
    // One run of staged tokens, walked in order. A warp issues in order, so a token's chain of shuffles
    // (each waits for the one before) would hold up the next token's sums: LA_GROUP tokens' shares are
    // kept and summed over the parts together, their chains side by side. A full run is unrolled.
    auto walk = [&](const float* qs, const float* ks, const float* vs, const float* bs, int r0, int nt) {
        qs += part * SEG;
        ks += part * SEG;
        vs += warp * CW + e_local;
        float* orow = out + (size_t)r0 * H * dv + h * dv + e;
        const bool writes = part == 0 && e < dv;
        int t = 0;
        if (nt == LA_RUN) {
#pragma unroll
            for (int g0 = 0; g0 < LA_RUN; g0 += LA_GROUP) {
                float o[LA_GROUP];
#pragma unroll
                for (int g = 0; g < LA_GROUP; ++g) o[g] = token(qs, ks, vs, g0 + g);
#pragma unroll
                for (int x = CW; x < 32; x <<= 1)
#pragma unroll
                    for (int g = 0; g < LA_GROUP; ++g) o[g] += __shfl_xor_sync(0xffffffffu, o[g], x);
                if (writes)
#pragma unroll
                    for (int g = 0; g < LA_GROUP; ++g)
                        orow[(size_t)(g0 + g) * H * dv] =
                            PRE ? fmaf(bs[g0 + g], vs[(g0 + g) * COLS], o[g] * o_scale) : o[g] * o_scale;
            }
            t = LA_RUN;
        }
        for (; t < nt; ++t) {
            float o = token(qs, ks, vs, t);
#pragma unroll
            for (int x = CW; x < 32; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
            if (writes) orow[(size_t)t * H * dv] = PRE ? fmaf(bs[t], vs[t * COLS], o * o_scale) : o * o_scale;
        }
    };
    float* qs = sm;
    float* ks = sm + LA_RUN * DR;
    float* as = sm + 2 * LA_RUN * DR;            // CH only
    float* vs = sm + ROWS * LA_RUN * DR;
    float* bs = vs + LA_RUN * COLS;              // PRE only
    for (int r0 = t0; r0 < t1; r0 += LA_RUN) {
        const int nt = min(LA_RUN, t1 - r0);
        __syncthreads();            // the run before has been walked
        for (int i = tid; i < nt * PARTS * JPT; i += LA_THREADS) {
            const int t = i / (PARTS * JPT), j = i - t * (PARTS * JPT);
            float qv = 0.0f, kv = 0.0f, av = 0.0f;
            if (j < d) {
                if (CH) av = alpha[(size_t)(r0 + t) * H * d + h * d + j];
                const float* row = u + (size_t)(r0 + t) * W + h * d + j;
                qv = la_act(la_parts_sum(row + q_col, S, split_stride), act);
                kv = la_act(la_parts_sum(row + k_col, S, split_stride), act);
            }
            qs[t * DR + (j / JPT) * SEG + j % JPT] = qv;
            ks[t * DR + (j / JPT) * SEG + j % JPT] = kv;
            if (CH) as[t * DR + (j / JPT) * SEG + j % JPT] = av;
        }
        for (int i = tid; i < nt * COLS; i += LA_THREADS) {
            const int t = i / COLS, c = i - t * COLS;
            vs[i] = e0 + c < dv
                ? la_act(la_parts_sum(u + (size_t)(r0 + t) * W + v_col + h * dv + e0 + c, S, split_stride), act) : 0.0f;
        }
        if (PRE && tid < nt) bs[tid] = bonus[(size_t)(r0 + tid) * H + h];
        __syncthreads();
        walk(qs, ks, vs, bs, r0, nt);
    }
#pragma unroll
    for (int i = 0; i < JPT; i += 2) {
        const int j = part * JPT + i;
        float lo, hi;
        f2_unpack(st[i / 2], lo, hi);
        if (j < d && e < dv) Sg[(size_t)j * dv + e] = lo;
        if (j + 1 < d && e < dv) Sg[(size_t)(j + 1) * dv + e] = hi;
    }
}

// Prompts: the walk from staged runs. u holds one sum a value, no activation left to apply (the dense
// buffer of linear_attn_prep_kernel, or a projection that is one already), q, k and v at columns that are
// multiples of 4, d and dv multiples of 4. Eight lanes share CPT columns, lane part p holding rows p JPT ..
// of each (d <= 8 JPT): the words of q, k and the decays that a lane reads from shared memory serve all its
// columns. A warp has 4 CPT columns, a block 16 CPT. In shared memory a token's q (and k, and decay) row is
// 8 segments of JPT + 4 values: the 4 values of padding put the segments that a warp reads together on
// different banks (segments of 4 values need none: 32 lanes then read 512 bytes in a row). FOLD: no
// queries and no outputs, every chunk's state from zero goes to its place in `chunks`. With `chunks` and
// not FOLD every chunk's walk starts from its place there, and a sequence's last chunk writes its state.
template <int JPT, int CPT, int MODE, bool FOLD>
__global__ void __launch_bounds__(LA_THREADS)
linear_attn_run_kernel(const float* __restrict__ u, int W, int q_col, int k_col, int v_col,
                       const float* __restrict__ decay, float* __restrict__ state, size_t slot_stride,
                       const int* __restrict__ cu_q, const int* __restrict__ seq_slot, float* __restrict__ out, int H, int d,
                       int dv, const float* __restrict__ alpha, const float* __restrict__ bonus, float o_scale,
                       float* __restrict__ chunks, int n_seqs) {
    constexpr bool CH = MODE != LA_FIXED, PRE = MODE == LA_BONUS && !FOLD;
    constexpr int COLS = 16 * CPT;
    constexpr int SEG = JPT + (JPT == 4 ? 0 : 4), DR = 8 * SEG;
    constexpr int ROWS = CH ? 3 : 2;
    constexpr int BUF = LA_RUN * (ROWS * DR + COLS + (PRE ? 1 : 0));
    constexpr int GROUP = CPT == 1 ? 8 : (CPT == 2 ? 4 : 2);       // tokens whose sums over the parts are taken together
    extern __shared__ __align__(16) float sm[];     // twice: q [LA_RUN][DR], k, (decays,) v [LA_RUN][COLS]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int part = lane >> 2, c0 = warp * 4 * CPT + (lane & 3) * CPT;      // this lane's first column in the block
    const int e0 = blockIdx.x * COLS, h = blockIdx.y, e = e0 + c0;
    const float a = CH ? 0.0f : decay[h];
    pdl_trigger();
    pdl_wait();
    int b = blockIdx.z, t0, t1, number;
    bool last = true;
    if (chunks) {
        if (!la_chunk(cu_q, n_seqs, blockIdx.z, b, number, t0, t1, last)) return;
        if (FOLD && last) return;                   // nobody starts from the end of a sequence's last chunk
    } else {
        t0 = cu_q[b], t1 = cu_q[b + 1];
        if (t1 <= t0) return;
    }
    float* Sg = state + (size_t)seq_slot[b] * slot_stride + (size_t)h * d * dv;
    float* Cg = chunks ? chunks + ((size_t)blockIdx.z * H + h) * d * dv : nullptr;
    const float* from = chunks ? Cg : Sg;
    f32x2 st[CPT][JPT / 2];
#pragma unroll
    for (int i = 0; i < JPT; i += 2) {
        const int j = part * JPT + i;               // d is a multiple of 4: rows j and j + 1 are both inside or both beyond
#pragma unroll
        for (int c = 0; c < CPT; ++c)
            st[c][i / 2] = !FOLD && j < d && e + c < dv
                ? f2_pack(from[(size_t)j * dv + e + c], from[(size_t)(j + 1) * dv + e + c]) : f2_pack(0.0f, 0.0f);
    }
    const f32x2 aa = f2_pack(a, a);
    // rows beyond d, the padding and columns beyond dv are zeros in both sets and are never copied over
    for (int i = tid; i < 2 * BUF; i += LA_THREADS) sm[i] = 0.0f;
    __syncthreads();
    const int qc = d >> 2, pieces = ROWS * qc + COLS / 4;    // 16-byte pieces a token: q, k, (decays,) v
    auto fetch = [&](int r0, int nt, float* buf) {
        for (int c = FOLD ? qc + tid : tid; c < pieces; c += LA_THREADS) {     // a thread copies its piece of every token
            const float* src;
            float* dst;
            size_t src_row = W;
            int dst_row = DR;
            if (c < ROWS * qc) {
                const int which_row = c / qc, j = 4 * (c - which_row * qc);    // JPT is a multiple of 4: a piece lies in one segment
                if (CH && which_row == 2) {
                    src_row = (size_t)H * d;
                    src = alpha + (size_t)r0 * src_row + h * d + j;
                } else {
                    src = u + (size_t)r0 * W + (which_row == 0 ? q_col : k_col) + h * d + j;
                }
                dst = buf + which_row * LA_RUN * DR + (j / JPT) * SEG + j % JPT;
            } else {
                const int j = 4 * (c - ROWS * qc);
                if (e0 + j >= dv) continue;
                src = u + (size_t)r0 * W + v_col + h * dv + e0 + j;
                dst = buf + ROWS * LA_RUN * DR + j;
                dst_row = COLS;
            }
            if (nt == LA_RUN) {
#pragma unroll
                for (int t = 0; t < LA_RUN; ++t) la_cp16(dst + t * dst_row, src + (size_t)t * src_row);
            } else {
                for (int t = 0; t < nt; ++t) la_cp16(dst + t * dst_row, src + (size_t)t * src_row);
            }
        }
        if (PRE && tid < nt)
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(
                             buf + LA_RUN * (ROWS * DR + COLS) + tid)),
                         "l"(bonus + (size_t)(r0 + tid) * H + h)
                         : "memory");
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // one token: the state moves on; what comes back is this part's share of its columns' outputs
    auto token = [&](const float* qs, const float* vs, int t, float (&o)[CPT]) {
        const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(qs + t * DR);
        const ulonglong2* k4 = q4 + LA_RUN * DR / 4;
        const ulonglong2* a4 = k4 + LA_RUN * DR / 4;      // CH only
        f32x2 v[CPT], s0[CPT], s1[CPT];
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            const float x = vs[t * COLS + c];
            v[c] = f2_pack(x, x);
            s0[c] = s1[c] = f2_pack(0.0f, 0.0f);
        }
#pragma unroll
        for (int i = 0; i < JPT / 4; ++i) {
            const ulonglong2 k = k4[i];
            ulonglong2 g = make_ulonglong2(aa, aa), q = g;
            if (CH) g = a4[i];
            if (!FOLD) q = q4[i];
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                if (PRE) {
                    s0[c] = f2_fma(st[c][2 * i], q.x, s0[c]);
                    s1[c] = f2_fma(st[c][2 * i + 1], q.y, s1[c]);
                }
                st[c][2 * i] = f2_fma(g.x, st[c][2 * i], f2_mul(k.x, v[c]));
                st[c][2 * i + 1] = f2_fma(g.y, st[c][2 * i + 1], f2_mul(k.y, v[c]));
                if (!FOLD && !PRE) {
                    s0[c] = f2_fma(st[c][2 * i], q.x, s0[c]);
                    s1[c] = f2_fma(st[c][2 * i + 1], q.y, s1[c]);
                }
            }
        }
        if (FOLD) return;
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            float x0, x1, x2, x3;
            f2_unpack(s0[c], x0, x1);
            f2_unpack(s1[c], x2, x3);
            o[c] = (x0 + x1) + (x2 + x3);
        }
    };
    // The columns' sums over the eight parts (lane bits 2, 3, 4), handed out to the lanes on the way: a lane
    // gives away the half of its columns that its partner keeps. Lane (part p) ends with column `mine`.
    const bool hi = lane & 16, mid = lane & 8;
    const int mine = CPT == 4 ? 2 * hi + mid : (CPT == 2 ? hi : 0);
    const bool writes = (CPT == 4 ? !(part & 1) : (CPT == 2 ? !(part & 3) : part == 0)) && e + mine < dv;
    auto gather = [&](const float (&o)[CPT]) -> float {
        float x;
        if (CPT == 4) {
            const float k0 = (hi ? o[2 % CPT] : o[0]) + __shfl_xor_sync(0xffffffffu, hi ? o[0] : o[2 % CPT], 16);
            const float k1 = (hi ? o[3 % CPT] : o[1 % CPT]) + __shfl_xor_sync(0xffffffffu, hi ? o[1 % CPT] : o[3 % CPT], 16);
            x = (mid ? k1 : k0) + __shfl_xor_sync(0xffffffffu, mid ? k0 : k1, 8);
        } else if (CPT == 2) {
            x = (hi ? o[1 % CPT] : o[0]) + __shfl_xor_sync(0xffffffffu, hi ? o[0] : o[1 % CPT], 16);
            x += __shfl_xor_sync(0xffffffffu, x, 8);
        } else {
            x = o[0] + __shfl_xor_sync(0xffffffffu, o[0], 16);
            x += __shfl_xor_sync(0xffffffffu, x, 8);
        }
        return x + __shfl_xor_sync(0xffffffffu, x, 4);
    };
    fetch(t0, min(LA_RUN, t1 - t0), sm);
    int which = 0;
    for (int r0 = t0; r0 < t1; r0 += LA_RUN, which ^= 1) {
        const int nt = min(LA_RUN, t1 - r0);
        float* buf = sm + which * BUF;
        if (r0 + LA_RUN < t1) {
            fetch(r0 + LA_RUN, min(LA_RUN, t1 - r0 - LA_RUN), sm + (which ^ 1) * BUF);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* qs = buf + part * SEG;
        const float* vs = buf + ROWS * LA_RUN * DR + c0;
        const float* bs = buf + LA_RUN * (ROWS * DR + COLS);        // PRE only
        const auto finish = [&](float x, int t) {
            return PRE ? fmaf(bs[t], vs[t * COLS + mine], x * o_scale) : x * o_scale;
        };
        float* orow = out + (size_t)r0 * H * dv + h * dv + e + mine;
        // A warp issues in order, so a token's chain of shuffles (each waits for the one before) would hold
        // up the next token's sums: GROUP tokens' shares are kept and gathered together.
        int t = 0;
        for (; t + GROUP <= nt; t += GROUP) {
            float o[GROUP][CPT];
#pragma unroll
            for (int g = 0; g < GROUP; ++g) token(qs, vs, t + g, o[g]);
            if (!FOLD) {
                float x[GROUP];
#pragma unroll
                for (int g = 0; g < GROUP; ++g) x[g] = gather(o[g]);
#pragma unroll
                for (int g = 0; g < GROUP; ++g)
                    if (writes) orow[(size_t)(t + g) * H * dv] = finish(x[g], t + g);
            }
        }
        for (; t < nt; ++t) {
            float o[CPT];
            token(qs, vs, t, o);
            if (!FOLD) {
                const float x = gather(o);
                if (writes) orow[(size_t)t * H * dv] = finish(x, t);
            }
        }
        __syncthreads();            // before the run after the next is copied over this one
    }
    if (!FOLD && !last) return;
    float* to = FOLD ? Cg : Sg;
#pragma unroll
    for (int i = 0; i < JPT; i += 2) {
        const int j = part * JPT + i;
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            float lo, up;
            f2_unpack(st[c][i / 2], lo, up);
            if (j < d && e + c < dv) {
                to[(size_t)j * dv + e + c] = lo;
                to[(size_t)(j + 1) * dv + e + c] = up;
            }
        }
    }
}

// prod[z, c] = the product of the decays of chunk z for the H d channels (alpha [N, H d], or decay [H]). A
// block takes 32 channels, a warp of it every eighth run of tokens.
__global__ void __launch_bounds__(256)
linear_attn_chunk_decay_kernel(const float* __restrict__ alpha, const float* __restrict__ decay, float* __restrict__ prod,
                               const int* __restrict__ cu_q, int n_seqs, int Hd, int d) {
    __shared__ float part[8][32];
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int c = blockIdx.x * 32 + lane, ci = min(c, Hd - 1);
    int b, i, t0, t1;
    bool last;
    if (!la_chunk(cu_q, n_seqs, blockIdx.y, b, i, t0, t1, last) || last) return;
    float v[LA_CHUNK / 8];
#pragma unroll
    for (int k = 0; k < LA_CHUNK / 8; ++k) {
        const int t = t0 + 8 * k + warp;
        v[k] = t < t1 ? (alpha ? alpha[(size_t)t * Hd + ci] : decay[ci / d]) : 1.0f;
    }
    float p = 1.0f;
#pragma unroll
    for (int k = 0; k < LA_CHUNK / 8; ++k) p *= v[k];
    part[warp][lane] = p;
    __syncthreads();
    if (warp == 0 && c < Hd) {
        for (int k = 1; k < 8; ++k) p *= part[k][lane];
        prod[(size_t)blockIdx.y * Hd + c] = p;
    }
}

// In place: the folds in `chunks` become the states the chunks start from. A thread a state number of a
// sequence: it walks the sequence's chunks in order, LA_AHEAD folds on their way at a time.
#define LA_AHEAD 8
__global__ void __launch_bounds__(256)
linear_attn_carry_kernel(float* __restrict__ chunks, const float* __restrict__ prod, const float* __restrict__ state,
                         size_t slot_stride, const int* __restrict__ cu_q, const int* __restrict__ seq_slot, int H, int d,
                         int dv) {
    // no early trigger: see linear_attn_prep_kernel
    pdl_wait();
    const int b = blockIdx.y, n = H * d * dv;
    const int i = blockIdx.x * 256 + threadIdx.x;
    if (i >= n) return;
    int z = 0;
    for (int k = 0; k < b; ++k) z += (cu_q[k + 1] - cu_q[k] + LA_CHUNK - 1) / LA_CHUNK;
    const int nc = (cu_q[b + 1] - cu_q[b] + LA_CHUNK - 1) / LA_CHUNK;
    if (nc <= 0) return;
    float s = state[(size_t)seq_slot[b] * slot_stride + i];
    float* at = chunks + (size_t)z * n + i;
    const float* pr = prod + (size_t)z * H * d + i / dv;
    for (int k0 = 0; k0 < nc; k0 += LA_AHEAD) {
        float fold[LA_AHEAD], p[LA_AHEAD];
#pragma unroll
        for (int k = 0; k < LA_AHEAD; ++k)
            if (k0 + k + 1 < nc) {
                fold[k] = at[(size_t)(k0 + k) * n];
                p[k] = pr[(size_t)(k0 + k) * H * d];
            }
#pragma unroll
        for (int k = 0; k < LA_AHEAD; ++k)
            if (k0 + k < nc) {
                at[(size_t)(k0 + k) * n] = s;
                if (k0 + k + 1 < nc) s = fmaf(p[k], s, fold[k]);
            }
    }
}

// Largest key size the kernel takes.
LUMEN_API int lumen_linear_attn_max_dim() { return 4 * 128; }

// 1 if a step of N tokens in n_seqs sequences takes the prompt path (it then needs a dense float32
// buffer of N (2 H d + H dv) values): at least LA_PRE_TOKENS tokens a sequence on average, head sizes
// that are multiples of 4.
#define LA_PRE_TOKENS 32
LUMEN_API int lumen_linear_attn_wants_dense(int N, int n_seqs, int d, int dv) {
    return (n_seqs > 0 && (long long)N >= (long long)LA_PRE_TOKENS * n_seqs && !(d & 3) && !(dv & 3)) ? 1 : 0;
}
// Chunks of a step that is walked in chunks (with chunk states of that many [H][d][dv] and products of that
// many [H d] as scratch); 0: the step is walked whole. In chunks where the sequences are long and one walk
// a (sequence, head, 64 columns) would leave the SMs with less than three blocks of four warps each.
LUMEN_API int lumen_linear_attn_chunks(int N, int n_seqs, int H, int d, int dv) {
    if (!lumen_linear_attn_wants_dense(N, n_seqs, d, dv) || (long long)N < 2LL * LA_CHUNK * n_seqs ||
        (long long)n_seqs * H * ((dv + 63) / 64) >= 3 * 148)
        return 0;
    return N / LA_CHUNK + n_seqs;
}
LUMEN_API int lumen_linear_attn_copies_from(const float* u, int n_split, int W, int q_col, int k_col, int v_col, int act) {
    return (n_split == 1 && !act && !((W | q_col | k_col | v_col) & 3) && !((uintptr_t)u & 15)) ? 1 : 0;
}

// The decays of a step from a projection of low rank: alpha[n, c] = sigmoid(z)^(1/tau) with
// z = bias[c] + sum_r t[n, r] w[r, c], t = columns c_col .. c_col + R of u (partial sums [S, N, W], added), w
// [R, C]; taken as exp(-softplus(-z) / tau), all in float32. A block takes LD_TOK tokens and 128 CPT channels,
// CPT a thread; the tokens' R numbers lie in shared memory, LD_RANK at a time, a rank's numbers of all tokens
// together, and the weights are fetched LD_AHEAD ranks ahead (the first ones before the kernel ahead has ended). With `twice` the numbers go through tanh
// first and alpha = exp(-exp(z)). The blocks behind the channels' (where `ub` is given) make the bonus of
// linear_attn_kernel instead, one head a block, a warp a token at a time: bonus[n, h] = sum_j q_j ub[h d + j] k_j
// with q and k columns of u.
struct BonusOf {
    const float* ub;           // [H d]
    float* out;                // [N, H]
    int q_col, k_col, H, d;
};
#define LD_TOK 16
#define LD_RANK 128
template <int CPT, int LD_AHEAD>
__global__ void __launch_bounds__(128)
low_rank_decay_kernel(const float* __restrict__ u, int S, size_t split_stride, int W, int c_col, int R,
                      const float* __restrict__ w, const float* __restrict__ bias, float inv_tau,
                      float* __restrict__ alpha, int N, int C, int twice, const BonusOf bo) {
    // no early trigger: see linear_attn_prep_kernel
    __shared__ __align__(16) float ts[LD_RANK][LD_TOK + 4];
    const int n0 = blockIdx.y * LD_TOK, channel_blocks = (C + 128 * CPT - 1) / (128 * CPT);
    if ((int)blockIdx.x >= channel_blocks) {
        pdl_wait();
        const int h = blockIdx.x - channel_blocks, lane = threadIdx.x & 31, n1 = n0 + 4 * (threadIdx.x >> 5);
        float sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        const float* row = u + (size_t)n1 * W + h * bo.d;
#pragma unroll 2
        for (int j = lane; j < bo.d; j += 32) {
            float q[4], k[4];
#pragma unroll
            for (int t = 0; t < 4; ++t) q[t] = n1 + t < N ? row[(size_t)t * W + bo.q_col + j] : 0.0f;
#pragma unroll
            for (int t = 0; t < 4; ++t) k[t] = n1 + t < N ? row[(size_t)t * W + bo.k_col + j] : 0.0f;
            for (int s = 1; s < S; ++s)
#pragma unroll
                for (int t = 0; t < 4; ++t)
                    if (n1 + t < N) {
                        q[t] += row[(size_t)s * split_stride + (size_t)t * W + bo.q_col + j];
                        k[t] += row[(size_t)s * split_stride + (size_t)t * W + bo.k_col + j];
                    }
            const float b = bo.ub[h * bo.d + j];
#pragma unroll
            for (int t = 0; t < 4; ++t) sum[t] = fmaf(q[t] * b, k[t], sum[t]);
        }
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            sum[t] = warp_sum(sum[t]);
            if (lane == 0 && n1 + t < N) bo.out[(size_t)(n1 + t) * bo.H + h] = sum[t];
        }
        return;
    }
    const int c0 = blockIdx.x * 128 * CPT + threadIdx.x;
    float wn[CPT][LD_AHEAD];
    auto fetch = [&](int r) {
#pragma unroll
        for (int k = 0; k < LD_AHEAD; ++k)
#pragma unroll
            for (int m = 0; m < CPT; ++m) wn[m][k] = r + k < R && c0 + 128 * m < C ? w[(size_t)(r + k) * C + c0 + 128 * m] : 0.0f;
    };
    fetch(0);
    f32x2 z[CPT][LD_TOK / 2];              // two tokens a lane and instruction
#pragma unroll
    for (int m = 0; m < CPT; ++m) {
        const float b = c0 + 128 * m < C ? bias[c0 + 128 * m] : 0.0f;
#pragma unroll
        for (int t = 0; t < LD_TOK / 2; ++t) z[m][t] = f2_pack(b, b);
    }
    pdl_wait();
    for (int r0 = 0; r0 < R; r0 += LD_RANK) {
        const int nr = min(LD_RANK, R - r0), nr8 = (nr + LD_AHEAD - 1) / LD_AHEAD * LD_AHEAD;   // zeros up to a whole step
        __syncthreads();
        // a thread takes one rank's numbers of some tokens, eight loads in flight
        const int lanes = 128 / nr8, r = threadIdx.x % nr8, tg = threadIdx.x / nr8;
        for (int t0 = tg; t0 < LD_TOK && tg < lanes; t0 += 8 * lanes) {
            float x[8];
            const float* src = u + (size_t)(n0 + t0) * W + c_col + r0 + r;
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = r < nr && t0 + j * lanes < min(LD_TOK, N - n0) ? src[(size_t)j * lanes * W] : 0.0f;
            for (int s = 1; s < S; ++s)
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    if (r < nr && t0 + j * lanes < min(LD_TOK, N - n0)) x[j] += src[(size_t)s * split_stride + (size_t)j * lanes * W];
#pragma unroll
            for (int j = 0; j < 8; ++j)
                if (t0 + j * lanes < LD_TOK) ts[r][t0 + j * lanes] = twice ? tanhf(x[j]) : x[j];
        }
        __syncthreads();
        for (int r1 = 0; r1 < nr8; r1 += LD_AHEAD) {
            float wv[CPT][LD_AHEAD];
#pragma unroll
            for (int k = 0; k < LD_AHEAD; ++k)
#pragma unroll
                for (int m = 0; m < CPT; ++m) wv[m][k] = wn[m][k];
            // the step after this one; behind a full run of ranks it begins at the next run
            fetch(r0 + r1 + LD_AHEAD < r0 + nr8 ? r0 + r1 + LD_AHEAD : r0 + LD_RANK);
#pragma unroll
            for (int k = 0; k < LD_AHEAD; ++k) {
                f32x2 w2[CPT];
#pragma unroll
                for (int m = 0; m < CPT; ++m) w2[m] = f2_pack(wv[m][k], wv[m][k]);
#pragma unroll
                for (int t = 0; t < LD_TOK / 2; t += 2) {
                    const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(&ts[r1 + k][2 * t]);
#pragma unroll
                    for (int m = 0; m < CPT; ++m) {
                        z[m][t] = f2_fma(x.x, w2[m], z[m][t]);
                        z[m][t + 1] = f2_fma(x.y, w2[m], z[m][t + 1]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int m = 0; m < CPT; ++m) {
        const int c = c0 + 128 * m;
        if (c >= C) break;
#pragma unroll
        for (int t = 0; t < LD_TOK; ++t)
            if (n0 + t < N) {
                float lo, hi;
                f2_unpack(z[m][t / 2], lo, hi);
                const float x = t & 1 ? hi : lo;
                if (twice) {
                    alpha[(size_t)(n0 + t) * C + c] = expf(-expf(x));
                } else {
                    const float softplus_neg = fmaxf(-x, 0.0f) + log1pf(expf(-fabsf(x)));
                    alpha[(size_t)(n0 + t) * C + c] = expf(-softplus_neg * inv_tau);
                }
            }
    }
}

LUMEN_API int lumen_low_rank_decay(const float* u, int n_split, long long split_stride, int W, int c0, int R,
                                   const float* w, const float* bias, float inv_tau, float* alpha, int N, int C,
                                   int twice, const float* ub, int q_col, int k_col, int H, int d, float* bonus,
                                   cudaStream_t stream) {
    if (N <= 0) return 0;
    if (ub && (!bonus || H <= 0 || d <= 0 || q_col < 0 || k_col < 0 || q_col + H * d > W || k_col + H * d > W))
        return LUMEN_ERR_BAD_ARGUMENT;
    const BonusOf bo = {ub, bonus, q_col, k_col, H, d};
    if (n_split < 1 || R <= 0 || C <= 0 || c0 < 0 || c0 + R > W || !(inv_tau > 0.0f)) return LUMEN_ERR_BAD_ARGUMENT;
    if ((N + LD_TOK - 1) / LD_TOK > 65535) return LUMEN_ERR_UNSUPPORTED;
    // few tokens: a channel a thread, so that the step has more blocks, and more weights ahead
    const int cols = N <= 4 * LD_TOK ? 128 : 256;
    const dim3 grid((C + cols - 1) / cols + (ub ? H : 0), (N + LD_TOK - 1) / LD_TOK);
    auto k = cols == 128 ? low_rank_decay_kernel<1, 16> : low_rank_decay_kernel<2, 8>;
    lumen_launch(k, grid, dim3(128), 0, stream, u, n_split, (size_t)split_stride, W, c0, R, w, bias, inv_tau, alpha, N, C,
                 twice, bo);
    LUMEN_LAUNCH_CHECK();
    return 0;
}

// u: [S, N, W] partial sums; decay float32 [H] (or null, with alpha float32 [N, H d] instead, and then bonus
// float32 [N, H] or null); state float32, sequence b's at state + seq_slot[b] *
// slot_stride as [H][d][dv], updated in place; cu_q int32 [B + 1]; out float32 [N, H dv]; dense: float32
// scratch of N (2 H d + H dv) values, 16-byte aligned, or null for the direct path. A prompt whose projection
// is one sum, without an activation and with every row piece on a 16-byte boundary needs no dense buffer:
// the walk copies from the projection itself (lumen_linear_attn_copies_from says so).
LUMEN_API int lumen_linear_attn(const float* u, int n_split, long long split_stride, int W, int q_col, int k_col,
                                int v_col, int act, const float* decay, float* state, long long slot_stride,
                                const int* cu_q, const int* seq_slot, int n_seqs, float* out, int H, int d, int dv,
                                float* dense, int N, const float* alpha, const float* bonus, float o_scale,
                                float* chunks, float* prod, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (bonus && !alpha) return LUMEN_ERR_BAD_ARGUMENT;
    if ((decay == nullptr) == (alpha == nullptr) || ((uintptr_t)alpha & 15)) return LUMEN_ERR_BAD_ARGUMENT;
    if (n_split < 1 || H <= 0 || d <= 0 || dv <= 0 || q_col < 0 || k_col < 0 || v_col < 0 || q_col + H * d > W ||
        k_col + H * d > W || v_col + H * dv > W)
        return LUMEN_ERR_BAD_ARGUMENT;
    if (d > lumen_linear_attn_max_dim() || H > 65535 || n_seqs > 65535) return LUMEN_ERR_UNSUPPORTED;
    const bool direct = lumen_linear_attn_wants_dense(N, n_seqs, d, dv) &&
                        lumen_linear_attn_copies_from(u, n_split, W, q_col, k_col, v_col, act);
    const bool pre = dense != nullptr || direct;
    if (pre && !direct) {
        if ((d & 3) || (dv & 3) || ((uintptr_t)dense & 15) || N <= 0) return LUMEN_ERR_BAD_ARGUMENT;
        const long long total = (long long)N * (2 * H * d + H * dv);
        long long blocks = (total + 255) / 256;
        if (blocks > 148 * 16) blocks = 148 * 16;
        lumen_launch(linear_attn_prep_kernel, dim3((int)blocks), dim3(256), 0, stream, u, n_split, (size_t)split_stride, W,
                     q_col, k_col, v_col, H * d, H * dv, act, dense, total);
        LUMEN_LAUNCH_CHECK();
        u = dense;
        W = 2 * H * d + H * dv;
        q_col = 0, k_col = H * d, v_col = 2 * H * d, act = 0, n_split = 1, split_stride = 0;
    }
    const int n_chunks = chunks ? lumen_linear_attn_chunks(N, n_seqs, H, d, dv) : 0;
    if (chunks && (!n_chunks || !pre || !prod)) return LUMEN_ERR_BAD_ARGUMENT;
    if (n_chunks > 65535) return LUMEN_ERR_UNSUPPORTED;
#define LA_RUN_(JPT_, CPT_, MODE_, FOLD_)                                                                            \
    do {                                                                                                             \
        constexpr int cols = 16 * CPT_, seg = JPT_ + (JPT_ == 4 ? 0 : 4);                                            \
        const size_t smem = 2 * (size_t)LA_RUN * ((MODE_ ? 3 : 2) * 8 * seg + cols + 1) * sizeof(float);             \
        auto kern = linear_attn_run_kernel<JPT_, CPT_, MODE_, FOLD_>;                                                  \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
        lumen_launch(kern, dim3((dv + cols - 1) / cols, H, n_chunks ? n_chunks : n_seqs), dim3(LA_THREADS), smem,    \
                     stream, u, W, q_col, k_col, v_col, decay, state, (size_t)slot_stride, cu_q, seq_slot, out, H,   \
                     d, dv, alpha, bonus, o_scale, chunks, n_seqs);                                                  \
    } while (0)
    // columns a lane: as many as leave its share of the state in registers, where there are blocks enough
#define LA_RUNS(JPT_, CPT_, FOLD_)                                                                                   \
    do {                                                                                                             \
        if (wide) {                                                                                                  \
            if (bonus && !FOLD_) LA_RUN_(JPT_, CPT_, LA_BONUS, false);                                               \
            else if (alpha) LA_RUN_(JPT_, CPT_, LA_CHANNEL, FOLD_);                                                  \
            else LA_RUN_(JPT_, CPT_, LA_FIXED, FOLD_);                                                               \
        } else {                                                                                                     \
            if (bonus) LA_RUN_(JPT_, 1, LA_BONUS, false);                                                            \
            else if (alpha) LA_RUN_(JPT_, 1, LA_CHANNEL, false);                                                     \
            else LA_RUN_(JPT_, 1, LA_FIXED, false);                                                                  \
        }                                                                                                            \
    } while (0)
#define LA_BY_D(FOLD_)                                                                                               \
    do {                                                                                                             \
        if (d <= 32) LA_RUNS(4, 4, FOLD_);                                                                           \
        else if (d <= 64) LA_RUNS(8, 4, FOLD_);                                                                      \
        else if (d <= 128) LA_RUNS(16, 4, FOLD_);                                                                    \
        else if (d <= 256) LA_RUNS(32, 2, FOLD_);                                                                    \
        else LA_RUNS(64, 1, FOLD_);                                                                                  \
    } while (0)
    if (pre) {
        const bool wide = n_chunks || (long long)n_seqs * H * ((dv + 63) / 64) >= 2 * 148;
        if (n_chunks) {
            LA_BY_D(true);
            LUMEN_LAUNCH_CHECK();
            lumen_launch(linear_attn_chunk_decay_kernel, dim3((H * d + 31) / 32, n_chunks), dim3(256), 0, stream, alpha,
                         decay, prod, cu_q, n_seqs, H * d, d);
            LUMEN_LAUNCH_CHECK();
            lumen_launch(linear_attn_carry_kernel, dim3((H * d * dv + 255) / 256, n_seqs), dim3(256), 0, stream, chunks,
                         (const float*)prod, (const float*)state, (size_t)slot_stride, cu_q, seq_slot, H, d, dv);
            LUMEN_LAUNCH_CHECK();
        }
        LA_BY_D(false);
    } else {
        // 4 lanes a column, a sector of the state a part
#define LA_GO_(JPT_, MODE_)                                                                                            \
    do {                                                                                                             \
        constexpr int cols = 32;                                                                                     \
        const size_t smem = (size_t)LA_RUN * ((MODE_ ? 3 : 2) * 4 * (JPT_ + 4) + cols + 1) * sizeof(float);          \
        auto kern = linear_attn_kernel<JPT_, 4, MODE_>;                                                                \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
        lumen_launch(kern, dim3((dv + cols - 1) / cols, H, n_seqs), dim3(LA_THREADS), smem, stream, u, n_split,      \
                     (size_t)split_stride, W, q_col, k_col, v_col, act, decay, state, (size_t)slot_stride, cu_q,     \
                     seq_slot, out, H, d, dv, alpha, bonus, o_scale);                                                \
    } while (0)
#define LA_GO(JPT_)                                                                                                  \
    do { if (bonus) LA_GO_(JPT_, LA_BONUS); else if (alpha) LA_GO_(JPT_, LA_CHANNEL); else LA_GO_(JPT_, LA_FIXED); } while (0)
        if (d <= 32) LA_GO(8);
        else if (d <= 64) LA_GO(16);
        else if (d <= 128) LA_GO(32);
        else if (d <= 256) LA_GO(64);
        else LA_GO(128);
    }
#undef LA_GO
#undef LA_GO_
#undef LA_BY_D
#undef LA_RUNS
#undef LA_RUN_
    LUMEN_LAUNCH_CHECK();
    return 0;
}
