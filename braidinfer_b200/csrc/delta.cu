// The gated delta rule with a decay a key channel: per sequence and head a state S [dk, dv], float32, and per token
//     S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
// with g = exp(-rate softplus(z + bias)) a channel and beta = sigmoid(b) a head.  (The delta rule as a fast-weight update is
// Schlag, Irie, Schmidhuber: "Linear Transformers Are Secretly Fast Weight Programmers", 2021; the form over chunks follows
// Yang, Wang, Zhang, Shen, Kim: "Parallelizing Linear Transformers with the Delta Rule over Sequence Length", 2024, here with
// a decay a channel.)  q, k, v arrive as float32 rows (convolved, of unit length and scaled: conv_heads.cu), z as float32
// logits, b in the run's type; everything here is float32 arithmetic on the ordinary pipes.
//
// Short steps are walked token by token (delta_walk_kernel).  Long ones are cut into chunks of 64 tokens.  With D(s, t) the product
// of the decays of the tokens after s up to t (a channel; 0: the chunk's start) and S_0 the state a chunk starts from, the
// walk over a chunk is
//     A_ts = sum_i k_t k_s D(s, t)  (s < t),     P_ts = sum_i q_t k_s D(s, t)  (s <= t)
//     (I + diag(beta) A) [W | U0] = diag(beta) [k_t D(0, t) | v_t]                    (forward substitution)
//     U = U0 - W S_0
//     O = (q_t D(0, t)) S_0 + P U
//     S_64 = diag(D(0, 64)) S_0 + (k_t D(t, 64))^T U
// so all but the two products with S_0 that make U and the next S run for all chunks side by side:
//     delta_intra_kernel   W, U0, P and the decayed q and k of every chunk
//     delta_state_kernel   chunk after chunk, a tile of value columns a CTA: U, and the state every chunk starts from
//     delta_out_kernel     O of every chunk
// No logarithm is taken: the decay between two tokens is a product of at most 16 decays at a time, which rounds like the walk
// does.  Sub-chunks of 16 tokens are related through the products at their edges (never above one).  Inside a sub-chunk the
// decay from s to t is taken as (edge to t) / (edge to s) for the channels whose decays over the sub-chunk multiply to 2^-60 or
// more, and multiplied up pair by pair for the others.
#include "common.cuh"
#include "gated_norm.cuh"

#define DELTA_MAX_DK 256
#define DELTA_CV 4
#define DELTA_WALK_THREADS 128
#define DELTA_C 64                 // tokens a chunk
#define DELTA_SUB 16               // tokens a sub-chunk
#define DELTA_NSUB (DELTA_C / DELTA_SUB)
#define DELTA_DVT 16               // value columns a CTA of the chunk-after-chunk kernel
#define DELTA_OUT_COLS 64          // value columns a CTA of the output kernel
#define DELTA_SPREAD 8.6736174e-19f      // 2^-60

struct DeltaArgs {
    const float* q; long long q_stride;          // [rows, groups * dk]
    const float* k; long long k_stride;
    const float* v; long long v_stride;          // [rows, heads * dv]
    const float* z; long long z_stride;          // [rows, heads * dk]: decay logits
    const float* bias;                           // [heads * dk]
    const float* rate;                           // [heads], positive
    const void* b; long long b_stride;           // [rows, heads], run type: the step sizes' logits
    float* out; long long out_stride;            // [rows, heads * dv]
    uint8_t* state; long long state_stride, state_offset;
    const int *q_start, *q_len, *slot_ids;
    int heads, groups, dk, dv;
    // scratch of the chunked form: blocks a (chunk, head), see delta_block
    float *w, *u, *qd, *kd, *p;                  // [64][LD], [tiles][64][16], [64][LD], [64][LD], [64][64]
    float *gc, *sc;                              // [DKP], [tiles][DKP][16]
    int tiles, max_chunks;                       // tiles of 16 value columns
};

// The place of chunk c of sequence seq among all chunks of the step: a sequence's chunks lie one after the other, and two
// sequences' never meet (a sequence of n rows takes ceil(n / 64) places, the next one starts at least so many further on).
__device__ __forceinline__ size_t delta_block(const DeltaArgs& a, int seq, int c, int h) {
    return (size_t)(a.q_start[seq] / DELTA_C + seq + c) * a.heads + h;
}

// a decay from its logit: exp(-rate softplus(x))
__device__ __forceinline__ float delta_decay(float x, float rate) {
    return expf(-rate * (fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)))));
}
__device__ __forceinline__ float delta_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// ------------------------------------------------------------------ token by token
// A CTA of 128 threads owns (head, sequence, a tile of value columns); a thread keeps R rows x 4 columns of S in registers,
// the RG row groups of a column lie in one warp.  The read-out of the new state is taken from the decayed one,
// S_new^T q = (g S)^T q + (k . q) u, so that a token costs one round of sums.  The state is asked for before the wait for
// the kernel's predecessor: no other kernel of a step touches it.
template <typename T, int RG, int R>
__global__ void __launch_bounds__(DELTA_WALK_THREADS)
delta_walk_kernel(DeltaArgs a) {
    constexpr int CV = DELTA_CV, CG = DELTA_WALK_THREADS / RG, DVT = CG * CV, DKP = RG * R;
    constexpr int TB = DKP <= 128 ? 8 : 4;
    constexpr int NQ = TB * DKP / DELTA_WALK_THREADS, NV = TB * DVT / DELTA_WALK_THREADS;
    static_assert((TB * DKP) % DELTA_WALK_THREADS == 0 && (TB * DVT) % DELTA_WALK_THREADS == 0, "a batch is a whole number of elements a thread");
    __shared__ __align__(16) float sq[TB * DKP], sk[TB * DKP], sa[TB * DKP], sv[TB * DVT], sb[TB];
    pdl_trigger();
    const int h = blockIdx.x, seq = blockIdx.y, dvt = blockIdx.z, tid = threadIdx.x;
    const int rg = (tid >> 1) % RG, cg = (tid & 1) | ((tid / (2 * RG)) << 1);
    const int j0 = dvt * DVT + cg * CV;
    const int n = a.q_len[seq], r0 = a.q_start[seq];
    if (n <= 0) return;
    const int dk = a.dk, dv = a.dv, g = h / (a.heads / a.groups);
    float* S_area = (float*)(a.state + (size_t)a.slot_ids[seq] * a.state_stride + a.state_offset) + (size_t)h * dk * dv;
    float s[R][CV];
#pragma unroll
    for (int e = 0; e < R; ++e)
#pragma unroll
        for (int x = 0; x < CV; ++x) {
            const int i = rg * R + e, j = j0 + x;
            s[e][x] = (i < dk && j < dv) ? S_area[(size_t)i * dv + j] : 0.f;
        }
    const float rate = a.rate[h];
    pdl_wait();
    float pq[NQ], pk[NQ], pz[NQ], pv[NV], pb = 0.f;
    auto fetch = [&](int t0) {
        const int nt = min(TB, n - t0);
#pragma unroll
        for (int w = 0; w < NQ; ++w) {
            const int idx = tid + w * DELTA_WALK_THREADS, t = idx / DKP, i = idx - t * DKP;
            const size_t row = (size_t)(r0 + t0 + t);
            const bool in = t < nt && i < dk;
            pq[w] = in ? a.q[row * a.q_stride + (size_t)g * dk + i] : 0.f;
            pk[w] = in ? a.k[row * a.k_stride + (size_t)g * dk + i] : 0.f;
            pz[w] = in ? a.z[row * a.z_stride + (size_t)h * dk + i] : 0.f;
        }
#pragma unroll
        for (int w = 0; w < NV; ++w) {
            const int idx = tid + w * DELTA_WALK_THREADS, t = idx / DVT, jj = idx - t * DVT, col = dvt * DVT + jj;
            pv[w] = (t < nt && col < dv) ? a.v[(size_t)(r0 + t0 + t) * a.v_stride + (size_t)h * dv + col] : 0.f;
        }
        if (tid < nt) pb = to_f32(((const T*)a.b)[(size_t)(r0 + t0 + tid) * a.b_stride + h]);
    };
    fetch(0);
    for (int t0 = 0; t0 < n; t0 += TB) {
        const int nt = min(TB, n - t0);
        __syncthreads();                                    // the batch before has been read
#pragma unroll
        for (int w = 0; w < NQ; ++w) {
            const int idx = tid + w * DELTA_WALK_THREADS, t = idx / DKP, i = idx - t * DKP;
            sq[idx] = pq[w];
            sk[idx] = pk[w];
            if (t < nt) sa[idx] = i < dk ? delta_decay(pz[w] + a.bias[(size_t)h * dk + i], rate) : 0.f;
        }
#pragma unroll
        for (int w = 0; w < NV; ++w) sv[tid + w * DELTA_WALK_THREADS] = pv[w];
        if (tid < nt) sb[tid] = delta_sigmoid(pb);
        if (t0 + TB < n) fetch(t0 + TB);
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            float qv[R], kv[R], av[R], vv[CV];
#pragma unroll
            for (int e = 0; e < R; e += 4) {
                *reinterpret_cast<float4*>(kv + e) = *reinterpret_cast<const float4*>(sk + t * DKP + rg * R + e);
                *reinterpret_cast<float4*>(qv + e) = *reinterpret_cast<const float4*>(sq + t * DKP + rg * R + e);
                *reinterpret_cast<float4*>(av + e) = *reinterpret_cast<const float4*>(sa + t * DKP + rg * R + e);
            }
            *reinterpret_cast<float4*>(vv) = *reinterpret_cast<const float4*>(sv + t * DVT + cg * CV);
            float sums[2 * CV + 1];
#pragma unroll
            for (int x = 0; x < 2 * CV + 1; ++x) sums[x] = 0.f;
#pragma unroll
            for (int e = 0; e < R; ++e) {
                sums[2 * CV] = fmaf(kv[e], qv[e], sums[2 * CV]);
#pragma unroll
                for (int x = 0; x < CV; ++x) {
                    s[e][x] *= av[e];
                    sums[x] = fmaf(s[e][x], kv[e], sums[x]);
                    sums[CV + x] = fmaf(s[e][x], qv[e], sums[CV + x]);
                }
            }
#pragma unroll
            for (int o = RG; o >= 2; o >>= 1)               // the row groups are lane bits 1 ...
#pragma unroll
                for (int x = 0; x < 2 * CV + 1; ++x) sums[x] += __shfl_xor_sync(0xffffffffu, sums[x], o);
            const float beta = sb[t];
            float u[CV];
#pragma unroll
            for (int x = 0; x < CV; ++x) u[x] = beta * (vv[x] - sums[x]);
#pragma unroll
            for (int e = 0; e < R; ++e)
#pragma unroll
                for (int x = 0; x < CV; ++x) s[e][x] = fmaf(kv[e], u[x], s[e][x]);
            if (rg == 0) {
                float* orow = a.out + (size_t)(r0 + t0 + t) * a.out_stride + (size_t)h * dv;
#pragma unroll
                for (int x = 0; x < CV; ++x)
                    if (j0 + x < dv) orow[j0 + x] = fmaf(sums[2 * CV], u[x], sums[CV + x]);
            }
        }
    }
#pragma unroll
    for (int e = 0; e < R; ++e)
#pragma unroll
        for (int x = 0; x < CV; ++x) {
            const int i = rg * R + e, j = j0 + x;
            if (i < dk && j < dv) S_area[(size_t)i * dv + j] = s[e][x];
        }
}

// ------------------------------------------------------------------ inside every chunk
#define DELTA_INTRA_THREADS 256
template <int DKP> constexpr int delta_intra_smem() { return (3 * DELTA_C * (DKP + 4) + DELTA_C + 3 * DKP) * 4; }

template <typename T, int DKP>
__global__ void __launch_bounds__(DELTA_INTRA_THREADS, DKP <= 128 ? 2 : 1)
delta_intra_kernel(DeltaArgs a) {
    constexpr int C = DELTA_C, SUB = DELTA_SUB, LD = DKP + 4, NT = DELTA_INTRA_THREADS;
    static_assert(DKP >= C, "A's rows fit where q's were");
    constexpr int LA = LD;
    static_assert(DKP <= NT, "a thread a channel");
    extern __shared__ __align__(16) float sm[];
    float* sK = sm;                          // k, then k over the decays up to it, then k times the decays after it
    float* sQ = sK + C * LD;                 // q, then q times the decays from its sub-chunk's edge
    float* sG = sQ + C * LD;                 // g, then k times the decays from the edge, then from the chunk's start
    float* sA = sQ;                          // beta_t A_ts, in the place of q's rows once those have been used
    float* sB = sG + C * LD;                 // beta
    float* sT = sB + C;                      // the product of a sub-chunk's decays
    float* sE = sT + DKP;                    // the product of all decays before the sub-chunk
    int* steep = (int*)(sE + DKP);           // the channels whose factors cannot be split, their number in n_steep
    __shared__ int n_steep;
    const int h = blockIdx.x, seq = blockIdx.y, c = blockIdx.z, tid = threadIdx.x;
    const int n = min(C, a.q_len[seq] - c * C), r0 = a.q_start[seq] + c * C;
    if (n <= 0) return;
    const int dk = a.dk, dv = a.dv, g = h / (a.heads / a.groups);
    const float rate = a.rate[h];
    if (tid == 0) n_steep = 0;
    pdl_wait();
#pragma unroll 8
    for (int idx = tid; idx < C * DKP; idx += NT) {
        const int t = idx / DKP, i = idx - t * DKP;
        const size_t row = (size_t)(r0 + t);
        const bool in = t < n && i < dk;
        sK[t * LD + i] = in ? a.k[row * a.k_stride + (size_t)g * dk + i] : 0.f;
        sQ[t * LD + i] = in ? a.q[row * a.q_stride + (size_t)g * dk + i] : 0.f;
        sG[t * LD + i] = in ? delta_decay(a.z[row * a.z_stride + (size_t)h * dk + i] + a.bias[(size_t)h * dk + i], rate) : 1.f;
    }
    if (tid < C) sB[tid] = tid < n ? delta_sigmoid(to_f32(((const T*)a.b)[(size_t)(r0 + tid) * a.b_stride + h])) : 0.f;
    if (tid < DKP) sE[tid] = 1.f;
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;
    const size_t block = delta_block(a, seq, c, h);
    float *gP = a.p + block * (C * C), *gQ = a.qd + block * (C * LD), *gK = a.kd + block * (C * LD);
#pragma unroll 1
    for (int J = 0; J < DELTA_NSUB; ++J) {
        const int row0 = J * SUB, t = row0 + ty;
        // a thread a channel: the factors of this sub-chunk's rows
        float e[SUB], kd[SUB];
        bool split = true;
        if (tid < DKP) {
            float prod = 1.f;
#pragma unroll
            for (int r = 0; r < SUB; ++r) {
                prod *= sG[(row0 + r) * LD + tid];
                e[r] = prod;
            }
            sT[tid] = prod;
            split = prod >= DELTA_SPREAD;
            if (split) {
#pragma unroll
                for (int r = 0; r < SUB; ++r) {
                    const int at = (row0 + r) * LD + tid;
                    const float kk = sK[at];
                    sQ[at] *= e[r];
                    sG[at] = kk * e[r];
                    sK[at] = __fdividef(kk, e[r]);
                }
            } else {
                steep[atomicAdd(&n_steep, 1)] = tid;
                float after = 1.f;
#pragma unroll
                for (int r = SUB - 1; r >= 0; --r) {
                    const int at = (row0 + r) * LD + tid;
                    kd[r] = sK[at] * after;
                    after *= sG[at];
                }
            }
        }
        __syncthreads();
        float dA = 0.f, dP = 0.f;                                   // the diagonal block's sums over the steep channels
        const int ns = n_steep;
        if (ns > 0) {
            if (tx <= ty)
                for (int w = 0; w < ns; ++w) {
                    const int i = steep[w];
                    float ks = sK[(row0 + tx) * LD + i];
                    for (int r = tx + 1; r <= ty; ++r) ks *= sG[(row0 + r) * LD + i];
                    dA = fmaf(sK[t * LD + i], ks, dA);
                    dP = fmaf(sQ[t * LD + i], ks, dP);
                }
            __syncthreads();
            if (!split) {
#pragma unroll
                for (int r = 0; r < SUB; ++r) {
                    const int at = (row0 + r) * LD + tid;
                    sQ[at] *= e[r];
                    sG[at] = sK[at] * e[r];
                    sK[at] = 0.f;
                }
            }
            if (tid == 0) n_steep = 0;
            __syncthreads();
        }
        float accA[DELTA_NSUB], accP[DELTA_NSUB];
#pragma unroll
        for (int I = 0; I < DELTA_NSUB; ++I) { accA[I] = 0.f; accP[I] = 0.f; }
        {
            const float *ra = sG + t * LD, *rq = sQ + t * LD, *rk = sK + tx * LD;
#pragma unroll 2
            for (int i = 0; i < DKP; i += 4) {
                const float4 ka = *reinterpret_cast<const float4*>(ra + i), qa = *reinterpret_cast<const float4*>(rq + i);
#pragma unroll
                for (int I = 0; I < DELTA_NSUB; ++I)
                    if (I <= J) {
                        const float4 kb = *reinterpret_cast<const float4*>(rk + I * SUB * LD + i);
                        accA[I] = fmaf(ka.x, kb.x, fmaf(ka.y, kb.y, fmaf(ka.z, kb.z, fmaf(ka.w, kb.w, accA[I]))));
                        accP[I] = fmaf(qa.x, kb.x, fmaf(qa.y, kb.y, fmaf(qa.z, kb.z, fmaf(qa.w, kb.w, accP[I]))));
                    }
            }
#pragma unroll
            for (int I = 0; I < DELTA_NSUB; ++I)
                if (I == J) { accA[I] += dA; accP[I] += dP; }
        }
#pragma unroll
        for (int I = 0; I < DELTA_NSUB; ++I)
            if (I <= J) {
                const int s = I * SUB + tx;
                gP[t * C + s] = s <= t ? accP[I] : 0.f;
            }
        __syncthreads();
        // k on to the sub-chunk's end; k and q from the chunk's start (q goes out)
        for (int idx = tid; idx < (J + 1) * SUB * DKP; idx += NT) {
            const int r = idx / DKP, i = idx - r * DKP, at = r * LD + i;
            if (r < row0) sK[at] *= sT[i];
            else {
                const float E = sE[i];
                sG[at] *= E;
                gQ[at] = sQ[at] * E;
            }
        }
        if (tid < DKP) {
#pragma unroll
            for (int r = 0; r < SUB; ++r) {
                float* at = sK + (row0 + r) * LD + tid;
                *at = split ? *at * e[SUB - 1] : kd[r];
            }
        }
        __syncthreads();
        if (tid < DKP) sE[tid] *= sT[tid];
        const float beta = sB[t];
#pragma unroll
        for (int I = 0; I < DELTA_NSUB; ++I)
            if (I <= J) {
                const int s = I * SUB + tx;
                sA[t * LA + s] = s < t ? beta * accA[I] : 0.f;
            }
        __syncthreads();
    }
    for (int idx = tid; idx < C * DKP; idx += NT) {
        const int r = idx / DKP, at = r * LD + idx - r * DKP;
        gK[at] = sK[at];
    }
    if (tid < DKP) a.gc[block * DKP + tid] = sE[tid];
    // forward substitution: a thread a column, its 64 numbers in registers
    for (int col = tid; col < DKP + a.tiles * DELTA_DVT; col += NT) {
        const bool is_w = col < DKP;
        const int vc = col - DKP;
        float x[C];
#pragma unroll
        for (int t = 0; t < C; ++t)
            x[t] = is_w ? sG[t * LD + col] : (t < n && vc < dv) ? a.v[(size_t)(r0 + t) * a.v_stride + (size_t)h * dv + vc] : 0.f;
#pragma unroll
        for (int t = 0; t < C; ++t) {
            float acc = x[t] * sB[t];
#pragma unroll
            for (int s = 0; s < t; s += 4) {                       // columns at and beyond t hold zeros
                const float4 m = *reinterpret_cast<const float4*>(sA + t * LA + s);
                acc = fmaf(-m.x, x[s], acc);
                if (s + 1 < t) acc = fmaf(-m.y, x[s + 1], acc);
                if (s + 2 < t) acc = fmaf(-m.z, x[s + 2], acc);
                if (s + 3 < t) acc = fmaf(-m.w, x[s + 3], acc);
            }
            x[t] = acc;
        }
        float* dst = is_w ? a.w + block * (C * LD) + col
                          : a.u + (block * a.tiles + vc / DELTA_DVT) * (C * DELTA_DVT) + vc % DELTA_DVT;
        const int step = is_w ? LD : DELTA_DVT;
#pragma unroll
        for (int t = 0; t < C; ++t) dst[t * step] = x[t];
    }
    pdl_trigger();
}

// ------------------------------------------------------------------ chunk after chunk
__device__ __forceinline__ void delta_cp16(void* smem, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void delta_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void delta_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
// N floats (a multiple of 4) that lie one after the other, by NT threads
template <int N, int NT>
__device__ __forceinline__ void delta_copy(float* dst, const float* src, int tid) {
#pragma unroll
    for (int u = 0; u < (N / 4 + NT - 1) / NT; ++u) {
        const int at = (tid + u * NT) * 4;
        if ((N / 4) % NT == 0 || at < N) delta_cp16(dst + at, src + at);
    }
}

// A CTA owns (head, sequence, 16 value columns) and walks the chunks.  Both products of a chunk, W S [64 x 16] and K^T U
// [DKP x 16], are cut along their inner dimension over the eight warps, so that a lane's tile is 8 x 4 (a smaller one would be
// bound by the reads of shared memory); the warps' partial tiles meet in shared memory, where the thread that owns four numbers
// of U or of S adds them up.
#define DELTA_STATE_THREADS 256
#define DELTA_ALONE_SMEM (120 * 1024)
template <int DKP> constexpr int delta_state_smem() {
    return (2 * DELTA_C * (DKP + 4) + (DKP + DELTA_C) * DELTA_DVT + 8 * DELTA_C * DELTA_DVT) * 4;
}

template <int DKP>
__global__ void __launch_bounds__(DELTA_STATE_THREADS, DKP <= 128 ? 2 : 1)
delta_state_kernel(DeltaArgs a) {
    constexpr int C = DELTA_C, LD = DKP + 4, N = DELTA_DVT, NT = DELTA_STATE_THREADS;
    constexpr int RB = DKP / 64, KS = 8 / RB;             // row blocks of S, and slices of the tokens a row block
    constexpr int KU = DKP / 8;                            // W's columns a warp
    static_assert(C * N == 4 * NT, "a thread owns four neighbouring numbers of U, and of every row block of S");
    extern __shared__ __align__(16) float sm[];
    float* sW = sm;                          // [C][LD]
    float* sK = sW + C * LD;                 // [C][LD]
    float* sS = sK + C * LD;                 // [DKP][16]
    float* sU = sS + DKP * N;                // [C][16]
    float* sP = sU + C * N;                  // [8 warps][64][16]
    const int h = blockIdx.x, seq = blockIdx.y, tile = blockIdx.z, tid = threadIdx.x;
    const int warp = tid >> 5, lr = (tid & 31) >> 2, lc = tid & 3;
    const int n_all = a.q_len[seq];
    if (n_all <= 0) return;
    const int dk = a.dk, dv = a.dv, n_chunks = (n_all + C - 1) / C;
    const int own = tid * 4, own_p = own / N, own_c = own % N, j0 = tile * N + own_c;
    // the rows of S a thread owns: partial tiles hold row lr * 8 + e at place e * 8 + lr
    const int own_i = (own_p & 7) * 8 + (own_p >> 3);
    float* S_area = (float*)(a.state + (size_t)a.slot_ids[seq] * a.state_stride + a.state_offset) + (size_t)h * dk * dv;
    float s[RB][4];
#pragma unroll
    for (int b = 0; b < RB; ++b) {
        const int i = b * 64 + own_i;
#pragma unroll
        for (int x = 0; x < 4; ++x) s[b][x] = (i < dk && j0 + x < dv) ? S_area[(size_t)i * dv + j0 + x] : 0.f;
        *reinterpret_cast<float4*>(sS + i * N + own_c) = make_float4(s[b][0], s[b][1], s[b][2], s[b][3]);
    }
    pdl_wait();
    const size_t block0 = delta_block(a, seq, 0, h), step = a.heads;      // block of chunk c: block0 + c * step
    float4 u0;
    float gn[RB];
    auto ahead = [&](int c) {                               // what the owners need of chunk c
        const size_t blk = block0 + c * step;
        u0 = *reinterpret_cast<const float4*>(a.u + (blk * a.tiles + tile) * (C * N) + own);
#pragma unroll
        for (int b = 0; b < RB; ++b) gn[b] = a.gc[blk * DKP + b * 64 + own_i];
    };
    delta_copy<C * LD, NT>(sW, a.w + block0 * (C * LD), tid);
    delta_cp_commit();
    delta_copy<C * LD, NT>(sK, a.kd + block0 * (C * LD), tid);
    delta_cp_commit();
    ahead(0);
    for (int c = 0; c < n_chunks; ++c) {
        const size_t blk = block0 + c * step;
        const bool more = c + 1 < n_chunks;
        // the state that this chunk starts from, for the output kernel
        float* sc = a.sc + (blk * a.tiles + tile) * (DKP * N);
#pragma unroll
        for (int b = 0; b < RB; ++b)
            *reinterpret_cast<float4*>(sc + (b * 64 + own_i) * N + own_c) = make_float4(s[b][0], s[b][1], s[b][2], s[b][3]);
        delta_cp_wait<1>();                                 // this chunk's W
        __syncthreads();
        {
            float acc[8][4];
#pragma unroll
            for (int e = 0; e < 8; ++e)
#pragma unroll
                for (int x = 0; x < 4; ++x) acc[e][x] = 0.f;
            const float *w0 = sW + lr * LD + warp * KU, *s0 = sS + warp * KU * N + lc * 4;
#pragma unroll
            for (int i = 0; i < KU; i += 4) {
                float sv[4][4];
#pragma unroll
                for (int d = 0; d < 4; ++d) *reinterpret_cast<float4*>(sv[d]) = *reinterpret_cast<const float4*>(s0 + (i + d) * N);
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    float wv[4];
                    *reinterpret_cast<float4*>(wv) = *reinterpret_cast<const float4*>(w0 + e * 8 * LD + i);
#pragma unroll
                    for (int d = 0; d < 4; ++d)
#pragma unroll
                        for (int x = 0; x < 4; ++x) acc[e][x] = fmaf(wv[d], sv[d][x], acc[e][x]);
                }
            }
            float* part = sP + warp * (C * N) + lr * N + lc * 4;
#pragma unroll
            for (int e = 0; e < 8; ++e) *reinterpret_cast<float4*>(part + e * 8 * N) = make_float4(acc[e][0], acc[e][1], acc[e][2], acc[e][3]);
        }
        __syncthreads();                                    // W and S have been read, the partial tiles are there
        if (more) delta_copy<C * LD, NT>(sW, a.w + (blk + step) * (C * LD), tid);
        delta_cp_commit();
        {
            float4 u = u0;
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                const float4 q = *reinterpret_cast<const float4*>(sP + w * (C * N) + own);
                u.x -= q.x; u.y -= q.y; u.z -= q.z; u.w -= q.w;
            }
            *reinterpret_cast<float4*>(sU + own) = u;
            *reinterpret_cast<float4*>(a.u + (blk * a.tiles + tile) * (C * N) + own) = u;
        }
#pragma unroll
        for (int b = 0; b < RB; ++b)
#pragma unroll
            for (int x = 0; x < 4; ++x) s[b][x] *= gn[b];
        if (more) ahead(c + 1);
        delta_cp_wait<1>();                                 // this chunk's k
        __syncthreads();
        {
            float acc[8][4];
#pragma unroll
            for (int e = 0; e < 8; ++e)
#pragma unroll
                for (int x = 0; x < 4; ++x) acc[e][x] = 0.f;
            const int rb = warp % RB, ks = warp / RB;
            const float *k0 = sK + (ks * (C / KS)) * LD + rb * 64 + lr * 8, *v0 = sU + (ks * (C / KS)) * N + lc * 4;
#pragma unroll 4
            for (int t = 0; t < C / KS; ++t) {
                float kv[8], uv[4];
                *reinterpret_cast<float4*>(kv) = *reinterpret_cast<const float4*>(k0 + t * LD);
                *reinterpret_cast<float4*>(kv + 4) = *reinterpret_cast<const float4*>(k0 + t * LD + 4);
                *reinterpret_cast<float4*>(uv) = *reinterpret_cast<const float4*>(v0 + t * N);
#pragma unroll
                for (int e = 0; e < 8; ++e)
#pragma unroll
                    for (int x = 0; x < 4; ++x) acc[e][x] = fmaf(kv[e], uv[x], acc[e][x]);
            }
            float* part = sP + (rb * KS + ks) * (64 * N) + lr * N + lc * 4;
#pragma unroll
            for (int e = 0; e < 8; ++e) *reinterpret_cast<float4*>(part + e * 8 * N) = make_float4(acc[e][0], acc[e][1], acc[e][2], acc[e][3]);
        }
        __syncthreads();                                    // k and U have been read, the partial tiles are there
        if (more) delta_copy<C * LD, NT>(sK, a.kd + (blk + step) * (C * LD), tid);
        delta_cp_commit();
#pragma unroll
        for (int b = 0; b < RB; ++b) {
#pragma unroll
            for (int w = 0; w < KS; ++w) {
                const float4 q = *reinterpret_cast<const float4*>(sP + (b * KS + w) * (64 * N) + own);
                s[b][0] += q.x; s[b][1] += q.y; s[b][2] += q.z; s[b][3] += q.w;
            }
            *reinterpret_cast<float4*>(sS + (b * 64 + own_i) * N + own_c) = make_float4(s[b][0], s[b][1], s[b][2], s[b][3]);
        }
    }
    pdl_trigger();
    delta_cp_wait<0>();
#pragma unroll
    for (int b = 0; b < RB; ++b)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = b * 64 + own_i;
            if (i < dk && j0 + x < dv) S_area[(size_t)i * dv + j0 + x] = s[b][x];
        }
}

// ------------------------------------------------------------------ outputs of every chunk
// A CTA owns 64 tokens x 64 value columns of one (chunk, head); a lane's tile is 8 x 4.
#define DELTA_OUT_THREADS 128
template <int DKP> constexpr int delta_out_smem() {
    return (DELTA_C * (DKP + 4) + DKP * (DELTA_OUT_COLS + 4) + DELTA_C * (DELTA_C + 4) + DELTA_C * (DELTA_OUT_COLS + 4)) * 4;
}

template <int DKP>
__global__ void __launch_bounds__(DELTA_OUT_THREADS)
delta_out_kernel(DeltaArgs a) {
    constexpr int C = DELTA_C, LD = DKP + 4, LS = DELTA_OUT_COLS + 4, LP = C + 4, NT = DELTA_OUT_THREADS, N = DELTA_DVT;
    extern __shared__ __align__(16) float sm[];
    float* sQ = sm;                          // [C][LD]
    float* sS = sQ + C * LD;                 // [DKP][LS]
    float* sP = sS + DKP * LS;               // [C][LP]
    float* sU = sP + C * LP;                 // [C][LS]
    pdl_trigger();
    const int spans = (a.tiles * N + DELTA_OUT_COLS - 1) / DELTA_OUT_COLS;
    const int h = blockIdx.x, seq = blockIdx.y, c = blockIdx.z / spans, col0 = (blockIdx.z - c * spans) * DELTA_OUT_COLS, tid = threadIdx.x;
    const int n = min(C, a.q_len[seq] - c * C), r0 = a.q_start[seq] + c * C;
    if (n <= 0) return;
    const size_t block = delta_block(a, seq, c, h);
    const int tile0 = col0 / N, tiles = min(DELTA_OUT_COLS / N, a.tiles - tile0);
    pdl_wait();
    delta_copy<C * LD, NT>(sQ, a.qd + block * (C * LD), tid);
    const float *sc = a.sc + (block * a.tiles + tile0) * (DKP * N), *gu = a.u + (block * a.tiles + tile0) * (C * N), *gp = a.p + block * (C * C);
    for (int w = 0; w < tiles; ++w) {
#pragma unroll 4
        for (int idx = tid; idx < DKP * (N / 4); idx += NT) delta_cp16(sS + (idx / (N / 4)) * LS + w * N + (idx % (N / 4)) * 4, sc + w * (DKP * N) + idx * 4);
#pragma unroll
        for (int idx = tid; idx < C * (N / 4); idx += NT) delta_cp16(sU + (idx / (N / 4)) * LS + w * N + (idx % (N / 4)) * 4, gu + w * (C * N) + idx * 4);
    }
    for (int idx = tid; idx < C * (C / 4); idx += NT) {
        const int t = idx / (C / 4), s = (idx % (C / 4)) * 4;
        if (s / DELTA_SUB <= t / DELTA_SUB) delta_cp16(sP + t * LP + s, gp + idx * 4);       // the blocks beyond were not written
    }
    delta_cp_commit();
    delta_cp_wait<0>();
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;                // rows r * 8 + ty, columns tx * 4 ...
    float o[8][4];
#pragma unroll
    for (int r = 0; r < 8; ++r)
#pragma unroll
        for (int x = 0; x < 4; ++x) o[r][x] = 0.f;
    if (tx * 4 < tiles * N) {
#pragma unroll 2
        for (int i = 0; i < DKP; i += 4) {
            float sv[4][4];
#pragma unroll
            for (int e = 0; e < 4; ++e) *reinterpret_cast<float4*>(sv[e]) = *reinterpret_cast<const float4*>(sS + (i + e) * LS + tx * 4);
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                float mv[4];
                *reinterpret_cast<float4*>(mv) = *reinterpret_cast<const float4*>(sQ + (r * 8 + ty) * LD + i);
#pragma unroll
                for (int e = 0; e < 4; ++e)
#pragma unroll
                    for (int x = 0; x < 4; ++x) o[r][x] = fmaf(mv[e], sv[e][x], o[r][x]);
            }
        }
        // P is lower triangular: 16 keys at a time, the rows of earlier sub-chunks stay out
#pragma unroll
        for (int I = 0; I < DELTA_NSUB; ++I)
#pragma unroll 2
            for (int s = I * DELTA_SUB; s < (I + 1) * DELTA_SUB; s += 4) {
                float uv[4][4];
#pragma unroll
                for (int e = 0; e < 4; ++e) *reinterpret_cast<float4*>(uv[e]) = *reinterpret_cast<const float4*>(sU + (s + e) * LS + tx * 4);
#pragma unroll
                for (int r = 2 * I; r < 8; ++r) {
                    float mv[4];
                    *reinterpret_cast<float4*>(mv) = *reinterpret_cast<const float4*>(sP + (r * 8 + ty) * LP + s);
#pragma unroll
                    for (int e = 0; e < 4; ++e)
#pragma unroll
                        for (int x = 0; x < 4; ++x) o[r][x] = fmaf(mv[e], uv[e][x], o[r][x]);
                }
            }
    }
#pragma unroll
    for (int r = 0; r < 8; ++r) {
        const int t = r * 8 + ty;
        if (t >= n) continue;
        float* orow = a.out + (size_t)(r0 + t) * a.out_stride + (size_t)h * a.dv;
#pragma unroll
        for (int x = 0; x < 4; ++x)
            if (col0 + tx * 4 + x < a.dv) orow[col0 + tx * 4 + x] = o[r][x];
    }
}

// ------------------------------------------------------------------ host side
static int delta_dkp(int dk) { return dk <= 64 ? 64 : dk <= 128 ? 128 : 256; }
static long long delta_blocks(int rows, int n_seqs, int heads) { return ((long long)rows / DELTA_C + n_seqs + 1) * heads; }

// Floats of scratch that the chunked form of a step needs.
extern "C" long long braid_delta_work_floats(int rows, int n_seqs, int heads, int dk, int dv) {
    const long long dkp = delta_dkp(dk), dvp = (dv + DELTA_DVT - 1) / DELTA_DVT * DELTA_DVT;
    return delta_blocks(rows, n_seqs, heads) * (3 * DELTA_C * (dkp + 4) + DELTA_C * dvp + DELTA_C * DELTA_C + dkp + dkp * dvp);
}

template <typename T, int DKP>
static int launch_delta_chunks(const DeltaArgs& a, int n_seqs, cudaStream_t s) {
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(delta_intra_kernel<T, DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize, delta_intra_smem<DKP>());
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_state_kernel<DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                         delta_state_smem<DKP>() > DELTA_ALONE_SMEM ? delta_state_smem<DKP>() : DELTA_ALONE_SMEM);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_out_kernel<DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize, delta_out_smem<DKP>());
        if (e != cudaSuccess) { braid_set_error("delta_rule: cannot reserve shared memory: %s", cudaGetErrorString(e)); return (int)e; }
        configured = true;
    }
    const int spans = (a.tiles * DELTA_DVT + DELTA_OUT_COLS - 1) / DELTA_OUT_COLS;
    braid_launch(delta_intra_kernel<T, DKP>, dim3(a.heads, n_seqs, a.max_chunks), dim3(DELTA_INTRA_THREADS), delta_intra_smem<DKP>(), s, a);
    // where one CTA an SM covers the step, each asks for more than half of an SM's shared memory: launched while the kernel before
    // drains, they would otherwise settle two and more on the SMs that are free first (8 heads of 128 x 256: 287 -> 220 us in all)
    const bool alone = (long long)a.heads * n_seqs * a.tiles <= 148;
    const int state_smem = alone && delta_state_smem<DKP>() < DELTA_ALONE_SMEM ? DELTA_ALONE_SMEM : delta_state_smem<DKP>();
    braid_launch(delta_state_kernel<DKP>, dim3(a.heads, n_seqs, a.tiles), dim3(DELTA_STATE_THREADS), state_smem, s, a);
    braid_launch(delta_out_kernel<DKP>, dim3(a.heads, n_seqs, a.max_chunks * spans), dim3(DELTA_OUT_THREADS), delta_out_smem<DKP>(), s, a);
    BRAID_LAUNCH_CHECK();
}

template <typename T>
static int launch_delta(const DeltaArgs& a, int n_seqs, bool chunked, cudaStream_t s) {
    if (chunked) {
        if (a.dk <= 64) return launch_delta_chunks<T, 64>(a, n_seqs, s);
        if (a.dk <= 128) return launch_delta_chunks<T, 128>(a, n_seqs, s);
        return launch_delta_chunks<T, 256>(a, n_seqs, s);
    }
    const int rg = a.dk <= 32 ? 4 : a.dk <= 64 ? 8 : 16;
    const int dvt = (DELTA_WALK_THREADS / rg) * DELTA_CV;
    const dim3 grid(a.heads, n_seqs, (a.dv + dvt - 1) / dvt), block(DELTA_WALK_THREADS);
    if (rg == 4) braid_launch(delta_walk_kernel<T, 4, 8>, grid, block, 0, s, a);
    else if (rg == 8) braid_launch(delta_walk_kernel<T, 8, 8>, grid, block, 0, s, a);
    else if (a.dk <= 128) braid_launch(delta_walk_kernel<T, 16, 8>, grid, block, 0, s, a);
    else braid_launch(delta_walk_kernel<T, 16, 16>, grid, block, 0, s, a);
    BRAID_LAUNCH_CHECK();
}

// `work`: braid_delta_work_floats floats, on 16 bytes, for the chunked form; null: token by token.
extern "C" int braid_delta_rule(const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                                long long v_stride, const float* z, long long z_stride, const float* bias, const float* rate,
                                const void* b, long long b_stride, int dtype, float* out, long long out_stride, void* state,
                                long long state_stride, long long state_offset, const int* q_start, const int* q_len,
                                const int* slot_ids, int rows, int n_seqs, int max_q_len, int heads, int groups, int dk, int dv,
                                float* work, long long work_floats, void* stream) {
    if (n_seqs <= 0 || rows <= 0 || max_q_len <= 0) return BRAID_OK;
    if (heads <= 0 || groups <= 0 || heads % groups) BRAID_REFUSE("delta_rule: %d heads do not divide into %d groups", heads, groups);
    if (dk <= 0 || dk > DELTA_MAX_DK || dv <= 0) BRAID_REFUSE("delta_rule: key size %d must be in (0, %d], value size %d positive", dk, DELTA_MAX_DK, dv);
    if (!state || (state_offset & 3) || (state_stride & 3)) BRAID_REFUSE("delta_rule: the state area must be given, in multiples of 4 bytes");
    if (dtype != BRAID_F32 && dtype != BRAID_BF16) BRAID_REFUSE("delta_rule: unknown dtype code %d", dtype);
    DeltaArgs a{q, q_stride, k, k_stride, v, v_stride, z, z_stride, bias, rate, b, b_stride, out, out_stride, (uint8_t*)state,
                state_stride, state_offset, q_start, q_len, slot_ids, heads, groups, dk, dv,
                nullptr, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr, (dv + DELTA_DVT - 1) / DELTA_DVT,
                (max_q_len + DELTA_C - 1) / DELTA_C};
    const long long spans = (a.tiles * DELTA_DVT + DELTA_OUT_COLS - 1) / DELTA_OUT_COLS;
    if (n_seqs > 65535 || a.tiles > 65535 || (work && a.max_chunks * spans > 65535)) BRAID_REFUSE("delta_rule: the step exceeds the grid limits");
    if (work) {
        const long long need = braid_delta_work_floats(rows, n_seqs, heads, dk, dv);
        if (need > work_floats || ((uintptr_t)work & 15)) BRAID_REFUSE("delta_rule: the chunked form needs %lld floats of scratch on 16 bytes, it was given %lld", need, work_floats);
        const long long blocks = delta_blocks(rows, n_seqs, heads), dkp = delta_dkp(dk), wide = blocks * DELTA_C * (dkp + 4);
        a.w = work;
        a.qd = a.w + wide;
        a.kd = a.qd + wide;
        a.u = a.kd + wide;
        a.p = a.u + blocks * a.tiles * DELTA_C * DELTA_DVT;
        a.gc = a.p + blocks * DELTA_C * DELTA_C;
        a.sc = a.gc + blocks * dkp;
    }
    if (dtype == BRAID_F32) return launch_delta<float>(a, n_seqs, work != nullptr, (cudaStream_t)stream);
    return launch_delta<__nv_bfloat16>(a, n_seqs, work != nullptr, (cudaStream_t)stream);
}

// The read-out's norm and gate (gated_norm.cuh), the gate's logits in float32.
extern "C" int braid_delta_gated_norm(const float* y, const float* gate, long long gate_stride, const void* w, int w_len, void* out,
                                      long long out_stride, const int* token_seq, int dtype, int rows, int width, int group,
                                      float eps, void* stream) {
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == BRAID_F32)
        return gated_norm_launch(y, gate, gate_stride, (const float*)w, w_len, (float*)out, out_stride, token_seq, rows, width, group, 0, 1, eps, 1.f, s);
    if (dtype == BRAID_BF16)
        return gated_norm_launch(y, gate, gate_stride, (const __nv_bfloat16*)w, w_len, (__nv_bfloat16*)out, out_stride, token_seq, rows, width, group, 0, 1, eps, 1.f, s);
    BRAID_REFUSE("gated_norm: unknown dtype code %d", dtype);
}
