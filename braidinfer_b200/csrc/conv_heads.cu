// A short causal convolution over time on projected heads, and what the heads need right after it, in one kernel:
//     u_t = x_t + bias                                        (x: projected rows in the run's type, bias optional)
//     y_t[c] = sum_j w[c, j] u_(t - taps + 1 + j)[c]          (zeros before the sequence's start)
// then, head by head, silu, a norm (root mean square with a weight of the head's size; or unit length,
// y / sqrt(sum y^2 + eps)), a constant factor, a rotation of the head's first numbers (neighbouring pairs, or halves), zeros
// up to a padded head size, and the store: rows of a buffer (float32 or the run's type), or the key or value plane of the
// paged cache at the token's position.
//
// The channels fall into up to three segments (queries, keys, values), each with heads of its own size and its own choice
// of these.  A sequence's state is its last taps - 1 rows u, float32 [taps - 1][channels] at state + slot * state_stride +
// state_offset, the newest last, zero at the start: rows before the step come from there.  A sequence that brings one token
// has its state moved on by the threads that read it; the others by conv_heads_state_kernel.  Everything is float32
// arithmetic.
#include "common.cuh"

#define CONV_MAX_SEGS 3
#define CONV_NORM_NONE 0
#define CONV_NORM_RMS 1
#define CONV_NORM_UNIT 2
#define CONV_MAX_SIZE 512

struct ConvSegment {
    int heads, size, pad;        // heads of `size` channels, written as heads of `pad` numbers
    int norm, silu, rotate;
    int plane;                   // -1: to `out`; 0, 1: the cache's key or value plane
    float factor;
    float inv_count;             // 1 / size for CONV_NORM_RMS, else 1
    const void* weight;          // CONV_NORM_RMS: [size] in the run's type
    void* out;                   // [rows, out_stride], head h at column h * pad
    long long out_stride;
};

struct ConvHeadsArgs {
    const void* x;               // [rows, x_stride]: segment after segment, head after head
    long long x_stride;
    const void* bias;            // [channels] or null
    const void* w;               // [channels, taps]
    uint8_t* state;              // null with one tap
    long long state_stride, state_offset;
    const int *token_seq, *positions, *q_start, *q_len, *slot_ids;
    const int* page_table;       // [n_seqs, table_cols]
    void* cache;                 // one layer: [page][2][kv heads][page_size][pad], or null
    int page_size, table_cols, num_pages;
    const float* inv_freq;       // [rope_dim / 2]
    int rope_dim, adjacent;
    float amp, eps;
    int rows, channels, taps, n_segs, turns;     // turns: some segment is rotated
    int* error_flag;
    ConvSegment seg[CONV_MAX_SEGS];
};

// Where head `h` of segment s and row `row` is stored (its first number), or null.
template <typename T, typename TO>
__device__ __forceinline__ TO* conv_dst(const ConvHeadsArgs& a, const ConvSegment& s, int h, int row, int seq, int pos, bool flag) {
    if (s.plane < 0) return (TO*)s.out + (size_t)row * s.out_stride + (size_t)h * s.pad;
    if (!a.cache) return nullptr;
    const int block = pos / a.page_size, off = pos - block * a.page_size;
    const int page = (block < a.table_cols) ? a.page_table[(size_t)seq * a.table_cols + block] : -1;
    if (page < 0 || page >= a.num_pages) {
        if (flag) atomicExch(a.error_flag, 1);
        return nullptr;
    }
    return (TO*)a.cache + ((((size_t)page * 2 + s.plane) * s.heads + h) * a.page_size + off) * s.pad;
}

// ---- 16 bytes of neighbouring channels a thread, LPH lanes a head: for sizes, strides and taps that allow it (neighbouring
// pairs in the rotation).  TO: the type of what is stored.
#define CONV_MAX_PAIRS 128

// A thread's place among the segments' channels.
struct ConvPlace {
    ConvSegment s;
    int head, c0, i0, l;         // head of the segment, first channel of all, of the head, lane of the head
    bool live, in;               // a head at all; channels of one
};
template <typename T, int LPH>
__device__ __forceinline__ ConvPlace conv_place(const ConvHeadsArgs& a) {
    constexpr int VEC = 16 / sizeof(T), HPC = 128 / LPH;
    ConvPlace p;
    int c_seg = 0;
    p.l = threadIdx.x % LPH;
    p.i0 = p.l * VEC;
    p.head = blockIdx.x * HPC + threadIdx.x / LPH;         // the segments' heads are counted through
    p.s = a.seg[0];
#pragma unroll
    for (int si = 1; si < CONV_MAX_SEGS; ++si)
        if (si < a.n_segs && p.head >= p.s.heads) {
            p.head -= p.s.heads;
            c_seg += p.s.heads * p.s.size;
            p.s = a.seg[si];
        }
    p.live = p.head < p.s.heads;
    p.in = p.live && p.i0 < p.s.size;
    p.c0 = c_seg + p.head * p.s.size + p.i0;
    return p;
}

// The taps and biases of a thread's channels.
template <typename T, int TAPS, int VEC>
__device__ __forceinline__ void conv_weights(const ConvHeadsArgs& a, const ConvPlace& p, float* wl, float* bl) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) bl[e] = 0.f;
#pragma unroll
    for (int e = 0; e < VEC * TAPS; ++e) wl[e] = 0.f;
    if (!p.in) return;
#pragma unroll
    for (int u = 0; u < TAPS; ++u) load_run<T, VEC>((const T*)a.w + (size_t)p.c0 * TAPS + u * VEC, wl + u * VEC);
    if (a.bias) load_run<T, VEC>((const T*)a.bias + p.c0, bl);
}

// silu, norm, rotation and store of one row's channels; the whole warp calls.  `turn`: the row's sines and cosines.
template <typename T, typename TO, int LPH, int VEC>
__device__ __forceinline__ void conv_finish(const ConvHeadsArgs& a, const ConvPlace& p, float* y, const float2* turn, TO* dst) {
    if (p.s.silu) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = sizeof(T) == 2 ? glu_act_fast(y[e], BRAID_ACT_SILU) : silu_f32(y[e]);
    }
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(y[e], y[e], ss);
#pragma unroll
    for (int b = LPH / 2; b > 0; b >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, b);       // whatever the lanes' segments
    if (p.s.norm != CONV_NORM_NONE) {
        const float m = ss * p.s.inv_count + a.eps;
        const float r = p.s.factor * (sizeof(T) == 2 ? rsqrtf(m) : 1.f / sqrtf(m));
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] *= r;
        if (p.in && p.s.norm == CONV_NORM_RMS) {
            float nw[VEC];
            load_run<T, VEC>((const T*)p.s.weight + p.i0, nw);
#pragma unroll
            for (int e = 0; e < VEC; ++e) y[e] *= nw[e];
        }
    } else if (p.s.factor != 1.f) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] *= p.s.factor;
    }
    if (!dst || p.i0 >= p.s.pad) return;
    if (p.s.rotate && p.i0 < a.rope_dim) {
#pragma unroll
        for (int e = 0; e < VEC; e += 2) {
            const int k = (p.i0 + e) >> 1;
            if (2 * k < a.rope_dim) {
                const float2 t = turn[k];
                const float u = y[e], v = y[e + 1];
                y[e] = u * t.y - v * t.x;
                y[e + 1] = v * t.y + u * t.x;
            }
        }
    }
    constexpr int VO = 16 / sizeof(TO) < VEC ? 16 / sizeof(TO) : VEC;
#pragma unroll
    for (int e = 0; e < VEC; e += VO) store_run<TO, VO>(dst + p.i0 + e, y + e);
}

// One row whose taps may reach before the step: every tap's row is looked up, in the step or in the state.  `st` is the row's
// sequence's state; with `move` (a sequence of one token, whose channels nobody else reads) it takes the new row.
template <typename T, int TAPS, int VEC>
__device__ __forceinline__ void conv_row(const ConvHeadsArgs& a, const ConvPlace& p, const float* wl, const float* bl, int row, int o, float* st,
                                         bool move, float* y) {
    float u[TAPS][VEC];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
        const int back = TAPS - 1 - j;
        if (o - back >= 0) {
            load_run<T, VEC>((const T*)a.x + (size_t)(row - back) * a.x_stride + p.c0, u[j]);
#pragma unroll
            for (int e = 0; e < VEC; ++e) u[j][e] += bl[e];
        } else {
            const float* sp = st + (size_t)(TAPS - 1 + (o - back)) * a.channels + p.c0;
#pragma unroll
            for (int e = 0; e < VEC; e += 4) load_run<float, 4>(sp + e, u[j] + e);
        }
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(wl[e * TAPS + j], u[j][e], y[e]);
    if (move) {
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
            for (int e = 0; e < VEC; e += 4) store_run<float, 4>(st + (size_t)k * a.channels + p.c0 + e, u[k + 1] + e);
    }
}

// Sines and cosines of rows row0 .. row0 + n - 1, by the whole CTA; their positions are pos0 and on, or (pos0 < 0) looked up.
__device__ __forceinline__ void conv_turns(const ConvHeadsArgs& a, int row0, int n, int pos0, float2 (*turn)[CONV_MAX_PAIRS]) {
    const int half = a.rope_dim / 2;
    for (int idx = threadIdx.x; idx < n * half; idx += 128) {
        const int r = idx / half, k = idx - r * half;
        const int ps = pos0 >= 0 ? pos0 + r : row0 + r < a.rows ? a.positions[row0 + r] : 0;
        float sn, cs;
        sincosf((float)ps * a.inv_freq[k], &sn, &cs);
        turn[r][k] = make_float2(sn * a.amp, cs * a.amp);
    }
}

// Few rows: one a CTA.
template <typename T, typename TO, int TAPS, int LPH>
__global__ void __launch_bounds__(128)
conv_heads_row_kernel(ConvHeadsArgs a) {
    constexpr int VEC = 16 / sizeof(T);
    __shared__ float2 turn[1][CONV_MAX_PAIRS];
    pdl_trigger();
    const ConvPlace p = conv_place<T, LPH>(a);
    const int row = blockIdx.y;
    // the step's tables are on the device before its first kernel: read before the wait
    const int seq = a.token_seq[row];
    if (seq < 0) return;
    const int o = row - a.q_start[seq];
    const bool move = TAPS > 1 && a.q_len[seq] == 1;
    float* st = a.state ? (float*)(a.state + (size_t)a.slot_ids[seq] * a.state_stride + a.state_offset) : nullptr;
    TO* dst = p.live ? conv_dst<T, TO>(a, p.s, p.head, row, seq, a.positions[row], p.l == 0) : nullptr;
    if (a.turns) {
        conv_turns(a, row, 1, -1, turn);
        __syncthreads();
    }
    float wl[VEC * TAPS], bl[VEC], y[VEC];
    conv_weights<T, TAPS, VEC>(a, p, wl, bl);
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = 0.f;
    pdl_wait();
    if (p.in) conv_row<T, TAPS, VEC>(a, p, wl, bl, row, o, st, move, y);
    conv_finish<T, TO, LPH, VEC>(a, p, y, turn[0], dst);
}

// Many rows: a CTA walks `span` neighbouring rows, four at a time, the next four on their way.  Where four rows and what their
// taps reach lie inside one sequence's step (nearly everywhere), every row is loaded and converted once, the window of rows
// moves along, and the bias comes through the sum of the taps.
#define CONV_RPT 4
template <typename T, typename TO, int TAPS, int LPH>
__global__ void __launch_bounds__(128, 3)
conv_heads_span_kernel(ConvHeadsArgs a, int span) {
    constexpr int VEC = 16 / sizeof(T), R = CONV_RPT;
    __shared__ float2 turn[2][R][CONV_MAX_PAIRS];
    pdl_trigger();
    const ConvPlace p = conv_place<T, LPH>(a);
    const int begin = blockIdx.y * span, end = min(a.rows, begin + span);
    float wl[VEC * TAPS], bl[VEC], yb[VEC];
    conv_weights<T, TAPS, VEC>(a, p, wl, bl);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) sum += wl[e * TAPS + j];
        yb[e] = sum * bl[e];
    }
    int first = a.token_seq[begin], last = a.token_seq[min(begin + R, end) - 1], known = -1, q0 = 0, p0 = 0;
    pdl_wait();
    const T* x = (const T*)a.x + p.c0;
    uint4 next[R];
    auto ask = [&](int row0) {
#pragma unroll
        for (int r = 0; r < R; ++r)
            next[r] = p.in && row0 + r < end ? *reinterpret_cast<const uint4*>(x + (size_t)(row0 + r) * a.x_stride) : make_uint4(0, 0, 0, 0);
    };
    ask(begin);
    float win[TAPS][VEC];                                  // row begin - (TAPS - 1) + u at place u % TAPS
    bool fresh = true;                                     // the window is still to be filled from the rows before
    int buf = 0;
    for (int row0 = begin; row0 < end; row0 += R) {
        uint4 cur[R];
#pragma unroll
        for (int r = 0; r < R; ++r) cur[r] = next[r];
        const int seq = first;
        const bool one = seq >= 0 && seq == last && row0 + R <= end;
        if (row0 + R < end) {
            ask(row0 + R);
            first = a.token_seq[row0 + R];
            last = a.token_seq[min(row0 + 2 * R, end) - 1];
        }
        if (one && seq != known) {                         // where the sequence's rows start, and its position there
            known = seq;
            q0 = a.q_start[seq];
            p0 = a.positions[q0];
        }
        const bool inner = one && row0 - q0 >= TAPS - 1;
        const int pos0 = p0 + row0 - q0;
        if (a.turns) {
            conv_turns(a, row0, R, inner ? pos0 : -1, turn[buf]);
            __syncthreads();                               // two tables take turns: one barrier a round is enough
        }
        if (inner) {
            TO* dst[R];
#pragma unroll
            for (int r = 0; r < R; ++r) dst[r] = p.live ? conv_dst<T, TO>(a, p.s, p.head, row0 + r, seq, pos0 + r, p.l == 0) : nullptr;
            if (fresh) {
#pragma unroll
                for (int u = 0; u < TAPS - 1; ++u) {
                    if (p.in) load_run<T, VEC>(x + (size_t)(row0 - (TAPS - 1) + u) * a.x_stride, win[u]);
                    else
#pragma unroll
                        for (int e = 0; e < VEC; ++e) win[u][e] = 0.f;
                }
                fresh = false;
            }
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const T* c = reinterpret_cast<const T*>(&cur[r]);
#pragma unroll
                for (int e = 0; e < VEC; ++e) win[TAPS - 1][e] = to_f32(c[e]);
                float y[VEC];
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    y[e] = yb[e];
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) y[e] = fmaf(wl[e * TAPS + j], win[j][e], y[e]);
                }
                conv_finish<T, TO, LPH, VEC>(a, p, y, turn[buf][r], dst[r]);
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) win[j][e] = win[j + 1][e];
            }
        } else {
            fresh = true;
#pragma unroll 1
            for (int r = 0; r < R && row0 + r < end; ++r) {
                const int row = row0 + r, sq = a.token_seq[row];
                if (sq < 0) continue;
                float* st = a.state ? (float*)(a.state + (size_t)a.slot_ids[sq] * a.state_stride + a.state_offset) : nullptr;
                TO* dst = p.live ? conv_dst<T, TO>(a, p.s, p.head, row, sq, a.positions[row], p.l == 0) : nullptr;
                float y[VEC];
#pragma unroll
                for (int e = 0; e < VEC; ++e) y[e] = 0.f;
                if (p.in) conv_row<T, TAPS, VEC>(a, p, wl, bl, row, row - a.q_start[sq], st, false, y);
                conv_finish<T, TO, LPH, VEC>(a, p, y, turn[buf][r], dst);
            }
        }
        buf ^= 1;
    }
}

// Any sizes, taps and pairing: a warp a (row, head), lane-strided pairs of channels.
#define CONV_ANY_WARPS 4
template <typename T, typename TO>
__global__ void __launch_bounds__(CONV_ANY_WARPS * 32)
conv_heads_kernel(ConvHeadsArgs a) {
    __shared__ float stage[CONV_ANY_WARPS][CONV_MAX_SIZE];
    pdl_trigger();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int h = blockIdx.x * CONV_ANY_WARPS + warp, si = 0, c_seg = 0;
    for (; si < a.n_segs; ++si) {
        if (h < a.seg[si].heads) break;
        h -= a.seg[si].heads;
        c_seg += a.seg[si].heads * a.seg[si].size;
    }
    if (si == a.n_segs) return;
    const ConvSegment& s = a.seg[si];
    const int row = blockIdx.y, seq = a.token_seq[row];
    if (seq < 0) return;
    const int o = row - a.q_start[seq], c0 = c_seg + h * s.size;
    float* st = a.state ? (float*)(a.state + (size_t)a.slot_ids[seq] * a.state_stride + a.state_offset) : nullptr;
    const bool alone = a.q_len[seq] == 1;
    float* y = stage[warp];
    float ss = 0.f;
    for (int i = lane; i < s.size; i += 32) {
        const int c = c0 + i;
        const float b = a.bias ? to_f32(((const T*)a.bias)[c]) : 0.f;
        float acc = 0.f, u = 0.f;
        for (int j = 0; j < a.taps; ++j) {
            const int back = a.taps - 1 - j;
            if (o - back >= 0) u = to_f32(((const T*)a.x)[(size_t)(row - back) * a.x_stride + c]) + b;
            else u = st[(size_t)(a.taps - 1 + (o - back)) * a.channels + c];
            // one token: the state moves on behind the reads (entry j - 1 takes what entry j held; nobody else reads it)
            if (alone && j > 0) st[(size_t)(j - 1) * a.channels + c] = u;
            acc = fmaf(to_f32(((const T*)a.w)[(size_t)c * a.taps + j]), u, acc);
        }
        if (s.silu) acc = silu_f32(acc);
        ss = fmaf(acc, acc, ss);
        y[i] = acc;
    }
    float r = s.factor;
    if (s.norm != CONV_NORM_NONE) {
        ss = warp_sum(ss);
        r = s.factor / sqrtf(ss * s.inv_count + a.eps);
    }
    __syncwarp();
    for (int i = lane; i < s.size; i += 32) y[i] *= s.norm == CONV_NORM_RMS ? r * to_f32(((const T*)s.weight)[i]) : r;
    __syncwarp();
    if (s.rotate) {
        const int half = a.rope_dim / 2;
        const float pos = (float)a.positions[row];
        for (int p = lane; p < half; p += 32) {
            float sn, cs;
            sincosf(pos * a.inv_freq[p], &sn, &cs);
            sn *= a.amp; cs *= a.amp;
            const int e0 = a.adjacent ? 2 * p : p, e1 = a.adjacent ? 2 * p + 1 : p + half;
            const float u = y[e0], v = y[e1];
            y[e0] = u * cs - v * sn;
            y[e1] = v * cs + u * sn;
        }
        __syncwarp();
    }
    TO* dst = conv_dst<T, TO>(a, s, h, row, seq, a.positions[row], lane == 0);
    if (!dst) return;
    for (int i = lane; i < s.pad; i += 32) dst[i] = from_f32<TO>(i < s.size ? y[i] : 0.f);
}

// The state after the step of every sequence that brings at least `from` tokens: its last taps - 1 rows.  One thread per
// (sequence, channel) reads what it needs of the old state before it writes, in rising order.
template <typename T>
__global__ void __launch_bounds__(256)
conv_heads_state_kernel(ConvHeadsArgs a, int n_seqs, int from) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, seq = blockIdx.y;
    if (c >= a.channels || seq >= n_seqs) return;
    const int n = a.q_len[seq], r0 = a.q_start[seq], keep = a.taps - 1;
    if (n < from) return;
    const float b = a.bias ? to_f32(((const T*)a.bias)[c]) : 0.f;
    float* st = (float*)(a.state + (size_t)a.slot_ids[seq] * a.state_stride + a.state_offset);
    for (int i = 0; i < keep; ++i) {
        const int o = n - keep + i;                  // the step's token that entry i holds, if not negative
        st[(size_t)i * a.channels + c] = o >= 0 ? to_f32(((const T*)a.x)[(size_t)(r0 + o) * a.x_stride + c]) + b
                                                : st[(size_t)(i + n) * a.channels + c];
    }
}

// Returns the tokens from which on a sequence's state is still to be moved on.
template <typename T, typename TO, int TAPS, int LPH>
static int launch_conv_vec(const ConvHeadsArgs& a, cudaStream_t s) {
    constexpr int HPC = 128 / LPH;
    int heads = 0;
    for (int i = 0; i < a.n_segs; ++i) heads += a.seg[i].heads;
    const int groups = (heads + HPC - 1) / HPC;
    if ((long long)a.rows * groups < 148 * 16) {
        braid_launch(conv_heads_row_kernel<T, TO, TAPS, LPH>, dim3(groups, a.rows), dim3(128), 0, s, a);
        return 2;
    }
    // spans so long that one wave of CTAs (three an SM) covers the rows, in whole rounds
    long long span = ((long long)a.rows * groups + 148 * 3 - 1) / (148 * 3);
    span = (span + CONV_RPT - 1) / CONV_RPT * CONV_RPT;
    braid_launch(conv_heads_span_kernel<T, TO, TAPS, LPH>, dim3(groups, (unsigned)((a.rows + span - 1) / span)), dim3(128), 0, s, a, (int)span);
    return 1;
}

template <typename T, typename TO>
static int launch_conv(const ConvHeadsArgs& a, bool wide, int lanes, cudaStream_t s) {
    if (wide) {
#define CONV_LPH(TAPS)                                                        \
    do {                                                                      \
        if (lanes <= 4) return launch_conv_vec<T, TO, TAPS, 4>(a, s);                \
        if (lanes <= 8) return launch_conv_vec<T, TO, TAPS, 8>(a, s);           \
        if (lanes <= 16) return launch_conv_vec<T, TO, TAPS, 16>(a, s);         \
        return launch_conv_vec<T, TO, TAPS, 32>(a, s);                          \
    } while (0)
        if (a.taps == 2) CONV_LPH(2);
        else if (a.taps == 3) CONV_LPH(3);
        else CONV_LPH(4);
#undef CONV_LPH
    }
    int heads = 0;
    for (int i = 0; i < a.n_segs; ++i) heads += a.seg[i].heads;
    braid_launch(conv_heads_kernel<T, TO>, dim3((heads + CONV_ANY_WARPS - 1) / CONV_ANY_WARPS, a.rows), dim3(CONV_ANY_WARPS * 32), 0, s, a);
    return 2;
}

// `segs`: n_segs records of 7 ints {heads, size, pad, norm, silu, rotate, plane}; factors, weights, outs, out_strides: one
// entry a segment.  out_f32: what goes to `outs` is float32 whatever the run's type (no cache then).
extern "C" int braid_conv_heads(const void* x, long long x_stride, const void* bias, const void* w, int dtype, void* state,
                                long long state_stride, long long state_offset, const int* token_seq, const int* positions,
                                const int* q_start, const int* q_len, const int* slot_ids, const int* page_table, void* cache,
                                int page_size, int table_cols, int num_pages, const float* inv_freq, int rope_dim, int adjacent,
                                float amp, float eps, int rows, int n_seqs, int max_q_len, int taps, int n_segs, const int* segs,
                                const float* factors, const void* const* weights, void* const* outs,
                                const long long* out_strides, int out_f32, int* error_flag, void* stream) {
    if (rows <= 0 || n_seqs <= 0) return BRAID_OK;
    if (n_segs < 1 || n_segs > CONV_MAX_SEGS) BRAID_REFUSE("conv_heads: %d segments, 1 to %d are built", n_segs, CONV_MAX_SEGS);
    if (taps < 1 || (taps > 1 && !state) || (state_offset & 3) || (state_stride & 3))
        BRAID_REFUSE("conv_heads: %d taps want a state area in multiples of 4 bytes", taps);
    if (dtype != BRAID_F32 && dtype != BRAID_BF16) BRAID_REFUSE("conv_heads: unknown dtype code %d", dtype);
    if (!error_flag) BRAID_REFUSE("conv_heads: error_flag is required");
    if (rope_dim < 0 || (rope_dim & 1)) BRAID_REFUSE("conv_heads: rope_dim=%d must be even", rope_dim);
    ConvHeadsArgs a{x, x_stride, bias, w, (uint8_t*)(taps > 1 ? state : nullptr), state_stride, state_offset, token_seq, positions,
                    q_start, q_len, slot_ids, page_table, cache, page_size, table_cols, num_pages, inv_freq, rope_dim, adjacent,
                    amp, eps, rows, 0, taps, n_segs, 0, error_flag, {}};
    const int vec = dtype == BRAID_F32 ? 4 : 8;
    bool wide = taps >= 2 && taps <= 4 && x_stride % vec == 0 && state_stride % 16 == 0 && state_offset % 16 == 0 &&
                (((uintptr_t)x | (uintptr_t)bias | (uintptr_t)w | (uintptr_t)cache | (uintptr_t)state) & 15) == 0 && rows <= 65535;
    int widest = 0;
    for (int i = 0; i < n_segs; ++i) {                      // (inv_freq is read only where something turns)
        const int* g = segs + 7 * i;
        a.seg[i] = ConvSegment{g[0], g[1], g[2], g[3], g[4], g[5], g[6], factors[i],
                               g[3] == CONV_NORM_RMS ? 1.f / (float)g[1] : 1.f, weights[i], outs[i], out_strides[i]};
        const ConvSegment& s = a.seg[i];
        if (s.heads <= 0 || s.size <= 0 || s.pad < s.size || s.pad > CONV_MAX_SIZE || (s.rotate && rope_dim > s.size))
            BRAID_REFUSE("conv_heads: heads of %d in %d numbers (at most %d), %d of them rotated", s.size, s.pad, CONV_MAX_SIZE, rope_dim);
        if (s.norm == CONV_NORM_RMS && !s.weight) BRAID_REFUSE("conv_heads: this norm has a weight");
        if (s.plane < 0 ? !s.out : (out_f32 || (cache && (!page_table || page_size <= 0 || num_pages <= 0))))
            BRAID_REFUSE("conv_heads: a segment goes to a buffer, or to a cache with pages in the run's type");
        if (s.plane > 1) BRAID_REFUSE("conv_heads: the cache has a key plane (0) and a value plane (1)");
        a.channels += s.heads * s.size;
        if (s.rotate && rope_dim > 0) a.turns = 1;
        if (s.pad > widest) widest = s.pad;
        wide = wide && s.size % vec == 0 && s.pad % vec == 0 && (!s.rotate || adjacent || rope_dim == 0) &&
               (((uintptr_t)s.weight | (uintptr_t)s.out) & 15) == 0 && (s.plane >= 0 || s.out_stride % vec == 0);
    }
    // heads of channels that nothing ties together are cut to the size of the others, so that no lane of those is idle
    int tied = 0;
    auto loose = [](const ConvSegment& s) { return s.norm == CONV_NORM_NONE && !s.rotate && s.plane < 0 && s.pad == s.size; };
    for (int i = 0; i < n_segs; ++i)
        if (!loose(a.seg[i]) && a.seg[i].pad > tied) tied = a.seg[i].pad;
    if (tied > 0 && tied % vec == 0) {
        widest = tied;
        for (int i = 0; i < n_segs; ++i) {
            ConvSegment& s = a.seg[i];
            if (loose(s) && s.size > tied && s.size % tied == 0) {
                s.heads *= s.size / tied;
                s.size = s.pad = tied;
            } else if (s.pad > widest) widest = s.pad;
        }
    }
    const int lanes = (widest + vec - 1) / vec;
    wide = wide && lanes <= 32 && rope_dim <= 2 * CONV_MAX_PAIRS;
    if (rows > 65535 || n_seqs > 65535) BRAID_REFUSE("conv_heads: %d rows exceed one launch", rows);
    cudaStream_t st = (cudaStream_t)stream;
    const int from = dtype == BRAID_F32 ? launch_conv<float, float>(a, wide, lanes, st)
                     : out_f32 ? launch_conv<__nv_bfloat16, float>(a, wide, lanes, st)
                               : launch_conv<__nv_bfloat16, __nv_bfloat16>(a, wide, lanes, st);
    if (taps > 1 && max_q_len >= from) {
        const dim3 grid((a.channels + 255) / 256, n_seqs);
        if (dtype == BRAID_F32) braid_launch(conv_heads_state_kernel<float>, grid, dim3(256), 0, st, a, n_seqs, from);
        else braid_launch(conv_heads_state_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a, n_seqs, from);
    }
    BRAID_LAUNCH_CHECK();
}
