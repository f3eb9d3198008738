// Residual streams that are mixed at every sublayer (hyper-connections: Zhu, Huang, Huang, Zeng, Mao, Wu, Min, Zhou,
// "Hyper-Connections", 2024): instead of one residual row a token has n of them, X_1 .. X_n, float32.  A sublayer reads
// u = sum_s a[s] X_s, and what it returns goes back as
//     X_t <- sum_s M[s, t] X_s + b[t] y          for all t at once, from the old streams (M is indexed [from, to]).
// One kernel does what lies between two sublayers: the write of the sublayer before (its y taken from wherever it
// was left: finished float32 rows, the partial sums of a stream-k product, or the outputs of a token's experts, which
// are weighted and added here) and the read of the next one with its RMS norm:
//     out = u / sqrt(mean(u^2) + eps) * w        in the run's type
// so the n streams of a token make one trip to memory a sublayer.  Everything is float32 but `out`.
//
// Rows: x holds n_in = n streams a row [rows][n][width], or one (n_in = 1: all streams are that row, as an embedding
// leaves them).  With `row_index` (the end of the model) row r of the output is read from row row_index[r] and the
// streams are not written back.  A row is shared by the CTAs of one cluster (1 to 8, more where a step has few
// rows), which meet once, for the sum of squares.
#include "common.cuh"
#include "streamk.cuh"
#include <cooperative_groups.h>
namespace cg = cooperative_groups;

#define STREAMS_MAX 16
#define Y_NONE 0
#define Y_ROWS 1          // y float32 [rows][width]
#define Y_PARTIAL 2       // a stream-k product's partial sums
#define Y_EXPERTS 3       // y[slot of (row, choice)] in the run's type, times wgt[row, choice] (null: 1), choices in order

struct StreamsArgs {
    const float* x; float* x_out;            // x_out null: the streams are not written back
    int n, n_in, width, rows;
    const int* row_index;
    // the write of the sublayer before
    int y_kind;
    const float* mix;                        // [n][n] float32, [from][to]
    const float* back;                       // [n] float32: b
    const void* y; int y_bf16; long long ldy;
    const int* pair_slot; const float* wgt; int top;
    StreamK part;
    // the read of the next
    const float* read;                       // [n] float32: a; null: ones
    const void* w; int w_bf16;               // the norm's weights; null: u itself is written
    void* out; int out_bf16;                 // null: no read
    float eps;
    int cols;                                // columns a CTA of the cluster owns (a multiple of 4)
};

// y of four neighbouring columns of a row
__device__ __forceinline__ void sublayer_result(const StreamsArgs& a, int row, int c, const int* slots, const float* wgts, float* y) {
    y[0] = y[1] = y[2] = y[3] = 0.f;
    const bool whole = c + 4 <= a.width && (a.width & 3) == 0;
    if (a.y_kind == Y_ROWS) {
        const float* p = (const float*)a.y + (size_t)row * a.ldy + c;
        if (whole) {
            const float4 v = *reinterpret_cast<const float4*>(p);
            y[0] = v.x; y[1] = v.y; y[2] = v.z; y[3] = v.w;
        } else {
            for (int e = 0; e < 4; ++e) if (c + e < a.width) y[e] = p[e];
        }
    } else if (a.y_kind == Y_PARTIAL) {
        const float4 v = streamk_sum4(a.part, streamk_span(a.part, row, c), row, c);
        y[0] = v.x; y[1] = v.y; y[2] = v.z; y[3] = v.w;
    } else if (a.y_kind == Y_EXPERTS) {
        if (a.y_bf16 && whole && (a.ldy & 3) == 0) {
            constexpr int B = 4;                                 // choices asked for at once
            for (int k0 = 0; k0 < a.top; k0 += B) {
                uint2 raw[B];
#pragma unroll
                for (int i = 0; i < B; ++i) {
                    const int slot = k0 + i < a.top ? slots[k0 + i] : -1;
                    raw[i] = slot >= 0 ? *reinterpret_cast<const uint2*>((const __nv_bfloat16*)a.y + (size_t)slot * a.ldy + c) : make_uint2(0u, 0u);
                }
#pragma unroll
                for (int i = 0; i < B; ++i) {
                    if (k0 + i >= a.top || slots[k0 + i] < 0) continue;
                    const float f = wgts[k0 + i];
                    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[i].x));
                    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[i].y));
                    y[0] = fmaf(f, lo.x, y[0]); y[1] = fmaf(f, lo.y, y[1]);
                    y[2] = fmaf(f, hi.x, y[2]); y[3] = fmaf(f, hi.y, y[3]);
                }
            }
        } else {
            for (int k = 0; k < a.top; ++k) {
                const int slot = slots[k];
                if (slot < 0) continue;
                for (int e = 0; e < 4; ++e)
                    if (c + e < a.width) {
                        const size_t at = (size_t)slot * a.ldy + c + e;
                        y[e] = fmaf(wgts[k], a.y_bf16 ? to_f32(((const __nv_bfloat16*)a.y)[at]) : ((const float*)a.y)[at], y[e]);
                    }
            }
        }
    }
}

// N: the streams the registers hold (n <= N)
template <int N>
__global__ void __launch_bounds__(256)
streams_kernel(StreamsArgs a) {
    extern __shared__ float sm[];            // [cols] u of this CTA's columns, then [top] slots and weights
    __shared__ float coef[STREAMS_MAX * (STREAMS_MAX + 2)];
    __shared__ float red[32];
    __shared__ float share;
    cg::cluster_group cluster = cg::this_cluster();
    const int parts = cluster.num_blocks(), part = cluster.block_rank();
    const int r = blockIdx.x / parts;
    const int tid = threadIdx.x;
    float* mix = coef;                       // [n][n], then b [n], then a [n]
    float* back = coef + a.n * a.n;
    float* rd = back + a.n;
    if (a.y_kind != Y_NONE) {
        for (int i = tid; i < a.n * a.n; i += blockDim.x) mix[i] = a.mix[i];
        if (tid < a.n) back[tid] = a.back[tid];
    }
    if (tid < a.n) rd[tid] = a.read ? a.read[tid] : 1.f;
    const int row = a.row_index ? a.row_index[r] : r;        // the step's tables were there before its first kernel
    float* u_sm = sm;
    int* slots = (int*)(sm + a.cols);
    float* wgts = (float*)(slots + a.top);
    pdl_wait();
    pdl_trigger();                           // not before: the kernels of a whole layer would queue up on the SMs behind the experts
    if (a.y_kind == Y_EXPERTS)
        for (int k = tid; k < a.top; k += blockDim.x) {
            slots[k] = a.pair_slot[(size_t)row * a.top + k];
            wgts[k] = a.wgt ? a.wgt[(size_t)row * a.top + k] : 1.f;
        }
    __syncthreads();
    const int c_lo = part * a.cols, c_hi = min(a.width, c_lo + a.cols);
    const bool vec = (a.width & 3) == 0;
    float ss = 0.f;
    for (int c = c_lo + tid * 4; c < c_hi; c += blockDim.x * 4) {
        float x[N][4], y[4];
#pragma unroll
        for (int s = 0; s < N; ++s) {
            if (s < a.n_in) {
                const float* p = a.x + ((size_t)row * a.n_in + s) * a.width + c;
                if (vec) {
                    const float4 v = *reinterpret_cast<const float4*>(p);
                    x[s][0] = v.x; x[s][1] = v.y; x[s][2] = v.z; x[s][3] = v.w;
                } else {
#pragma unroll
                    for (int e = 0; e < 4; ++e) x[s][e] = c + e < a.width ? p[e] : 0.f;
                }
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) x[s][e] = a.n_in == 1 && s < a.n ? x[0][e] : 0.f;
            }
        }
        sublayer_result(a, row, c, slots, wgts, y);
        float u[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int t = 0; t < N; ++t) {
            if (t >= a.n) break;
            float xt[4];
            if (a.y_kind != Y_NONE) {
#pragma unroll
                for (int e = 0; e < 4; ++e) xt[e] = back[t] * y[e];
#pragma unroll
                for (int s = 0; s < N; ++s) {
                    if (s >= a.n) break;
                    const float m = mix[s * a.n + t];
#pragma unroll
                    for (int e = 0; e < 4; ++e) xt[e] = fmaf(m, x[s][e], xt[e]);
                }
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) xt[e] = x[t][e];
            }
            if (a.x_out) {
                float* p = a.x_out + ((size_t)row * a.n + t) * a.width + c;
                if (vec) *reinterpret_cast<float4*>(p) = make_float4(xt[0], xt[1], xt[2], xt[3]);
                else {
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (c + e < a.width) p[e] = xt[e];
                }
            }
            const float f = rd[t];
#pragma unroll
            for (int e = 0; e < 4; ++e) u[e] = fmaf(f, xt[e], u[e]);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            if (c + e >= a.width) u[e] = 0.f;
            u_sm[c - c_lo + e] = u[e];
            ss = fmaf(u[e], u[e], ss);
        }
    }
    if (!a.out) return;                      // uniform over the cluster
    float scale = 1.f;
    if (a.w) {
        float total = block_sum(ss, red);
        if (parts > 1) {
            if (tid == 0) share = total;
            cluster.sync();
            total = 0.f;
            for (int p = 0; p < parts; ++p) total += *cluster.map_shared_rank(&share, p);
            cluster.sync();                  // no CTA leaves while its share is still read
        }
        scale = 1.f / sqrtf(total / (float)a.width + a.eps);
    }
    // every thread reads back the columns it wrote itself
    for (int c = c_lo + tid * 4; c < c_hi; c += blockDim.x * 4) {
        float o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int ce = c + e < a.width ? c + e : c;
            const float wv = !a.w ? 1.f : a.w_bf16 ? to_f32(((const __nv_bfloat16*)a.w)[ce]) : ((const float*)a.w)[ce];
            o[e] = u_sm[c - c_lo + e] * scale * wv;
        }
        const size_t at = (size_t)r * a.width + c;
        if (a.out_bf16) {
            __nv_bfloat16* p = (__nv_bfloat16*)a.out + at;
            if (vec) {
                const __nv_bfloat162 b0 = __floats2bfloat162_rn(o[0], o[1]), b1 = __floats2bfloat162_rn(o[2], o[3]);
                *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&b0), *reinterpret_cast<const uint32_t*>(&b1));
            } else {
                for (int e = 0; e < 4; ++e)
                    if (c + e < a.width) p[e] = __float2bfloat16_rn(o[e]);
            }
        } else {
            float* p = (float*)a.out + at;
            if (vec) *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]);
            else {
                for (int e = 0; e < 4; ++e)
                    if (c + e < a.width) p[e] = o[e];
            }
        }
    }
}

extern "C" int braid_streams_max(void) { return STREAMS_MAX; }

// `rows`: rows of the output (row_index given) or of the streams.  `part_plan`: the plan of a stream-k product whose
// partial sums y points at (Y_PARTIAL), over `part_rows` rows.
extern "C" int braid_streams(const float* x, float* x_out, int n, int n_in, int width, int rows, const int* row_index, int y_kind,
                             const float* mix, const float* back, const void* y, int y_dtype, long long ldy, const int* pair_slot,
                             const float* wgt, int top, const int* part_plan, int part_rows, const float* read, const void* w,
                             int w_dtype, void* out, int out_dtype, float eps, int cluster, void* stream) {
    if (rows <= 0) return BRAID_OK;
    if (n < 1 || n > STREAMS_MAX || (n_in != n && n_in != 1)) BRAID_REFUSE("streams: %d streams (1 to %d are built), %d given", n, STREAMS_MAX, n_in);
    if (width <= 0) BRAID_REFUSE("streams: width=%d", width);
    if (y_kind < Y_NONE || y_kind > Y_EXPERTS || (y_kind != Y_NONE && (!mix || !back || !y))) BRAID_REFUSE("streams: a sublayer's result comes with its mix and its factors");
    if (y_kind == Y_PARTIAL && !part_plan) BRAID_REFUSE("streams: partial sums come with their plan");
    if (y_kind == Y_EXPERTS && (!pair_slot || top <= 0)) BRAID_REFUSE("streams: the experts' outputs come with the plan's slots");
    if (y_kind != Y_EXPERTS) top = 0;
    if (y_kind == Y_ROWS && y_dtype != BRAID_F32) BRAID_REFUSE("streams: a sublayer's finished rows are float32");
    if (x_out && row_index) BRAID_REFUSE("streams: gathered rows are not written back");
    if (x_out == x && n_in != n) BRAID_REFUSE("streams: one row cannot become %d in place", n);
    if (!x_out && !out) BRAID_REFUSE("streams: nothing to write");
    if (out && out_dtype != BRAID_F32 && out_dtype != BRAID_BF16) BRAID_REFUSE("streams: unknown dtype code %d", out_dtype);
    if ((width & 3) == 0 && ((((uintptr_t)x | (uintptr_t)x_out | (uintptr_t)out) & 15) || (y_kind == Y_ROWS && (((uintptr_t)y & 15) || (ldy & 3))) ||
                             (y_kind == Y_EXPERTS && y_dtype == BRAID_BF16 && ((uintptr_t)y & 7))))
        BRAID_REFUSE("streams: rows must start on 16 bytes");
    if (cluster != 1 && cluster != 2 && cluster != 4 && cluster != 8) BRAID_REFUSE("streams: clusters of 1, 2, 4 or 8 CTAs, not %d", cluster);
    if ((long long)rows * cluster > 0x7fffffffLL) BRAID_REFUSE("streams: %d rows exceed one launch", rows);
    StreamsArgs a{};
    a.x = x; a.x_out = x_out; a.n = n; a.n_in = n_in; a.width = width; a.rows = rows; a.row_index = row_index;
    a.y_kind = y_kind; a.mix = mix; a.back = back; a.y = y; a.y_bf16 = y_dtype == BRAID_BF16; a.ldy = ldy;
    a.pair_slot = pair_slot; a.wgt = wgt; a.top = top;
    if (y_kind == Y_PARTIAL) a.part = streamk_from_plan((const float*)y, part_plan, part_rows);
    a.read = read; a.w = w; a.w_bf16 = w_dtype == BRAID_BF16; a.out = out; a.out_bf16 = out_dtype == BRAID_BF16; a.eps = eps;
    const int groups = (width + 3) / 4;
    a.cols = (groups + cluster - 1) / cluster * 4;
    const int need = (a.cols / 4 + 31) / 32 * 32;
    const int threads = need < 64 ? 64 : need > 256 ? 256 : need;
    const size_t smem = ((size_t)a.cols + 2 * (size_t)top) * sizeof(float);
    if (smem > 40 * 1024) BRAID_REFUSE("streams: %d columns a CTA are more than its shared memory holds (width %d in clusters of %d)", a.cols, width, cluster);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)(rows * cluster));
    cfg.blockDim = dim3(threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = (cudaStream_t)stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = braid_pdl_enabled();
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    if (n <= 2) cudaLaunchKernelEx(&cfg, streams_kernel<2>, a);
    else if (n <= 4) cudaLaunchKernelEx(&cfg, streams_kernel<4>, a);
    else if (n <= 8) cudaLaunchKernelEx(&cfg, streams_kernel<8>, a);
    else cudaLaunchKernelEx(&cfg, streams_kernel<16>, a);
    BRAID_LAUNCH_CHECK();
}
