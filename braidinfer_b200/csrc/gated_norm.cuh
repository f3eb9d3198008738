// The gated RMS norm of the recurrent mixers, shared by the libraries that end a recurrence with it.
#pragma once
#include "common.cuh"

// ------------------------------------------------------------------ gated RMS norm
// y [rows, width] float32 (a recurrence's output), gate [rows, gate_stride] in the run's type or float32 (TG), in groups of `group`
// columns, each normed by its own root mean square:
//   gate_first = 0:  out = y / rms(y) * w * silu(gate) * out_scale         (norm, then gate)
//   gate_first = 1:  u = y * silu(gate);  out = u / rms(u) * w * out_scale (gate, then norm)
// With `gate_sigmoid` the gate goes through a sigmoid instead of silu, in either order.
// w has w_len numbers; column c of the row reads w[c % w_len] (w_len = group: one weight for every group;
// w_len = width: a weight per column).  One warp per (row, group).  Everything in float32; out in the run's type.
__device__ __forceinline__ float norm_gate(float z, int sigmoid) { return sigmoid ? 1.f / (1.f + expf(-z)) : silu_f32(z); }

template <typename T, typename TG>
__global__ void __launch_bounds__(128)
gated_norm_kernel(const float* __restrict__ y, const TG* __restrict__ gate, long long gate_stride, const T* __restrict__ w,
                  int w_len, T* __restrict__ out, long long out_stride, const int* __restrict__ token_seq, int rows,
                  int width, int group, int gate_first, int gate_sigmoid, float eps, float out_scale) {
    pdl_trigger();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int groups = width / group;
    const long long item = (long long)blockIdx.x * 4 + warp;
    if (item >= (long long)rows * groups) return;
    const int row = (int)(item / groups), gi = (int)(item - (long long)row * groups);
    if (token_seq[row] < 0) return;
    const float* yr = y + (size_t)row * width + (size_t)gi * group;
    const TG* gr = gate + (size_t)row * gate_stride + (size_t)gi * group;
    float ss = 0.f;
    for (int c = lane; c < group; c += 32) {
        float u = yr[c];
        if (gate_first) u *= norm_gate(to_f32(gr[c]), gate_sigmoid);
        ss = fmaf(u, u, ss);
    }
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / (float)group + eps);
    T* orow = out + (size_t)row * out_stride + (size_t)gi * group;
    for (int c = lane; c < group; c += 32) {
        const float sg = norm_gate(to_f32(gr[c]), gate_sigmoid);
        const float wv = to_f32(w[(gi * group + c) % w_len]);
        float u = yr[c];
        u = gate_first ? (u * sg) * r * wv : (u * r * wv) * sg;
        orow[c] = from_f32<T>(u * out_scale);
    }
}

// The same with a CTA of 128 threads a (row, group): for groups of more than 128 columns, where a warp alone would
// walk a long way (a decode step of 8 rows and 8 groups of 512 columns: 21 -> 11.5 us).
template <typename T, typename TG>
__global__ void __launch_bounds__(128)
gated_norm_block_kernel(const float* __restrict__ y, const TG* __restrict__ gate, long long gate_stride, const T* __restrict__ w,
                        int w_len, T* __restrict__ out, long long out_stride, const int* __restrict__ token_seq, int rows,
                        int width, int group, int gate_first, int gate_sigmoid, float eps, float out_scale) {
    pdl_trigger();
    pdl_wait();
    __shared__ float red[32];
    const int groups = width / group;
    const int row = blockIdx.x / groups, gi = blockIdx.x - row * groups;
    if (token_seq[row] < 0) return;
    const float* yr = y + (size_t)row * width + (size_t)gi * group;
    const TG* gr = gate + (size_t)row * gate_stride + (size_t)gi * group;
    float ss = 0.f;
    for (int c = threadIdx.x; c < group; c += blockDim.x) {
        float u = yr[c];
        if (gate_first) u *= norm_gate(to_f32(gr[c]), gate_sigmoid);
        ss = fmaf(u, u, ss);
    }
    ss = block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / (float)group + eps);
    T* orow = out + (size_t)row * out_stride + (size_t)gi * group;
    for (int c = threadIdx.x; c < group; c += blockDim.x) {
        const float sg = norm_gate(to_f32(gr[c]), gate_sigmoid);
        const float wv = to_f32(w[(gi * group + c) % w_len]);
        float u = yr[c];
        u = gate_first ? (u * sg) * r * wv : (u * r * wv) * sg;
        orow[c] = from_f32<T>(u * out_scale);
    }
}

// The same for wide groups whose rows allow 16-byte moves: a CTA of up to 512 threads a (row, group), V neighbouring columns
// a thread and turn, the first two runs of a thread kept in registers between the sum of squares and the result (a group of
// 4,096 columns of 8 rows: 49 -> 9 us with a CTA of 128 threads and single columns before).
template <typename T, typename TG, int V>
__global__ void __launch_bounds__(512)
gated_norm_wide_kernel(const float* __restrict__ y, const TG* __restrict__ gate, long long gate_stride, const T* __restrict__ w,
                       int w_len, T* __restrict__ out, long long out_stride, const int* __restrict__ token_seq, int rows,
                       int width, int group, int gate_first, int gate_sigmoid, float eps, float out_scale) {
    pdl_trigger();
    pdl_wait();
    __shared__ float red[32];
    const int groups = width / group;
    const int row = blockIdx.x / groups, gi = blockIdx.x - row * groups;
    if (token_seq[row] < 0) return;
    const float* yr = y + (size_t)row * width + (size_t)gi * group;
    const TG* gr = gate + (size_t)row * gate_stride + (size_t)gi * group;
    const T* wr = w + (w_len == group ? 0 : (size_t)gi * group);
    constexpr int KEEP = 2;
    float u[KEEP][V], sg[KEEP][V];
    constexpr int VG = V < 16 / (int)sizeof(TG) ? V : 16 / (int)sizeof(TG);       // gate numbers a load
    auto load_gate = [&](const TG* p, float* ss) {
#pragma unroll
        for (int e = 0; e < V; e += VG) load_run<TG, VG>(p + e, ss + e);
    };
    auto fetch = [&](int c, float* uu, float* ss) {
#pragma unroll
        for (int e = 0; e < V; e += 4) load_run<float, 4>(yr + c + e, uu + e);
        load_gate(gr + c, ss);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            ss[e] = norm_gate(ss[e], gate_sigmoid);
            if (gate_first) uu[e] *= ss[e];
        }
    };
    const int step = blockDim.x * V, c0 = threadIdx.x * V;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
        if (c0 + k * step < group) {
            fetch(c0 + k * step, u[k], sg[k]);
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(u[k][e], u[k][e], ss);
        }
    for (int c = c0 + KEEP * step; c < group; c += step) {
        float uu[V], gg[V];
        fetch(c, uu, gg);
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(uu[e], uu[e], ss);
    }
    ss = block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / (float)group + eps);
    T* orow = out + (size_t)row * out_stride + (size_t)gi * group;
    auto finish = [&](int c, const float* uu, const float* gg) {
        float wv[V], o[V];
        load_run<T, V>(wr + c, wv);
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = (gate_first ? uu[e] * r * wv[e] : (uu[e] * r * wv[e]) * gg[e]) * out_scale;
        store_run<T, V>(orow + c, o);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
        if (c0 + k * step < group) finish(c0 + k * step, u[k], sg[k]);
    for (int c = c0 + KEEP * step; c < group; c += step) {
        float uu[V], gg[V];
        fetch(c, uu, gg);
        finish(c, uu, gg);
    }
}

template <typename T, typename TG>
static int gated_norm_launch(const float* y, const TG* gate, long long gate_stride, const T* w, int w_len, T* out,
                             long long out_stride, const int* token_seq, int rows, int width, int group, int gate_first,
                             int gate_sigmoid, float eps, float out_scale, cudaStream_t s) {
    if (rows <= 0) return BRAID_OK;
    if (width <= 0 || group <= 0 || width % group) BRAID_REFUSE("gated_norm: width %d is not a whole number of groups of %d", width, group);
    if (w_len <= 0) BRAID_REFUSE("gated_norm: the weight has no numbers");
    const long long items = (long long)rows * (width / group);
    const long long blocks = (items + 3) / 4;
    if (blocks > 0x7fffffffLL) BRAID_REFUSE("gated_norm: %lld (row, group) pairs exceed one launch", items);
    constexpr int V = 16 / sizeof(T);
    if (group > 128 && items <= 0x7fffffffLL && group % V == 0 && gate_stride % V == 0 && out_stride % V == 0 &&
        (w_len == group || w_len == width) && (((uintptr_t)y | (uintptr_t)gate | (uintptr_t)w | (uintptr_t)out) & 15) == 0) {
        const int runs = (group / V + 31) / 32 * 32;
        braid_launch(gated_norm_wide_kernel<T, TG, V>, dim3((int)items), dim3(runs < 64 ? 64 : runs > 512 ? 512 : runs), 0, s, y, gate,
                     gate_stride, w, w_len, out, out_stride, token_seq, rows, width, group, gate_first, gate_sigmoid, eps, out_scale);
    } else if (group > 128 && items <= 0x7fffffffLL) {
        braid_launch(gated_norm_block_kernel<T, TG>, dim3((int)items), dim3(128), 0, s, y, gate, gate_stride, w, w_len, out, out_stride,
                     token_seq, rows, width, group, gate_first, gate_sigmoid, eps, out_scale);
    } else {
        braid_launch(gated_norm_kernel<T, TG>, dim3((int)blocks), dim3(128), 0, s, y, gate, gate_stride, w, w_len, out, out_stride,
                     token_seq, rows, width, group, gate_first, gate_sigmoid, eps, out_scale);
    }
    BRAID_LAUNCH_CHECK();
}
