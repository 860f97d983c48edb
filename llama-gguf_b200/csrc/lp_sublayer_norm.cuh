// lp_sublayer_norm.cuh — the layer form with the norm on a sublayer's output (program.post_norm = 2): x <- alpha x + norm(y), y the output of
// the sublayer before; the next sublayer reads the new x, in the compute type.  Included by layerprog.cu inside its anonymous namespace,
// behind lp_input_conv.cuh (FloatV, StepRoute) and lp_rows_tail.cuh (route_row).
#pragma once

// What has to happen to the stream before a sublayer reads it.  y null: nothing but the copy (the embedding).
struct SubNorm {
    int on = 0;
    const float* y = nullptr;       // [R][width] output of the sublayer before
    const float* w = nullptr;       // [width]
    float alpha = 1.0f, eps = 0.0f;
    int center = 0;                 // 1: layer norm (mean off first), 0: RMS norm
    float* xout = nullptr;          // the new stream (another buffer when several blocks read the old one)
};

// sum over the block's THREADS threads, for all of them; red: THREADS / 32 floats that nobody else touches until the next barrier
template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = wsum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int i = 0; i < THREADS / 32; i++) t += red[i];
    return t;
}

// One row by a block of THREADS threads: out (and out2 when given) = alpha x + norm(y) in the compute type, xout the same in f32 (null: not
// kept).  yf(c) returns channels c .. c + V - 1 of y.  Rows up to 16 THREADS channels (V = 4) stay in registers, every load issued before the
// first sum; wider ones are read again per pass.  par: 0 / 1 alternately for consecutive rows of a block.  Ends without a barrier behind
// its stores.
template <typename T, int THREADS, int V, typename YF>
__device__ __forceinline__ void sub_norm_row_v(const SubNorm& sn, const float* xr, float* xo, int width, int par, T* out, T* out2, YF yf) {
    __shared__ float red[4][THREADS / 32];
    constexpr int TG = 4;
    const float n = (float)width;
    if (width <= V * THREADS * TG) {
        FloatV<V> x[TG], y[TG], w[TG];
        float s = 0.0f;
#pragma unroll
        for (int q = 0; q < TG; q++) {
            const int c = (threadIdx.x + q * THREADS) * V;
            if (c < width) {
                x[q] = load_v<V>(xr + c);
                y[q] = yf(c);
                w[q] = load_v<V>(sn.w + c);
            }
        }
#pragma unroll
        for (int q = 0; q < TG; q++)
            if ((threadIdx.x + q * THREADS) * V < width)
#pragma unroll
                for (int e = 0; e < V; e++) s += y[q].v[e];
        const float mean = sn.center ? block_sum<THREADS>(s, red[2 * par]) / n : 0.0f;
        float ss = 0.0f;
#pragma unroll
        for (int q = 0; q < TG; q++)
            if ((threadIdx.x + q * THREADS) * V < width)
#pragma unroll
                for (int e = 0; e < V; e++) ss = fmaf(y[q].v[e] - mean, y[q].v[e] - mean, ss);
        const float inv = 1.0f / sqrtf(block_sum<THREADS>(ss, red[2 * par + 1]) / n + sn.eps);
#pragma unroll
        for (int q = 0; q < TG; q++) {
            const int c = (threadIdx.x + q * THREADS) * V;
            if (c < width) {
#pragma unroll
                for (int e = 0; e < V; e++) x[q].v[e] = fmaf(sn.alpha, x[q].v[e], (y[q].v[e] - mean) * inv * w[q].v[e]);
                if (xo) store_v<V>(xo + c, x[q]);
                store_v<V>(out + c, x[q]);
                if (out2) store_v<V>(out2 + c, x[q]);
            }
        }
        return;
    }
    float s = 0.0f;
    for (int c = threadIdx.x * V; c < width; c += THREADS * V) {
        const FloatV<V> y = yf(c);
#pragma unroll
        for (int e = 0; e < V; e++) s += y.v[e];
    }
    const float mean = sn.center ? block_sum<THREADS>(s, red[2 * par]) / n : 0.0f;
    float ss = 0.0f;
    for (int c = threadIdx.x * V; c < width; c += THREADS * V) {
        const FloatV<V> y = yf(c);
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(y.v[e] - mean, y.v[e] - mean, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum<THREADS>(ss, red[2 * par + 1]) / n + sn.eps);
    for (int c = threadIdx.x * V; c < width; c += THREADS * V) {
        const FloatV<V> y = yf(c), w = load_v<V>(sn.w + c);
        FloatV<V> x = load_v<V>(xr + c);
#pragma unroll
        for (int e = 0; e < V; e++) x.v[e] = fmaf(sn.alpha, x.v[e], (y.v[e] - mean) * inv * w.v[e]);
        if (xo) store_v<V>(xo + c, x);
        store_v<V>(out + c, x);
        if (out2) store_v<V>(out2 + c, x);
    }
}
template <typename T, int THREADS>
__device__ __forceinline__ void sub_norm_row(const SubNorm& sn, int r, const float* xr, float* xo, int width, int par, T* out, T* out2) {
    if (!sn.y) {
        for (int c = threadIdx.x; c < width; c += THREADS) {
            const float v = xr[c];
            if (xo && xo != xr) xo[c] = v;
            out[c] = from_f<T>(v);
            if (out2) out2[c] = from_f<T>(v);
        }
        return;
    }
    const float* yr = sn.y + (size_t)r * width;
    if (width & 3) sub_norm_row_v<T, THREADS, 1>(sn, xr, xo, width, par, out, out2, [&](int c) { return load_v<1>(yr + c); });
    else sub_norm_row_v<T, THREADS, 4>(sn, xr, xo, width, par, out, out2, [&](int c) { return load_v<4>(yr + c); });
}

// One block per row: the new stream (in place) and its copy `out`; before a mixture of experts also the router's logits and the choice.
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS) lp_sub_norm_kernel(SubNorm sn, const float* x, int width, T* __restrict__ out, StepRoute rt) {
    extern __shared__ __align__(16) uint8_t sn_smem[];
    T* hs = reinterpret_cast<T*>(sn_smem);     // [width] (with routing only)
    const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (rt.router)
        for (int e = warp; e < rt.rows; e += THREADS / 32) prefetch_row(reinterpret_cast<const T*>(rt.router) + (size_t)e * width, width, lane);
    sub_norm_row<T, THREADS>(sn, r, x + (size_t)r * width, sn.xout + (size_t)r * width, width, 0, out + (size_t)r * width, rt.router ? hs : (T*)nullptr);
    if (!rt.router) return;
    __syncthreads();
    step_route<T>(rt, hs, r, width);
}
