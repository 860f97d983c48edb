// lp_input_conv.cuh — the convolution on a sublayer's input (program.in_conv): h = norm(x) becomes h + conv(h), a causal convolution
// over time on every channel.  A slot keeps the last `taps` inputs h (f32) per sublayer and layer run as a ring: the input of position
// p lies at entry p % taps.  A step that brings one token per run reads the entries of the taps - 1 positions before it and writes its
// own, the one entry nobody reads, so reading and writing may share a kernel; longer runs write their last inputs in a kernel after the
// readers.  Included by layerprog.cu inside its anonymous namespace.
#pragma once

struct InConv {
    const float* w = nullptr;   // [width][taps], the last column meets the newest input
    int taps = 0;               // 0: no convolution
    size_t ring_off = 0;        // byte offset of the ring inside a slot's state block
};

// One row of a step with one token per run: where the run's ring is, the row's position, and whether this block writes the ring
struct InConvRow {
    float* ring;
    int pos, write;
};
__device__ __forceinline__ InConvRow input_conv_row(const InConv& ic, const StepMeta& sm, int r, bool write) {
    InConvRow c{nullptr, 0, 0};
    if (ic.taps > 0) {
        c.ring = reinterpret_cast<float*>(sm.run_rec[sm.row_run[r]] + ic.ring_off);
        c.pos = sm.row_pos[r];
        c.write = (write && ic.taps > 1) ? 1 : 0;
    }
    return c;
}
// h + conv(h) of channel k
__device__ __forceinline__ float input_conv_step(const InConv& ic, const InConvRow& c, int width, int k, float h) {
    const float* w = ic.w + (size_t)k * ic.taps;
    float acc = fmaf(w[ic.taps - 1], h, h);
    for (int b = 1; b < ic.taps; b++)
        if (c.pos >= b) acc = fmaf(w[ic.taps - 1 - b], c.ring[(size_t)((c.pos - b) % ic.taps) * width + k], acc);
    if (c.write) c.ring[(size_t)(c.pos % ic.taps) * width + k] = h;
    return acc;
}

__device__ __forceinline__ float block_sum_sq(const float* xr, int width, float* red) {   // every thread receives the sum; red: 33 floats
    float ss = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) ss += xr[c] * xr[c];
    ss = wsum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    if (threadIdx.x < 32) {
        float t = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.0f;
        t = wsum(t);
        if (threadIdx.x == 0) red[32] = t;
    }
    __syncthreads();
    return red[32];
}

// What a mixture of experts needs from the normed row (lp_norm_conv_step_kernel): rows of the router matrix (`experts`, plus the
// always-on expert's gate when shw is there), the bias, where the choice goes
struct StepRoute {
    const void* router = nullptr;   // null: no routing
    const float* bias = nullptr;    // [rows]
    int rows = 0, E = 0, top = 0, mode = 0;
    float scale = 0.0f;
    float *logits = nullptr, *wts = nullptr, *selw = nullptr, *shw = nullptr;
    int* sel = nullptr;
};

// One token per run (decoding), one block per row: norm, convolution, the row in the compute type; then, before a mixture of experts,
// the router's logits on that row (a warp per logit) and the choice.
template <typename T>
__global__ void __launch_bounds__(512) lp_norm_conv_step_kernel(StepMeta sm, InConv ic, const float* __restrict__ x, const float* __restrict__ g, int width,
                                                                float eps, T* __restrict__ out, StepRoute rt) {
    extern __shared__ __align__(16) uint8_t nc_smem[];
    T* hs = reinterpret_cast<T*>(nc_smem);     // [width] (with routing only)
    __shared__ float red[33];
    const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    const float* xr = x + (size_t)r * width;
    const float inv = 1.0f / sqrtf(block_sum_sq(xr, width, red) / (float)width + eps);
    const InConvRow cr = input_conv_row(ic, sm, r, true);
    for (int k = threadIdx.x; k < width; k += blockDim.x) {
        const T v = from_f<T>(input_conv_step(ic, cr, width, k, xr[k] * inv * g[k]));
        out[(size_t)r * width + k] = v;
        if (rt.router) hs[k] = v;
    }
    if (!rt.router) return;
    __syncthreads();
    constexpr int VN = Vec8<T>::N;
    const T* rw = reinterpret_cast<const T*>(rt.router);
    float* z = rt.logits + (size_t)r * rt.rows;
    for (int e = warp; e < rt.rows; e += nw) {
        const T* wr = rw + (size_t)e * width;
        float acc = 0.0f;
        if (width % VN == 0) {
#pragma unroll 4
            for (int c = lane * VN; c < width; c += 32 * VN) {
                float wv[VN], xv[VN];
                Vec8<T>::load(wr + c, wv);
                Vec8<T>::load(hs + c, xv);
#pragma unroll
                for (int j = 0; j < VN; j++) acc = fmaf(wv[j], xv[j], acc);
            }
        } else {
            for (int c = lane; c < width; c += 32) acc = fmaf(to_f(wr[c]), to_f(hs[c]), acc);
        }
        acc = wsum(acc);
        if (lane == 0) z[e] = acc + (rt.bias ? rt.bias[e] : 0.0f);
    }
    __syncthreads();
    if (warp == 0) {
        route_row(z, rt.E, rt.top, rt.wts + (size_t)r * rt.E, rt.sel + (size_t)r * rt.top, rt.selw + (size_t)r * rt.top, lane, rt.mode, rt.scale);
        if (rt.shw && lane == 0) rt.shw[r] = sigmoid_f(z[rt.E]);
    }
}

// Runs of any length: a block of 8 warps takes NC_ROWS rows; the warps first sum the squares of those rows and of the taps - 1 rows before
// them, then every thread walks down the rows in its channels.  A row's earlier inputs come from the rows above it while those belong to
// its run (normed again: x is a few KB away), before that from the ring, before the sequence's start they are zero.  V channels per
// thread (4: width a multiple of 4); TAPS = 0: taps at run time, every input normed anew, else the last TAPS - 1 stay in registers.
constexpr int NC_ROWS = 8;
template <int V> struct FloatV { float v[V]; };
template <int V> __device__ __forceinline__ FloatV<V> load_v(const float* p) {
    FloatV<V> r;
    if (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else r.v[0] = p[0];
    return r;
}
template <int V> __device__ __forceinline__ void store_v(float* p, const FloatV<V>& f) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f.v[0], f.v[1], f.v[2], f.v[3]);
    else p[0] = f.v[0];
}
template <int V> __device__ __forceinline__ void store_v(bf16* p, const FloatV<V>& f) {
    if (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(f.v[0], f.v[1]), b = __floats2bfloat162_rn(f.v[2], f.v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    } else p[0] = from_f<bf16>(f.v[0]);
}
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(256) lp_norm_conv_rows_kernel(StepMeta sm, InConv ic, const float* __restrict__ x, const float* __restrict__ g, int width,
                                                                float eps, T* __restrict__ out, int R) {
    extern __shared__ float nc_inv[];      // [NC_ROWS + taps - 1]: row r0 - (taps - 1) + i
    const int taps = TAPS > 0 ? TAPS : ic.taps, back = taps - 1;
    const int r0 = blockIdx.x * NC_ROWS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int i = warp; i < NC_ROWS + back; i += 8) {
        const int r = r0 - back + i;
        float ss = 0.0f;
        if (r >= 0 && r < R) {
            const float* xr = x + (size_t)r * width;
            for (int c = lane * V; c < width; c += 32 * V) {
                const FloatV<V> f = load_v<V>(xr + c);
#pragma unroll
                for (int e = 0; e < V; e++) ss = fmaf(f.v[e], f.v[e], ss);
            }
        }
        ss = wsum(ss);
        if (lane == 0) nc_inv[i] = 1.0f / sqrtf(ss / (float)width + eps);
    }
    __syncthreads();
    const int nr = min(NC_ROWS, R - r0);
    for (int c = threadIdx.x * V; c < width; c += 256 * V) {
        const FloatV<V> gv = load_v<V>(g + c);
        auto input = [&](int r) {          // h of row r >= 0, r > r0 - taps
            FloatV<V> f = load_v<V>(x + (size_t)r * width + c);
            const float inv = nc_inv[r - r0 + back];
#pragma unroll
            for (int e = 0; e < V; e++) f.v[e] = f.v[e] * inv * gv.v[e];
            return f;
        };
        constexpr int KEEP = TAPS > 1 ? TAPS - 1 : 1;
        FloatV<V> wr[TAPS > 0 ? TAPS : 1];  // wr[b]: the weight of the input b rows above
        if (TAPS > 0) {
#pragma unroll
            for (int b = 0; b < TAPS; b++)
#pragma unroll
                for (int e = 0; e < V; e++) wr[b].v[e] = ic.w[(size_t)(c + e) * TAPS + back - b];
        }
        auto weight = [&](int b, int e) { return TAPS > 0 ? wr[TAPS > 0 ? b : 0].v[e] : ic.w[(size_t)(c + e) * taps + back - b]; };
        FloatV<V> prev[KEEP];              // prev[b - 1]: the input b rows above
        if (TAPS > 1) {
#pragma unroll
            for (int b = 1; b < TAPS; b++)
                if (r0 - b >= 0) prev[b - 1] = input(r0 - b);
        }
        for (int i = 0; i < nr; i++) {
            const int r = r0 + i, run = sm.row_run[r], t = r - sm.run_start[run], pos = sm.row_pos[r];
            const float* ring = reinterpret_cast<const float*>(sm.run_rec[run] + ic.ring_off);
            const FloatV<V> h = input(r);
            FloatV<V> acc;
#pragma unroll
            for (int e = 0; e < V; e++) acc.v[e] = fmaf(weight(0, e), h.v[e], h.v[e]);
#pragma unroll
            for (int b = 1; b < (TAPS > 0 ? TAPS : taps); b++) {
                if (pos < b) continue;
                FloatV<V> p;
                if (t < b) p = load_v<V>(ring + (size_t)((pos - b) % taps) * width + c);
                else if (TAPS > 1) p = prev[b - 1 < KEEP ? b - 1 : 0];
                else p = input(r - b);
#pragma unroll
                for (int e = 0; e < V; e++) acc.v[e] = fmaf(weight(b, e), p.v[e], acc.v[e]);
            }
            store_v<V>(out + (size_t)r * width + c, acc);
            if (TAPS > 1) {
#pragma unroll
                for (int b = KEEP - 1; b > 0; b--) prev[b] = prev[b - 1];
                prev[0] = h;
            }
        }
    }
}

// The last taps - 1 inputs of every run into the ring: block (run, b) norms the run's row b places before its last one.  Launched after
// the readers; entries of positions before this step's stay where they are.
__global__ void __launch_bounds__(256) lp_norm_conv_tail_kernel(StepMeta sm, InConv ic, const float* __restrict__ x, const float* __restrict__ g, int width,
                                                                float eps) {
    __shared__ float red[33];
    const int run = blockIdx.x, r = sm.run_start[run + 1] - 1 - (int)blockIdx.y;
    if (r < sm.run_start[run]) return;
    const float* xr = x + (size_t)r * width;
    float* ring = reinterpret_cast<float*>(sm.run_rec[run] + ic.ring_off) + (size_t)(sm.row_pos[r] % ic.taps) * width;
    const float inv = 1.0f / sqrtf(block_sum_sq(xr, width, red) / (float)width + eps);
    for (int k = threadIdx.x; k < width; k += blockDim.x) ring[k] = xr[k] * inv * g[k];
}

// The embedding's norm, in place; with xcat the result also goes, in the compute type, behind the `width` columns that the stream itself
// will take there ([x; x0] of program.loop_in).
template <typename T>
__global__ void __launch_bounds__(256) lp_embed_norm_kernel(float* __restrict__ x, const float* __restrict__ g, int width, float eps, int norm,
                                                            T* __restrict__ xcat) {
    __shared__ float red[33];
    float* xr = x + (size_t)blockIdx.x * width;
    const float inv = norm ? 1.0f / sqrtf(block_sum_sq(xr, width, red) / (float)width + eps) : 1.0f;
    for (int k = threadIdx.x; k < width; k += blockDim.x) {
        const float v = norm ? xr[k] * inv * g[k] : xr[k];
        xr[k] = v;
        if (xcat) xcat[(size_t)blockIdx.x * 2 * width + width + k] = from_f<T>(v);
    }
}
// the stream in the compute type, `ld` columns apart
template <typename T>
__global__ void lp_cast_rows_kernel(const float* __restrict__ x, int width, T* __restrict__ out, int ld, int R) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)R * width) return;
    const int r = (int)(i / width), c = (int)(i - (size_t)r * width);
    out[(size_t)r * ld + c] = from_f<T>(x[i]);
}

// v[0 .. n) = s[0]: a norm's single number for every coordinate
__global__ void lp_fill_kernel(float* __restrict__ v, const float* __restrict__ s, int n) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) v[i] = s[0];
}
