// lp_input_conv.cuh — the convolution on a sublayer's input (program.in_conv): h = norm(x) becomes h + conv(h), a causal convolution
// over time on every channel.  A slot keeps the last `taps` inputs h (f32) per sublayer and layer run as a ring: the input of position
// p lies at entry p % taps.  A step that brings one token per run reads the entries of the taps - 1 positions before it and writes its
// own, the one entry nobody reads, so reading and writing may share a kernel; the last inputs of longer runs wait in a buffer and go into
// the rings at the end of the step.  Included by layerprog.cu inside its anonymous namespace.
#pragma once

struct InConv {
    const float* w = nullptr;   // [taps][width], the last row meets the newest input
    int taps = 0;               // 0: no convolution
    size_t ring_off = 0;        // byte offset of the ring inside a slot's state block
    float* pend = nullptr;      // longer runs: [runs][taps - 1][width], a run's last inputs until the step's end
};

template <int V> struct FloatV { float v[V]; };
template <int V> __device__ __forceinline__ FloatV<V> load_v(const float* p) {
    FloatV<V> r;
    if (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1 % V] = f.y; r.v[2 % V] = f.z; r.v[3 % V] = f.w;
    } else r.v[0] = p[0];
    return r;
}
template <int V> __device__ __forceinline__ void store_v(float* p, const FloatV<V>& f) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f.v[0], f.v[1 % V], f.v[2 % V], f.v[3 % V]);
    else p[0] = f.v[0];
}
template <int V> __device__ __forceinline__ void store_v(bf16* p, const FloatV<V>& f) {
    if (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(f.v[0], f.v[1 % V]), b = __floats2bfloat162_rn(f.v[2 % V], f.v[3 % V]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    } else p[0] = from_f<bf16>(f.v[0]);
}

// Row r of a step with one token per run, by a block of THREADS threads: h = rmsnorm(x) * g, out = h + conv(h) in the compute type (and a
// copy in out2 when given); `write`: this block moves the ring on.  Up to 2 * 4 * THREADS channels every load is issued before the sum of
// squares is known: the earlier inputs do not depend on it.  Ends without a barrier behind its stores.
template <typename T, int THREADS>
__device__ __forceinline__ void norm_conv_row(const InConv& ic, const StepMeta& sm, int r, const float* __restrict__ xr, const float* __restrict__ g, int width,
                                              float eps, bool write, T* out, T* out2) {
    __shared__ float red[2][THREADS / 32];
    constexpr int TG = 2;
    const int pos = sm.row_pos[r], pm = pos % ic.taps, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* ring = reinterpret_cast<float*>(sm.run_rec[sm.row_run[r]] + ic.ring_off);
    write = write && ic.taps > 1;
    auto slot = [&](int b) { return ring + (size_t)(pm >= b ? pm - b : pm - b + ic.taps) * width; };   // the input b positions back, b < taps
    auto row_inv = [&](float ss) {      // (two buffers: row r + 2 writes behind row r + 1's barrier)
        ss = wsum(ss);
        if (lane == 0) red[r & 1][warp] = ss;
        __syncthreads();
        float t = 0.0f;
#pragma unroll
        for (int i = 0; i < THREADS / 32; i++) t += red[r & 1][i];
        return 1.0f / sqrtf(t / (float)width + eps);
    };
    const float* wlast = ic.w + (size_t)(ic.taps - 1) * width;
    if ((width & 3) == 0 && width <= 4 * THREADS * TG) {
        FloatV<4> x[TG], gv[TG], wl[TG], part[TG];
        float ss = 0.0f;
#pragma unroll
        for (int q = 0; q < TG; q++) {
            const int c = (threadIdx.x + q * THREADS) * 4;
            if (c < width) {
                x[q] = load_v<4>(xr + c);
                gv[q] = load_v<4>(g + c);
                wl[q] = load_v<4>(wlast + c);
#pragma unroll
                for (int e = 0; e < 4; e++) part[q].v[e] = 0.0f;
                auto add = [&](int b) {
                    const FloatV<4> w = load_v<4>(ic.w + (size_t)(ic.taps - 1 - b) * width + c), h = load_v<4>(slot(b) + c);
#pragma unroll
                    for (int e = 0; e < 4; e++) part[q].v[e] = fmaf(w.v[e], h.v[e], part[q].v[e]);
                };
                const int n = min(ic.taps - 1, pos);
                if (n >= 3) { add(1); add(2); add(3); }
                else for (int b = 1; b <= n; b++) add(b);
                for (int b = 4; b <= n; b++) add(b);
#pragma unroll
                for (int e = 0; e < 4; e++) ss = fmaf(x[q].v[e], x[q].v[e], ss);
            }
        }
        const float inv = row_inv(ss);
#pragma unroll
        for (int q = 0; q < TG; q++) {
            const int c = (threadIdx.x + q * THREADS) * 4;
            if (c < width) {
                FloatV<4> h, o;
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    h.v[e] = x[q].v[e] * inv * gv[q].v[e];
                    o.v[e] = fmaf(wl[q].v[e], h.v[e], h.v[e]) + part[q].v[e];
                }
                store_v<4>(out + c, o);
                if (out2) store_v<4>(out2 + c, o);
                if (write) store_v<4>(ring + (size_t)pm * width + c, h);
            }
        }
        return;
    }
    float ss = 0.0f;
    for (int c = threadIdx.x; c < width; c += THREADS) ss = fmaf(xr[c], xr[c], ss);
    const float inv = row_inv(ss);
    for (int c = threadIdx.x; c < width; c += THREADS) {
        const float h = xr[c] * inv * g[c];
        float part = 0.0f;
        for (int b = 1; b < ic.taps && b <= pos; b++) part = fmaf(ic.w[(size_t)(ic.taps - 1 - b) * width + c], slot(b)[c], part);
        const T o = from_f<T>(fmaf(wlast[c], h, h) + part);
        out[c] = o;
        if (out2) out2[c] = o;
        if (write) ring[(size_t)pm * width + c] = h;
    }
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
    const float* corr = nullptr;    // [E] added to the scores that choose
    int rows = 0, E = 0, top = 0, mode = 0;
    float scale = 0.0f;
    float *logits = nullptr, *wts = nullptr, *selw = nullptr, *shw = nullptr;
    int* sel = nullptr;
};

// The router's logits on a row in shared memory (a warp per logit) and the choice, by the whole block
template <typename T>
__device__ __forceinline__ void step_route(const StepRoute& rt, const T* hs, int r, int width) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
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
        route_row(z, rt.E, rt.top, rt.wts + (size_t)r * rt.E, rt.sel + (size_t)r * rt.top, rt.selw + (size_t)r * rt.top, lane, rt.mode, rt.scale, rt.corr);
        if (rt.shw && lane == 0) rt.shw[r] = sigmoid_f(z[rt.E]);
    }
}

// One token per run (decoding), one block per row: norm, convolution, the row in the compute type; then, before a mixture of experts,
// the router's logits on that row (a warp per logit) and the choice.
template <typename T>
__global__ void __launch_bounds__(512) lp_norm_conv_step_kernel(StepMeta sm, InConv ic, const float* __restrict__ x, const float* __restrict__ g, int width,
                                                                float eps, T* __restrict__ out, StepRoute rt) {
    extern __shared__ __align__(16) uint8_t nc_smem[];
    T* hs = reinterpret_cast<T*>(nc_smem);     // [width] (with routing only)
    const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    if (rt.router)
        for (int e = warp; e < rt.rows; e += nw) prefetch_row(reinterpret_cast<const T*>(rt.router) + (size_t)e * width, width, lane);
    norm_conv_row<T, 512>(ic, sm, r, x + (size_t)r * width, g, width, eps, true, out + (size_t)r * width, rt.router ? hs : (T*)nullptr);
    if (!rt.router) return;
    __syncthreads();
    step_route<T>(rt, hs, r, width);
}

// Runs of any length: a block of 8 warps takes NC_ROWS rows; the warps first sum the squares of those rows and of the taps - 1 rows before
// them, then every thread walks down the rows in its channels.  A row's earlier inputs come from the rows above it while those belong to
// its run (normed again: x is a few KB away), before that from the ring, before the sequence's start they are zero.  V channels per
// thread (4: width a multiple of 4); TAPS = 0: taps at run time, every input normed anew, else the last TAPS - 1 stay in registers.
constexpr int NC_ROWS = 8;
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
                for (int e = 0; e < V; e++) wr[b].v[e] = ic.w[(size_t)(back - b) * width + c + e];
        }
        auto weight = [&](int b, int e) { return TAPS > 0 ? wr[TAPS > 0 ? b : 0].v[e] : ic.w[(size_t)(back - b) * width + c + e]; };
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
            const int left = sm.run_start[run + 1] - 1 - r;       // rows of the run behind this one
            if (left < back) store_v<V>(ic.pend + ((size_t)run * back + left) * width + c, h);
            if (TAPS > 1) {
#pragma unroll
                for (int b = KEEP - 1; b > 0; b--) prev[b] = prev[b - 1];
                prev[0] = h;
            }
        }
    }
}

// The end of a step with longer runs: every convolution's pending inputs go into the rings (entries of positions before this step's stay
// where they are).  Block (convolution, run, b): the input b places before the run's last; ring_offs[i]: the ring of convolution i inside
// a slot's state block; pend [convolutions][runs][taps - 1][width].
__global__ void __launch_bounds__(256) lp_ring_commit_kernel(StepMeta sm, const size_t* __restrict__ ring_offs, const float* __restrict__ pend, int taps, int width) {
    const int run = blockIdx.y, b = blockIdx.z, r = sm.run_start[run + 1] - 1 - b;
    if (r < sm.run_start[run]) return;
    const float* src = pend + (((size_t)blockIdx.x * gridDim.y + run) * (taps - 1) + b) * width;
    float* dst = reinterpret_cast<float*>(sm.run_rec[run] + ring_offs[blockIdx.x]) + (size_t)(sm.row_pos[r] % taps) * width;
    for (int k = threadIdx.x; k < width; k += blockDim.x) dst[k] = src[k];
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
// the stream in the compute type, `ld` columns apart; V channels per thread (4: width and ld multiples of 4)
template <typename T, int V>
__global__ void lp_cast_rows_kernel(const float* __restrict__ x, int width, T* __restrict__ out, int ld) {
    const int r = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    if (c < width) store_v<V>(out + (size_t)r * ld + c, load_v<V>(x + (size_t)r * width + c));
}

// v[0 .. n) = s[0]: a norm's single number for every coordinate
__global__ void lp_fill_kernel(float* __restrict__ v, const float* __restrict__ s, int n) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) v[i] = s[0];
}
