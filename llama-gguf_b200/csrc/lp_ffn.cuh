// lp_ffn.cuh — the norm-after-sum layer form and the feed-forward kinds beside relu^2: the gated tanh-GELU layer and the mixture of
// experts (router, top-k weights, expert activations).  Included by layerprog.cu inside its anonymous namespace.
#pragma once

// x <- (alpha x + y) / sqrt(mean((alpha x + y)^2) + eps) * w, kept in f32; xc receives the same row in the compute type (the
// sublayers of such a layer read x itself, so this copy is the next GEMM's operand).  w = null: x is only copied (the embedding);
// y = null: nothing is added.
template <typename OutT>
__global__ void lp_postnorm_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, OutT* __restrict__ xc, int width,
                                   float alpha, float eps) {
    const int r = blockIdx.x;
    float* xr = x + (size_t)r * width;
    OutT* cr = xc + (size_t)r * width;
    if (!w) {
        for (int c = threadIdx.x; c < width; c += blockDim.x) cr[c] = from_f<OutT>(xr[c]);
        return;
    }
    const float* yr = y ? y + (size_t)r * width : nullptr;
    __shared__ float red[33];
    float ss = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const float v = yr ? fmaf(alpha, xr[c], yr[c]) : alpha * xr[c];
        xr[c] = v;
        ss += v * v;
    }
    ss = wsum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    if (threadIdx.x < 32) {
        float t = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.0f;
        t = wsum(t);
        if (threadIdx.x == 0) red[32] = 1.0f / sqrtf(t / (float)width + eps);
    }
    __syncthreads();
    const float inv = red[32];
    for (int c = threadIdx.x; c < width; c += blockDim.x) {   // (a thread reads back its own writes)
        const float v = xr[c] * inv * w[c];
        xr[c] = v;
        cr[c] = from_f<OutT>(v);
    }
}

__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

// out[r][n] = gelu_tanh(P[r][n]) * P[r][ff + n]: the fused projection holds [gate | up]
template <typename OutT>
__global__ void lp_gated_gelu_kernel(const float* __restrict__ P, int ldp, OutT* __restrict__ out, int ff, int R) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)R * ff) return;
    const int r = (int)(i / ff), n = (int)(i - (size_t)r * ff);
    const float* p = P + (size_t)r * ldp;
    out[i] = from_f<OutT>(gelu_tanh_f(p[n]) * p[ff + n]);
}

// out[r][n] = relu(P[r][n])^2 (the relu^2 layer when its up projection is part of a wider product)
template <typename OutT>
__global__ void lp_relu2_kernel(const float* __restrict__ P, int ldp, OutT* __restrict__ out, int ff, int R) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)R * ff) return;
    const int r = (int)(i / ff), n = (int)(i - (size_t)r * ff);
    const float z = fmaxf(P[(size_t)r * ldp + n], 0.0f);
    out[i] = from_f<OutT>(z * z);
}

// Router: one warp per row of the f32 logits P[r][0 .. E) (route_row, lp_rows_tail.cuh)
__global__ void lp_moe_route_kernel(const float* __restrict__ P, int ldp, int E, int top, float* __restrict__ wts, int* __restrict__ sel,
                                    float* __restrict__ selw, int R, int mode, float scale, float* __restrict__ shw, const float* __restrict__ corr) {
    const int r = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (r >= R) return;
    route_row(P + (size_t)r * ldp, E, top, wts + (size_t)r * E, sel + (size_t)r * top, selw + (size_t)r * top, lane, mode, scale, corr);
    if (shw && lane == 0) shw[r] = sigmoid_f(P[(size_t)r * ldp + E]);      // the always-on expert's gate: the logit behind the experts'
}

// an expert's activation: relu(z)^2 (B200_ACT_RELU2) or the exact GELU (B200_ACT_GELU)
__device__ __forceinline__ float expert_act(float z, int act) {
    if (act == B200_ACT_GELU) return gelu_erf_f(z);
    z = fmaxf(z, 0.0f);
    return z * z;
}

// What an expert's hidden units are made of.  The gated kinds (B200_ACT_SILU_GLU, B200_ACT_CLAMPED_GLU, B200_ACT_RELU_GLU) have two pre-activations per unit,
// their up matrix is [gate | up] rows.
struct ExpertAct {
    int kind, win;               // B200_ACT_*; 1: the expert's weight goes onto its input
    float limit, shared_limit, slope;
};
__host__ __device__ inline bool act_gated(int kind) { return kind == B200_ACT_SILU_GLU || kind == B200_ACT_CLAMPED_GLU || kind == B200_ACT_RELU_GLU; }
__device__ __forceinline__ int expert_rows(int eff, int kind) { return act_gated(kind) ? 2 * eff : eff; }
// min(z, limit) sigmoid(slope .) (clamp(zu, +-limit) + 1)
__device__ __forceinline__ float clamped_glu_f(float z, float zu, float limit, float slope) {
    const float g = fminf(z, limit), u = fminf(fmaxf(zu, -limit), limit);
    return g * sigmoid_f(slope * g) * (u + 1.0f);
}
// hidden unit of an expert from its pre-activation(s) and the expert's weight w: on the output, act(.) w, or on the input (win),
// where W (w h) = w (W h) puts it on the pre-activations
__device__ __forceinline__ float expert_unit(float z, float zu, float w, const ExpertAct& a, float limit) {
    if (a.win) { z *= w; zu *= w; }
    const float v = a.kind == B200_ACT_CLAMPED_GLU ? clamped_glu_f(z, zu, limit, a.slope) : a.kind == B200_ACT_SILU_GLU ? z * sigmoid_f(z) * zu
                  : a.kind == B200_ACT_RELU_GLU ? fmaxf(z, 0.0f) * zu : expert_act(z, a.kind);
    return a.win ? v : v * w;
}
// the always-on expert: the same form, its weight (1 without a gate) always on the output
__device__ __forceinline__ float shared_unit(float z, float zu, float w, ExpertAct a) {
    a.win = 0;
    return expert_unit(z, zu, w, a, a.shared_limit);
}

// out[r][c] = hidden unit c of the row: expert e = c / eff with its weight (0 = not chosen: the unit is 0), the always-on expert's
// units behind them with weight shw[r] (null: 1).  wts: [R][ldw].  P holds every expert's pre-activations side by side (expert_rows per expert).
template <typename OutT>
__global__ void lp_moe_act_kernel(const float* __restrict__ P, int ldp, int off, const float* __restrict__ wts, int ldw, const float* __restrict__ shw, int E,
                                  int eff, int sff, OutT* __restrict__ out, int R, ExpertAct a) {
    const int total = E * eff + sff;
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)R * total) return;
    const int r = (int)(i / total), c = (int)(i - (size_t)r * total);
    const int per = expert_rows(eff, a.kind);
    const bool glu = act_gated(a.kind);
    const float* p = P + (size_t)r * ldp + off;
    float v = 0.0f;
    if (c < E * eff) {
        const int e = c / eff, n = c - e * eff;
        const float w = wts[(size_t)r * ldw + e];
        if (w != 0.0f) v = expert_unit(p[e * per + n], glu ? p[e * per + eff + n] : 0.0f, w, a, a.limit);
    } else {
        const int n = c - E * eff;
        v = shared_unit(p[E * per + n], glu ? p[E * per + sff + n] : 0.0f, shw ? shw[r] : 1.0f, a);
    }
    out[i] = from_f<OutT>(v);
}

// The same for (token, choice) pairs in expert order: pair i = (row i / top, choice i % top) sits at row pos[i] of P (its expert's
// pre-activations, expert_rows wide) and of out (eff wide); its weight is selw[i].  V units per thread (4: eff a multiple of 4).
// Pairs of an identity expert have neither.
template <typename OutT, int V>
__global__ void lp_moe_pair_act_kernel(const float* __restrict__ P, int ldp, const int* __restrict__ pos, const int* __restrict__ sel, const float* __restrict__ selw,
                                       int E, int eff, OutT* __restrict__ out, int n_pairs, ExpertAct a) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)n_pairs * (eff / V)) return;
    const int pr = (int)(i / (eff / V)), n = (int)(i - (size_t)pr * (eff / V)) * V;
    if (sel[pr] >= E) return;
    const float* p = P + (size_t)pos[pr] * ldp;
    const FloatV<V> z = load_v<V>(p + n), zu = act_gated(a.kind) ? load_v<V>(p + eff + n) : z;
    FloatV<V> o;
#pragma unroll
    for (int e = 0; e < V; e++) o.v[e] = expert_unit(z.v[e], zu.v[e], selw[pr], a, a.limit);
    store_v<V>(out + (size_t)pos[pr] * eff + n, o);
}
// and for the always-on expert over all rows: P [R][expert_rows(sff)] -> out [R][sff]
template <typename OutT, int V>
__global__ void lp_moe_shared_act_kernel(const float* __restrict__ P, int ldp, const float* __restrict__ shw, int sff, OutT* __restrict__ out, int R, ExpertAct a) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)R * (sff / V)) return;
    const int r = (int)(i / (sff / V)), n = (int)(i - (size_t)r * (sff / V)) * V;
    const float* p = P + (size_t)r * ldp;
    const FloatV<V> z = load_v<V>(p + n), zu = act_gated(a.kind) ? load_v<V>(p + sff + n) : z;
    const float w = shw ? shw[r] : 1.0f;
    FloatV<V> o;
#pragma unroll
    for (int e = 0; e < V; e++) o.v[e] = shared_unit(z.v[e], zu.v[e], w, a);
    store_v<V>(out + (size_t)r * sff + n, o);
}

// Few rows (decoding): only the chosen experts' weights are read.  up_exp holds [e0 up | e1 up | ... | always-on up] rows of `width`
// columns (a gated expert: [gate | up], expert_rows each); segment k < top of a row's activations belongs to expert sel[r][k],
// segment `top` to the always-on expert.
//   act[r][k eff + n] = unit(up_e[n] . h_r, selw[r][k])        act[r][top eff + n] = unit(up_shared[n] . h_r, shw[r] or 1)
// A choice e >= E is an identity expert: its segment is not written.  One warp per (row, segment, n); h rows are staged in shared memory once per block.
template <typename T>
__global__ void __launch_bounds__(256) lp_moe_up_sel_kernel(const T* __restrict__ H, const T* __restrict__ up_exp, const int* __restrict__ sel,
                                                            const float* __restrict__ selw, const float* __restrict__ shw, int E, int top, int eff, int sff,
                                                            int width, int R, T* __restrict__ act, ExpertAct a) {
    extern __shared__ __align__(16) uint8_t mu_smem[];
    T* hs = reinterpret_cast<T*>(mu_smem);
    constexpr int VN = Vec8<T>::N;
    for (int i = threadIdx.x; i < R * width / VN; i += blockDim.x)
        *reinterpret_cast<uint4*>(hs + (size_t)i * VN) = *reinterpret_cast<const uint4*>(H + (size_t)i * VN);
    __syncthreads();
    const int lane = threadIdx.x & 31;
    const int per_row = top * eff + sff, per = expert_rows(eff, a.kind);
    const int total = R * per_row;
    const bool glu = act_gated(a.kind);
    for (int o = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5); o < total; o += gridDim.x * (blockDim.x >> 5)) {
        const int r = o / per_row, c = o - r * per_row;
        const int k = c < top * eff ? c / eff : top;
        const int n = c - k * eff;
        const int e = k < top ? sel[(size_t)r * top + k] : E;
        if (k < top && e >= E) continue;
        const T* wr = up_exp + ((size_t)e * per + n) * width;
        const T* wu = wr + (size_t)(k < top ? eff : sff) * width;          // (gated experts: the up row of the same unit)
        const T* hr = hs + (size_t)r * width;
        float acc = 0.0f, accu = 0.0f;
        for (int i = lane * VN; i < width; i += 32 * VN) {
            float wv[VN], xv[VN];
            Vec8<T>::load(wr + i, wv);
            Vec8<T>::load(hr + i, xv);
#pragma unroll
            for (int j = 0; j < VN; j++) acc = fmaf(wv[j], xv[j], acc);
            if (glu) {
                Vec8<T>::load(wu + i, wv);
#pragma unroll
                for (int j = 0; j < VN; j++) accu = fmaf(wv[j], xv[j], accu);
            }
        }
        acc = wsum(acc);
        accu = wsum(accu);
        if (lane == 0)
            act[o] = from_f<T>(k < top ? expert_unit(acc, accu, selw[(size_t)r * top + k], a, a.limit) : shared_unit(acc, accu, shw ? shw[r] : 1.0f, a));
    }
}

// y[r][c] = sum over the row's segments of down_e[c] . act segment; down_cat is [width][E eff + sff].  MD_SPLIT warps share one (row, c):
// each takes every MD_SPLIT-th 16-byte group of every segment (more loads in flight per output: a decode step has only `width` of
// them), the partial sums meet in shared memory and are added in warp order.  accum = 1: y += (y is the residual stream).  Identity experts
// (choices e >= E) have no segment: they add their weight times what the feed-forward reads, hf in f32 or, when that is null, h.
constexpr int MD_SPLIT = 4, MD_BATCH = 6;
template <typename T>
__global__ void __launch_bounds__(256) lp_moe_down_sel_kernel(const T* __restrict__ act, const T* __restrict__ down_cat, const int* __restrict__ sel,
                                                              int E, int top, int eff, int sff, int width, int R, float* __restrict__ y, RowsTail tail, int accum,
                                                              const float* __restrict__ selw, const T* __restrict__ h, const float* hf, int identity) {
    constexpr int VN = Vec8<T>::N, GROUPS = 8 / MD_SPLIT;
    __shared__ float part[8];
    __shared__ int sel_s[256];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, grp = warp / MD_SPLIT, sw = warp % MD_SPLIT;
    const bool sel_in = R * top <= 256;
    if (sel_in) {
        for (int i = threadIdx.x; i < R * top; i += blockDim.x) sel_s[i] = sel[i];
        __syncthreads();
    }
    const int per_row = top * eff + sff, kd = E * eff + sff, total = R * width;
    for (int base = blockIdx.x * GROUPS; base < total; base += gridDim.x * GROUPS) {
        const int o = base + grp;
        float acc = 0.0f;
        if (o < total) {
            const int r = o / width, c = o - r * width;
            const T* ar = act + (size_t)r * per_row;
            const T* dr = down_cat + (size_t)c * kd;
            // the row's segments as one list of 16-byte groups (expert sizes are multiples of VN), MD_BATCH of them in flight per lane
            for (int i0 = (sw * 32 + lane) * VN; i0 < per_row; i0 += MD_BATCH * MD_SPLIT * 32 * VN) {
                uint4 wv[MD_BATCH], xv[MD_BATCH];
#pragma unroll
                for (int u = 0; u < MD_BATCH; u++) {
                    const int i = i0 + u * MD_SPLIT * 32 * VN;
                    wv[u] = xv[u] = make_uint4(0u, 0u, 0u, 0u);
                    const int k = i < per_row ? min(i / eff, top) : 0;
                    const int e = i >= per_row ? 0 : k < top ? (sel_in ? sel_s[r * top + k] : sel[(size_t)r * top + k]) : E;
                    if (i < per_row && (k == top || e < E)) {
                        wv[u] = *reinterpret_cast<const uint4*>(dr + (size_t)e * eff + (i - k * eff));
                        xv[u] = *reinterpret_cast<const uint4*>(ar + i);
                    }
                }
#pragma unroll
                for (int u = 0; u < MD_BATCH; u++) {
                    float wf[VN], xf[VN];
                    Vec8<T>::load(reinterpret_cast<const T*>(&wv[u]), wf);
                    Vec8<T>::load(reinterpret_cast<const T*>(&xv[u]), xf);
#pragma unroll
                    for (int j = 0; j < VN; j++) acc = fmaf(wf[j], xf[j], acc);
                }
            }
        }
        acc = wsum(acc);
        if (lane == 0) part[warp] = acc;
        __syncthreads();
        if (o < total && sw == 0 && lane == 0) {
            float t = part[grp * MD_SPLIT];
#pragma unroll
            for (int i = 1; i < MD_SPLIT; i++) t += part[grp * MD_SPLIT + i];
            if (identity) {
                const int r = o / width;
                for (int k = 0; k < top; k++)
                    if (sel[(size_t)r * top + k] >= E) t = fmaf(selw[(size_t)r * top + k], hf ? hf[o] : to_f(h[o]), t);
            }
            y[o] = accum ? y[o] + t : t;
        }
        __syncthreads();
    }
    if (tail.on) rows_tail<T>(tail);
}

// Many rows: the (token, choice) pairs are put in expert order, so that every expert multiplies a contiguous block of rows.
// One block: counts per expert, their running sum (seg[e] = {first row, rows}), then every pair takes the next free row of its
// expert (pos[r top + k]).  Which pair of an expert gets which row does not matter: a row's result does not depend on its place.
__global__ void __launch_bounds__(1024) lp_moe_sort_kernel(const int* __restrict__ sel, int n_pairs, int E, int* __restrict__ seg, int* __restrict__ pos) {
    extern __shared__ int ms[];          // [E] counts, then [E] cursors
    int* cnt = ms;
    int* cur = ms + E;
    for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) atomicAdd(&cnt[sel[i]], 1);
    __syncthreads();
    if (threadIdx.x == 0) {
        int at = 0;
        for (int e = 0; e < E; e++) {
            seg[2 * e] = at;
            seg[2 * e + 1] = cnt[e];
            cur[e] = at;
            at += cnt[e];
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) pos[i] = atomicAdd(&cur[sel[i]], 1);
}

// Xp[pos[i]] = H[i / top]: one block per pair (pairs of an identity expert, sel[i] >= E, need no row)
template <typename T>
__global__ void lp_moe_gather_kernel(const T* __restrict__ H, const int* __restrict__ pos, const int* __restrict__ sel, int E, int top, int width, T* __restrict__ Xp) {
    const int i = blockIdx.x;
    if (sel[i] >= E) return;
    const T* src = H + (size_t)(i / top) * width;
    T* dst = Xp + (size_t)pos[i] * width;
    constexpr int VN = Vec8<T>::N;
    if (width % VN == 0) {
        for (int c = threadIdx.x; c < width / VN; c += blockDim.x) reinterpret_cast<uint4*>(dst)[c] = reinterpret_cast<const uint4*>(src)[c];
    } else {
        for (int c = threadIdx.x; c < width; c += blockDim.x) dst[c] = src[c];
    }
}

// Channels c .. c + V - 1 of sum_k selw[r][k] out_k, choices in the order they were taken: out_k = Yp[pos[r top + k]], or the row hr itself
// when choice k is an identity expert (sel >= E); selw = null: plain sum (the weights went into the experts' inputs)
template <int V>
__device__ __forceinline__ FloatV<V> moe_sum(const float* __restrict__ Yp, const int* __restrict__ pos, const int* __restrict__ sel, const float* __restrict__ selw, int top,
                                             int E, int width, int r, int c, const float* hr) {
    FloatV<V> sum;
#pragma unroll
    for (int e = 0; e < V; e++) sum.v[e] = 0.0f;
    for (int k = 0; k < top; k++) {
        const size_t at = (size_t)r * top + k;
        const FloatV<V> v = load_v<V>(sel[at] >= E ? hr + c : Yp + (size_t)pos[at] * width + c);
        const float w = selw ? selw[at] : 1.0f;
#pragma unroll
        for (int e = 0; e < V; e++) sum.v[e] = fmaf(w, v.v[e], sum.v[e]);
    }
    return sum;
}
// x <- alpha x + norm(that sum): the end of a mixture in the layer form with the norm on a sublayer's output (lp_sublayer_norm.cuh).  One block per row.
template <typename T>
__global__ void __launch_bounds__(256) lp_sub_norm_moe_kernel(SubNorm sn, const float* x, int width, T* __restrict__ out, const float* __restrict__ Yp,
                                                              const int* __restrict__ pos, const int* __restrict__ sel, const float* __restrict__ selw, int top, int E) {
    const int r = blockIdx.x;
    const float* xr = x + (size_t)r * width;
    float* xo = sn.xout + (size_t)r * width;
    T* o = out + (size_t)r * width;
    if (width & 3) {
        sub_norm_row_v<T, 256, 1>(sn, xr, xo, width, 0, o, (T*)nullptr, [&](int c) { return moe_sum<1>(Yp, pos, sel, selw, top, E, width, r, c, xr); });
    } else {
        sub_norm_row_v<T, 256, 4>(sn, xr, xo, width, 0, o, (T*)nullptr, [&](int c) { return moe_sum<4>(Yp, pos, sel, selw, top, E, width, r, c, xr); });
    }
}
// y[r] (+)= sum_k selw[r][k] Yp[pos[r top + k]], selw = null: plain sum; add = 1 when y already holds something to add to (the always-on expert's output, or the residual stream).
// Identity experts are left out (lp_moe_identity_kernel adds them).
__global__ void lp_moe_combine_kernel(const float* __restrict__ Yp, const int* __restrict__ pos, const int* __restrict__ sel, const float* __restrict__ selw, int top, int E,
                                      int width, int add, float* __restrict__ y) {
    const int r = blockIdx.x;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        float acc = add ? y[(size_t)r * width + c] : 0.0f, sum = 0.0f;
        for (int k = 0; k < top; k++) {
            const size_t at = (size_t)r * top + k;
            if (sel[at] < E) sum = fmaf(selw ? selw[at] : 1.0f, Yp[(size_t)pos[at] * width + c], sum);
        }
        y[(size_t)r * width + c] = acc + sum;
    }
}
// y[r] (+)= (sum of the row's weights for identity experts, wts[r][E .. E + n)) * what the feed-forward reads: hf in f32 or, when null, h
template <typename T>
__global__ void lp_moe_identity_kernel(const float* __restrict__ wts, int E, int n, const T* __restrict__ h, const float* hf, int width, int add, float* __restrict__ y) {
    const int r = blockIdx.x;
    float w = 0.0f;
    for (int e = 0; e < n; e++) w += wts[(size_t)r * (E + n) + E + e];
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const size_t o = (size_t)r * width + c;
        const float v = w == 0.0f ? 0.0f : w * (hf ? hf[o] : to_f(h[o]));
        y[o] = add ? y[o] + v : v;
    }
}
