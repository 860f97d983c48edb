// lp_latent_attn.cuh — what the latent-attention mixer (B200_MIX_LATENT_ATTN) does around the library's GEMMs and attention kernels.
// The cache of a layer run holds one row per position, [c (kv_rank) | rotated shared key part (rot_dim)], f32; the attention kernels
// of layerprog.cu read it as ONE K/V head whose keys are the whole row and whose values are the row's first kv_rank entries
// (AttnGeom.v_in_k).  For that, head n's query is carried into the latent: qbuf[r][n] = [W_uk[n]^T q_plain | rotated q part], and the
// summed latent comes back through W_uv[n] afterwards (two products batched over the heads).  Included by layerprog.cu inside its
// anonymous namespace, behind lp_input_conv.cuh (block_sum_sq) and lp_row_attn.cuh (the attention itself).  Norms, angles and the rotation are f32 (the angle, its sine and cosine in double).
#pragma once

struct LatentGeom {
    int H, dim, rot_dim, vdim, q_rank, kv_rank;
    int rot_n;               // rotated channels (even, <= rot_dim); channel i pairs with i + rot_n / 2, or 2i with 2i + 1 (pairs)
    int pairs;
    float rot_mult;          // factor on cos and sin
    int q_off, kv_off, g_off;   // columns of the fused input projection P: [W_dq h or W_q h | W_dkv h | W_g h]; kv_off < 0: no W_dkv (borrowed rows)
    int gate;                // B200_GATE_*
    size_t cache_off;        // byte offset of the rows inside a slot's cache block
    int cap;
    float eps;
};

// cos / sin of the row's position into shared memory: cs[i], sn[i], i < rot_n / 2
__device__ __forceinline__ void latent_angles(const LatentGeom& g, const double* __restrict__ freq, int pos, float* cs, float* sn) {
    for (int i = threadIdx.x; i < g.rot_n / 2; i += blockDim.x) {
        double s, c;
        sincos((double)pos * freq[i], &s, &c);
        cs[i] = (float)c * g.rot_mult;
        sn[i] = (float)s * g.rot_mult;
    }
}
__device__ __forceinline__ float latent_rot(const LatentGeom& g, const float* v, int i, const float* cs, const float* sn) {
    const int half = g.rot_n / 2;
    if (i >= g.rot_n) return v[i];
    if (g.pairs) return (i & 1) ? v[i] * cs[i >> 1] + v[i - 1] * sn[i >> 1] : v[i] * cs[i >> 1] - v[i + 1] * sn[i >> 1];
    return i < half ? v[i] * cs[i] - v[i + half] * sn[i] : v[i] * cs[i - half] + v[i - half] * sn[i - half];
}

// sigmoid of the gate column of value channel c (head c / vdim) of a row of P
__device__ __forceinline__ float latent_gate(const LatentGeom& g, const float* __restrict__ p, int c) {
    return g.gate == B200_GATE_NONE ? 1.0f : sigmoid_f(p[g.g_off + (g.gate == B200_GATE_HEAD ? c / g.vdim : c)]);
}

// The cache row of a row's position: c = rmsnorm(P[kv_off .. + kv_rank]) * kvw and the rotated last rot_dim columns.  sk: the squared sum of
// the first part; cs / sn: latent_angles of the position.
__device__ __forceinline__ void latent_cache_row(const LatentGeom& g, const StepMeta& sm, int r, const float* __restrict__ p, float sk,
                                                 const float* __restrict__ kvw, const float* cs, const float* sn) {
    const float ik = 1.0f / sqrtf(sk / (float)g.kv_rank + g.eps);
    float* row = reinterpret_cast<float*>(sm.run_kv[sm.row_run[r]] + g.cache_off) + (size_t)sm.row_pos[r] * (g.kv_rank + g.rot_dim);
    for (int c = threadIdx.x; c < g.kv_rank; c += blockDim.x) row[c] = p[g.kv_off + c] * ik * kvw[c];
    const float* kr = p + g.kv_off + g.kv_rank;
    for (int i = threadIdx.x; i < g.rot_dim; i += blockDim.x) row[g.kv_rank + i] = latent_rot(g, kr, i, cs, sn);
}

// A row's query q (per head [dim | rot_dim], f32): the plain part of every head in the compute type -> qn [H dim] (the operand of the
// product with W_uk^T), the rotated part -> qrow[n (kv_rank + rot_dim) + kv_rank ..].
template <typename T>
__device__ __forceinline__ void latent_query_row(const LatentGeom& g, const float* __restrict__ q, const float* cs, const float* sn, T* __restrict__ qn,
                                                 float* __restrict__ qrow) {
    const int per = g.dim + g.rot_dim, D = g.kv_rank + g.rot_dim;
    for (int i = threadIdx.x; i < g.H * per; i += blockDim.x) {
        const int n = i / per, c = i - n * per;
        if (c < g.dim) qn[n * g.dim + c] = from_f<T>(q[i]);
        else qrow[(size_t)n * D + g.kv_rank + (c - g.dim)] = latent_rot(g, q + n * per + g.dim, c - g.dim, cs, sn);
    }
}

// One block per row, after the fused input projection.  With a query latent: c_q = rmsnorm(P[q_off ..]) * qw -> cq (compute type, the
// operand of W_uq); without one (q_rank = 0) P holds the query itself, which goes to qn / qbuf (latent_query_row).  With a W_dkv of its
// own the row's cache row is written.
template <typename T>
__global__ void __launch_bounds__(256) lp_latent_prep_kernel(StepMeta sm, LatentGeom g, const float* __restrict__ P, int ldp,
                                                             const float* __restrict__ qw, const float* __restrict__ kvw,
                                                             const double* __restrict__ freq, T* __restrict__ cq, T* __restrict__ qn, float* __restrict__ qbuf) {
    extern __shared__ float lp_cs[];     // [rot_n / 2] cos, then sin
    __shared__ float red[2][8];
    const int r = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const float* p = P + (size_t)r * ldp;
    float* cs = lp_cs;
    float* sn = lp_cs + g.rot_n / 2;
    const bool own = g.kv_off >= 0, direct = g.q_rank == 0;
    if (own || direct) latent_angles(g, freq, sm.row_pos[r], cs, sn);
    float sq = 0.0f, sk = 0.0f;
    for (int c = threadIdx.x; c < g.q_rank; c += blockDim.x) sq = fmaf(p[g.q_off + c], p[g.q_off + c], sq);
    if (own)
        for (int c = threadIdx.x; c < g.kv_rank; c += blockDim.x) sk = fmaf(p[g.kv_off + c], p[g.kv_off + c], sk);
    sq = wsum(sq);
    sk = wsum(sk);
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
    __syncthreads();
    sq = 0.0f; sk = 0.0f;
    for (int i = 0; i < nw; i++) { sq += red[0][i]; sk += red[1][i]; }
    if (direct) latent_query_row(g, p + g.q_off, cs, sn, qn + (size_t)r * g.H * g.dim, qbuf + (size_t)r * g.H * (g.kv_rank + g.rot_dim));
    else {
        const float iq = 1.0f / sqrtf(sq / (float)g.q_rank + g.eps);
        for (int c = threadIdx.x; c < g.q_rank; c += blockDim.x) cq[(size_t)r * g.q_rank + c] = from_f<T>(p[g.q_off + c] * iq * qw[c]);
    }
    if (own) latent_cache_row(g, sm, r, p, sk, kvw, cs, sn);
}

// One block per row, after q = W_uq c_q (Q [R][H (dim + rot_dim)] f32)
template <typename T>
__global__ void __launch_bounds__(256) lp_latent_qprep_kernel(StepMeta sm, LatentGeom g, const float* __restrict__ Q, const double* __restrict__ freq,
                                                              T* __restrict__ qn, float* __restrict__ qbuf) {
    extern __shared__ float lq_cs[];
    const int r = blockIdx.x;
    float* cs = lq_cs;
    float* sn = lq_cs + g.rot_n / 2;
    latent_angles(g, freq, sm.row_pos[r], cs, sn);
    __syncthreads();
    latent_query_row(g, Q + (size_t)r * g.H * (g.dim + g.rot_dim), cs, sn, qn + (size_t)r * g.H * g.dim, qbuf + (size_t)r * g.H * (g.kv_rank + g.rot_dim));
}

// out[r][c] = V[r][c] * gate in the compute type: the operand of W_o.  N channels per thread (4: vdim a multiple of 4)
template <typename T, int N>
__global__ void lp_latent_gate_kernel(LatentGeom g, const float* __restrict__ V, const float* __restrict__ P, int ldp, T* __restrict__ out) {
    const int n = g.H * g.vdim, r = blockIdx.x;
    for (int c = threadIdx.x * N; c < n; c += blockDim.x * N) {
        FloatV<N> v = load_v<N>(V + (size_t)r * n + c);
#pragma unroll
        for (int e = 0; e < N; e++) v.v[e] *= latent_gate(g, P + (size_t)r * ldp, c + e);
        store_v<N>(out + (size_t)r * n + c, v);
    }
}

// ------------------------------------------------------------------------------------------------ few rows, one token per run (decoding)
// Three kernels take a layer from its input projection to the operand of W_o: the query into the latent (with the rotations and the cache
// row), the attention with the keys cut into splits (lp_row_split_kernel), and the merge of the splits with W_uv and the gate.  Everything between the two products is f32.

// Lanes that share one output of a per-head product of length K: the smallest power of two with VN values each, at most a warp
__host__ __device__ inline int latent_lanes(int K, int VN) {
    int l = 1;
    while (l < 32 && l * VN < K) l <<= 1;
    return l;
}
// acc[i] = w . rows[i] over K values, i < NR, summed over the `lanes` neighbouring lanes of the output (sub = place among them); rows past
// nr are the last again.  rows: 16-byte aligned, ld a multiple of 4.
template <typename T, int NR>
__device__ __forceinline__ void latent_dot_n(const T* __restrict__ w, const float* rows, int ld, int nr, int K, int lanes, int sub, bool live, float* acc) {
    constexpr int VN = Vec8<T>::N;
#pragma unroll
    for (int i = 0; i < NR; i++) acc[i] = 0.0f;
    if (live) {
#pragma unroll 2
        for (int k = sub * VN; k < K; k += lanes * VN) {
            float wv[VN];
            Vec8<T>::load(w + k, wv);
#pragma unroll
            for (int i = 0; i < NR; i++) {
                const float* x = rows + (size_t)min(i, nr - 1) * ld + k;
#pragma unroll
                for (int e = 0; e < VN; e += 4) {
                    const float4 v = *reinterpret_cast<const float4*>(x + e);
                    acc[i] = fmaf(wv[e], v.x, acc[i]);
                    acc[i] = fmaf(wv[e + 1], v.y, acc[i]);
                    acc[i] = fmaf(wv[e + 2], v.z, acc[i]);
                    acc[i] = fmaf(wv[e + 3], v.w, acc[i]);
                }
            }
        }
    }
    for (int o = lanes >> 1; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < NR; i++) acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], o);
}
template <typename T>
__device__ __forceinline__ void latent_dot(const T* __restrict__ w, const float* rows, int ld, int nr, int K, int lanes, int sub, bool live, float* acc) {
    if (nr == 1) latent_dot_n<T, 1>(w, rows, ld, nr, K, lanes, sub, live, acc);
    else latent_dot_n<T, GV_ROWS>(w, rows, ld, nr, K, lanes, sub, live, acc);
}

// Blocks [0, H nch): head n, a chunk of latent columns of all rows: qbuf[r][n][j] = W_uk[n]^T[j] . q_plain (ukT [H][kv_rank][dim]); the
// chunk 0 of a head also writes the head's rotated parts.  Blocks behind them (one per row, only with a W_dkv of the layer's own): the
// row's cache row.  Q: f32 queries [R][ldq], per head [dim | rot_dim].
template <typename T>
__global__ void __launch_bounds__(256) lp_latent_absorb_kernel(StepMeta sm, LatentGeom g, const float* __restrict__ Q, int ldq, const float* __restrict__ P, int ldp,
                                                               const T* __restrict__ ukT, const float* __restrict__ kvw, const double* __restrict__ freq,
                                                               float* __restrict__ qbuf, int R, int nch) {
    extern __shared__ __align__(16) float la_sm[];     // product blocks: [R][dim] plain queries; [rot_n] angles
    __shared__ float red[33];
    const int per = g.dim + g.rot_dim, D = g.kv_rank + g.rot_dim;
    if ((int)blockIdx.x >= g.H * nch) {
        const int r = blockIdx.x - g.H * nch;
        const float* p = P + (size_t)r * ldp;
        float* cs = la_sm;
        float* sn = la_sm + g.rot_n / 2;
        latent_angles(g, freq, sm.row_pos[r], cs, sn);
        const float sk = block_sum_sq(p + g.kv_off, g.kv_rank, red);
        latent_cache_row(g, sm, r, p, sk, kvw, cs, sn);
        return;
    }
    constexpr int VN = Vec8<T>::N;
    const int n = blockIdx.x / nch, ch = blockIdx.x - n * nch;
    const int lanes = latent_lanes(g.dim, VN), cols = 8 * (32 / lanes);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane % lanes;
    const int j = ch * cols + warp * (32 / lanes) + lane / lanes;
    {
        const int j0 = ch * cols + warp * (32 / lanes);
        if (j0 < g.kv_rank) prefetch_row(ukT + ((size_t)n * g.kv_rank + j0) * g.dim, min(32 / lanes, g.kv_rank - j0) * g.dim, lane);
    }
    for (int i = threadIdx.x; i < R * g.dim; i += 256) {
        const int r = i / g.dim, d = i - r * g.dim;
        la_sm[i] = Q[(size_t)r * ldq + n * per + d];
    }
    __syncthreads();
    for (int rb = 0; rb < R; rb += GV_ROWS) {
        const int nr = min(GV_ROWS, R - rb);
        float acc[GV_ROWS];
        latent_dot<T>(ukT + ((size_t)n * g.kv_rank + j) * g.dim, la_sm + (size_t)rb * g.dim, g.dim, nr, g.dim, lanes, sub, j < g.kv_rank, acc);
        if (sub == 0 && j < g.kv_rank) {
#pragma unroll
            for (int i = 0; i < GV_ROWS; i++)
                if (i < nr) qbuf[((size_t)(rb + i) * g.H + n) * D + j] = acc[i];
        }
    }
    if (ch == 0) {
        float* cs = la_sm + (size_t)R * g.dim;
        float* sn = cs + g.rot_n / 2;
        for (int r = 0; r < R; r++) {
            latent_angles(g, freq, sm.row_pos[r], cs, sn);
            __syncthreads();
            const float* q = Q + (size_t)r * ldq + n * per + g.dim;
            for (int i = threadIdx.x; i < g.rot_dim; i += 256) qbuf[((size_t)r * g.H + n) * D + g.kv_rank + i] = latent_rot(g, q, i, cs, sn);
            __syncthreads();
        }
    }
}

// The splits' parts of a head's rows summed into the latent (shared memory, f32), then a chunk of the head's value columns: W_uv[n] times
// the latent, times the gate, in the compute type: out[r][n vdim + c].
template <typename T>
__global__ void __launch_bounds__(256) lp_latent_merge_kernel(LatentGeom g, const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits,
                                                              const T* __restrict__ uv, const float* __restrict__ P, int ldp, T* __restrict__ out, int R, int nch) {
    extern __shared__ __align__(16) float lm_sm[];
    float* lat = lm_sm;                                  // [R][kv_rank]
    float* wgt = lm_sm + (size_t)R * g.kv_rank;          // [R][splits]
    constexpr int VN = Vec8<T>::N;
    const int n = blockIdx.x / nch, ch = blockIdx.x - n * nch, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    {
        const int per_warp = 32 / latent_lanes(g.kv_rank, VN), c0 = (ch * 8 + warp) * per_warp;
        if (c0 < g.vdim) prefetch_row(uv + ((size_t)n * g.vdim + c0) * g.kv_rank, min(per_warp, g.vdim - c0) * g.kv_rank, lane);
    }
    for (int r = warp; r < R; r += 8) {                  // a warp per row: the splits' weights, their sum taken off
        const float* ml = part_ml + ((size_t)r * g.H + n) * splits * 2;
        float M = -INFINITY, L = 0.0f;
        for (int s = lane; s < splits; s += 32) M = fmaxf(M, ml[2 * s]);
        M = wmax(M);
        for (int s = lane; s < splits; s += 32) L = fmaf(ml[2 * s + 1], expf(ml[2 * s] - M), L);
        L = wsum(L);
        for (int s = lane; s < splits; s += 32) wgt[r * splits + s] = expf(ml[2 * s] - M) / L;
    }
    __syncthreads();
    // a thread per (group of splits, row, 4 channels): as many groups as the block's threads allow
    const int v4 = g.kv_rank / 4, items = R * v4, groups = max(1, 256 / items);
    float* gsum = lm_sm + (((size_t)R * (g.kv_rank + splits) + 3) & ~(size_t)3);      // [groups][items][4] (groups > 1)
    for (int it = threadIdx.x; it < items * groups; it += 256) {
        const int q = it / items, i = it - q * items, r = i / v4, c = (i - r * v4) * 4;
        const float* po = part_o + ((size_t)r * g.H + n) * splits * g.kv_rank + c;
        const float* w = wgt + r * splits;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int s = q; s < splits; s += groups) {
            const float ws = w[s];
            const float4 o = ws > 0.0f ? *reinterpret_cast<const float4*>(po + (size_t)s * g.kv_rank) : make_float4(0.f, 0.f, 0.f, 0.f);   // (an empty split has written nothing)
            acc.x = fmaf(ws, o.x, acc.x); acc.y = fmaf(ws, o.y, acc.y); acc.z = fmaf(ws, o.z, acc.z); acc.w = fmaf(ws, o.w, acc.w);
        }
        *reinterpret_cast<float4*>(groups > 1 ? gsum + (size_t)it * 4 : lat + (size_t)i * 4) = acc;
    }
    __syncthreads();
    if (groups > 1) {
        for (int i = threadIdx.x; i < items * 4; i += 256) {
            float acc = 0.0f;
            for (int q = 0; q < groups; q++) acc += gsum[(size_t)q * items * 4 + i];
            lat[i] = acc;
        }
        __syncthreads();
    }
    const int lanes = latent_lanes(g.kv_rank, VN), cols = 8 * (32 / lanes), sub = lane % lanes;
    const int c = ch * cols + warp * (32 / lanes) + lane / lanes;
    for (int rb = 0; rb < R; rb += GV_ROWS) {
        const int nr = min(GV_ROWS, R - rb);
        float acc[GV_ROWS];
        latent_dot<T>(uv + ((size_t)n * g.vdim + c) * g.kv_rank, lat + (size_t)rb * g.kv_rank, g.kv_rank, nr, g.kv_rank, lanes, sub, c < g.vdim, acc);
        if (sub == 0 && c < g.vdim) {
#pragma unroll
            for (int i = 0; i < GV_ROWS; i++)
                if (i < nr) {
                    const int r = rb + i, o = n * g.vdim + c;
                    out[(size_t)r * g.H * g.vdim + o] = from_f<T>(acc[i] * latent_gate(g, P + (size_t)r * ldp, o));
                }
        }
    }
}
