// lp_row_attn.cuh — attention over cached rows that hold keys and values at once: the value of a position is the first vdim channels of
// its key row (AttnGeom.v_in_k).  Two mixers cache such rows.  Latent attention: ONE row [latent | rotated part] per position for all heads
// (G = 1).  The softmax mixer with values taken from the keys (v_from_k): one row per K/V head, the projected key, with one factor per row
// and head behind the rows, [cap][G] f32, that makes the key of it (AttnGeom.k_inv: 1 / root mean square).  Kernels: the preparation of the
// latter, split-key attention and its merge for decoding (f32), tile attention for prompts (bf16, tensor pipe).  Included by layerprog.cu
// inside its anonymous namespace.
#pragma once

// After the fused projection P[r] = [q | k | gate]: a warp per (row, head).  q over its root mean square times the temperature -> qbuf; k as
// it is -> the position's cache row, its factor behind the rows.  V channels per lane and load (4: dim and the columns multiples of 4).
template <int V>
__global__ void __launch_bounds__(256) lp_row_prep_kernel(StepMeta sm, AttnGeom a, const float* __restrict__ P, int ldp, float* __restrict__ qbuf, int R) {
    const int u = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, r = u / (a.H + a.G), h = u - r * (a.H + a.G);
    if (r >= R) return;
    const bool isq = h < a.H;
    const int run = sm.row_run[r], pos = sm.row_pos[r], g = h - a.H;
    const float* src = P + (size_t)r * ldp + (isq ? a.q_off + h * a.dim : a.k_off + g * a.dim);
    float* rows = reinterpret_cast<float*>(sm.run_kv[run] + a.kv_off);
    float* dst = isq ? qbuf + ((size_t)r * a.H + h) * a.dim : rows + ((size_t)pos * a.G + g) * a.dim;
    float ss = 0.0f;
    FloatV<V> f0;
#pragma unroll
    for (int e = 0; e < V; e++) f0.v[e] = 0.0f;
    if (lane * V < a.dim) f0 = load_v<V>(src + lane * V);
#pragma unroll
    for (int e = 0; e < V; e++) ss = fmaf(f0.v[e], f0.v[e], ss);
    for (int d = (lane + 32) * V; d < a.dim; d += 32 * V) {
        const FloatV<V> f = load_v<V>(src + d);
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(f.v[e], f.v[e], ss);
    }
    const float inv = a.k_inv ? 1.0f / sqrtf(wsum(ss) / (float)a.dim + a.eps) : 1.0f;
    const float mul = isq ? inv * attn_temp(a, pos) : 1.0f;
    for (int d = lane * V; d < a.dim; d += 32 * V) {
        FloatV<V> f = d == lane * V ? f0 : load_v<V>(src + d);
#pragma unroll
        for (int e = 0; e < V; e++) f.v[e] *= mul;
        store_v<V>(dst + d, f);
    }
    if (!isq && a.k_inv && lane == 0) rows[(size_t)a.cap * a.G * a.dim + (size_t)pos * a.G + g] = inv;
}

// Decoding: attention of one row over its cached rows, the keys cut into gridDim.x splits of whole 32-key tiles; a block stages its tiles in
// shared memory (two in flight, 16-byte cp.async) and each of its warps takes one head of K/V head g: a key per lane for the scores, online
// softmax, the value channels dealt over the lanes for the weighted sum.  blockIdx.z = g * (blocks per K/V head) + part.  part_o [R][H]
// [splits][vdim] receives the unnormalised sums, part_ml the running maximum and sum (an empty split: -inf, 0); the extra term of the
// denominator is split 0's first key.
// P != null (v_from_k): the preparation happens here too.  q comes from P; the row of this position is read from P by every block that
// needs it, and the block with the last tile (part 0) writes it to the cache, where no block of this launch reads it.
constexpr int LS_HEADS = 8, LS_KEYS = 32, LS_ROWS = 64;   // (LS_ROWS: the most rows these kernels take)
// warps of a block: heads of one K/V head, at most LS_HEADS
__host__ __device__ inline int row_block_heads(int per_group) {
    int n = 1;
    while (n < LS_HEADS && n < per_group) n <<= 1;
    return n;
}
__host__ __device__ inline size_t row_split_smem(int D, int heads) { return (size_t)(heads * D + 2 * LS_KEYS * (D + 4)) * 4; }
template <int VCH>
__global__ void __launch_bounds__(32 * LS_HEADS) lp_row_split_kernel(StepMeta sm, AttnGeom a, const float* __restrict__ qbuf, const float* __restrict__ P, int ldp,
                                                                     float* __restrict__ part_o, float* __restrict__ part_ml) {
    extern __shared__ __align__(16) float ls_sm[];
    const int D = a.dim, pitch = D + 4, nwarp = blockDim.x >> 5, hpg = a.H / a.G, zb = (hpg + nwarp - 1) / nwarp;
    float* qs = ls_sm;                         // [warps][D]
    float* ks = ls_sm + nwarp * D;             // [2][LS_KEYS][pitch]
    const int split = blockIdx.x, splits = gridDim.x, r = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = blockIdx.z / zb, zp = blockIdx.z - g * zb, hg = zp * nwarp + warp, h = g * hpg + hg;
    const bool live = hg < hpg;
    const int i = sm.row_pos[r], lo = attn_lo(a, i), ldk = a.G * D;
    float* base = reinterpret_cast<float*>(sm.run_kv[sm.row_run[r]] + a.kv_off);
    const float* rows = base + g * D;
    const float* kinv = a.k_inv ? base + (size_t)a.cap * ldk + g : nullptr;
    const float* own = P ? P + (size_t)r * ldp + a.k_off + g * D : rows + (size_t)i * ldk;      // the row of this position
    const int tiles = (i + 1 - lo + LS_KEYS - 1) / LS_KEYS, each = (tiles + splits - 1) / splits;
    const int t_beg = min(tiles, split * each), t_end = min(tiles, t_beg + each);
    const int vec = D / 4;
    auto stage = [&](int t, int buf) {
        const int j0 = lo + t * LS_KEYS;
        for (int u = threadIdx.x; u < LS_KEYS * vec; u += blockDim.x) {
            const int key = u / vec, c = (u - key * vec) * 4, j = j0 + key;
            cp_async16(smem_u32(ks + ((size_t)buf * LS_KEYS + key) * pitch + c), (j < i ? rows + (size_t)j * ldk : own) + c, j <= i ? 16u : 0u);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (t_beg < t_end) {
        stage(t_beg, 0);
        if (live && !P) {
            for (int d = lane * 4; d < D; d += 128)
                *reinterpret_cast<float4*>(qs + warp * D + d) = *reinterpret_cast<const float4*>(qbuf + ((size_t)r * a.H + h) * D + d);
        } else if (live) {
            const float* q = P + (size_t)r * ldp + a.q_off + h * D;
            float ss = 0.0f;
            for (int d = lane * 4; d < D; d += 128) {
                const FloatV<4> f = load_v<4>(q + d);
#pragma unroll
                for (int e = 0; e < 4; e++) ss = fmaf(f.v[e], f.v[e], ss);
            }
            const float mul = (a.k_inv ? 1.0f / sqrtf(wsum(ss) / (float)D + a.eps) : 1.0f) * attn_temp(a, i);
            for (int d = lane * 4; d < D; d += 128) {
                FloatV<4> f = load_v<4>(q + d);
#pragma unroll
                for (int e = 0; e < 4; e++) f.v[e] *= mul;
                store_v<4>(qs + warp * D + d, f);
            }
        }
    }
    float m = -INFINITY, l = 0.0f, acc[VCH];
    {
        float c;
        if (split == 0 && live && attn_sink(a, h, &c)) { m = c; l = 1.0f; }
    }
    const float slope = attn_slope(a, h);
#pragma unroll
    for (int c = 0; c < VCH; c++) acc[c] = 0.0f;
    for (int t = t_beg; t < t_end; t++) {
        const int buf = (t - t_beg) & 1, j = lo + t * LS_KEYS + lane;
        float kf = (kinv && j <= i && (j < i || !P)) ? kinv[(size_t)j * a.G] : 1.0f;
        if (t + 1 < t_end) {
            stage(t + 1, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const float* kt = ks + (size_t)buf * LS_KEYS * pitch;
        if (P && t + 1 == tiles) {     // this position's own row: its factor, and its way into the cache
            const float* kr = kt + (size_t)(i - lo - t * LS_KEYS) * pitch;
            if (kinv) {
                float ss = 0.0f;
                for (int d = lane; d < D; d += 32) ss = fmaf(kr[d], kr[d], ss);
                const float ki = 1.0f / sqrtf(wsum(ss) / (float)D + a.eps);
                if (j == i) kf = ki;
                if (zp == 0 && threadIdx.x == 0) base[(size_t)a.cap * ldk + (size_t)i * a.G + g] = ki;
            }
            if (zp == 0)
                for (int d = threadIdx.x * 4; d < D; d += blockDim.x * 4) store_v<4>(base + (size_t)i * ldk + g * D + d, load_v<4>(kr + d));
        }
        if (live) {
            const float* kr = kt + (size_t)lane * pitch;
            const float* q = qs + warp * D;
            float s0 = 0.0f, s1 = 0.0f, s2 = 0.0f, s3 = 0.0f;
#pragma unroll 8
            for (int d = 0; d < D; d += 4) {
                const float4 kv = *reinterpret_cast<const float4*>(kr + d), qv = *reinterpret_cast<const float4*>(q + d);
                s0 = fmaf(qv.x, kv.x, s0);
                s1 = fmaf(qv.y, kv.y, s1);
                s2 = fmaf(qv.z, kv.z, s2);
                s3 = fmaf(qv.w, kv.w, s3);
            }
            const float s = j <= i ? attn_score(a, ((s0 + s1) + (s2 + s3)) * kf * a.scale, slope, i, j) : -INFINITY;
            const float mn = fmaxf(m, wmax(s));       // (a tile of the split holds a visible key: mn is finite)
            const float p = expf(s - mn), corr = expf(m - mn);
            l = l * corr + wsum(p);
            m = mn;
#pragma unroll
            for (int c = 0; c < VCH; c++) acc[c] *= corr;
#pragma unroll 8
            for (int k = 0; k < LS_KEYS; k++) {
                const float pk = __shfl_sync(0xffffffffu, p, k);
#pragma unroll
                for (int c = 0; c < VCH; c++) {
                    const int chn = c * 32 + lane;
                    if (chn < a.vdim) acc[c] = fmaf(pk, kt[(size_t)k * pitch + chn], acc[c]);
                }
            }
        }
        __syncthreads();
    }
    if (!live) return;
    const size_t at = ((size_t)r * a.H + h) * splits + split;
    if (lane == 0) {
        part_ml[2 * at] = m;
        part_ml[2 * at + 1] = l;
    }
    if (t_beg < t_end) {
#pragma unroll
        for (int c = 0; c < VCH; c++)
            if (c * 32 + lane < a.vdim) part_o[at * a.vdim + c * 32 + lane] = acc[c];
    }
}

// The merge of the splits: every (row, head)'s weighted values in the compute type -> out[r][h vdim ..] (rows out_ld apart).  The block's
// warps deal the splits among themselves; V channels per lane (4: vdim a multiple of 4), LC_BATCH splits in flight.
constexpr int LC_BATCH = 8;
template <typename T, int V>
__global__ void __launch_bounds__(256) lp_row_combine_kernel(int H, int vdim, const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits,
                                                             T* __restrict__ out, int out_ld) {
    __shared__ float wgt[64], part[8][32 * V];              // (splits <= 64)
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const size_t at = ((size_t)blockIdx.x * H + blockIdx.y) * splits;
    if (warp == 0) {
        const float2* ml = reinterpret_cast<const float2*>(part_ml) + at;
        const float2 none = make_float2(-INFINITY, 0.0f);
        const float2 a = lane < splits ? ml[lane] : none, b = lane + 32 < splits ? ml[lane + 32] : none;
        const float M = wmax(fmaxf(a.x, b.x));
        const float wa = expf(a.x - M), wb = expf(b.x - M);
        const float L = wsum(a.y * wa + b.y * wb);
        wgt[lane] = wa / L;
        wgt[lane + 32] = wb / L;
    }
    __syncthreads();
    for (int c0 = 0; c0 < vdim; c0 += 32 * V) {
        const int c = c0 + lane * V;
        FloatV<V> acc;
#pragma unroll
        for (int e = 0; e < V; e++) acc.v[e] = 0.0f;
        for (int s0 = warp; s0 < splits; s0 += 8 * LC_BATCH) {
            FloatV<V> o[LC_BATCH];
#pragma unroll
            for (int u = 0; u < LC_BATCH; u++) {
                const int s = s0 + 8 * u;
#pragma unroll
                for (int e = 0; e < V; e++) o[u].v[e] = 0.0f;
                if (s < splits && c < vdim && wgt[s] > 0.0f) o[u] = load_v<V>(part_o + (at + s) * vdim + c);     // (an empty split has written nothing)
            }
#pragma unroll
            for (int u = 0; u < LC_BATCH; u++)
#pragma unroll
                for (int e = 0; e < V; e++) acc.v[e] = fmaf(wgt[min(s0 + 8 * u, 63)], o[u].v[e], acc.v[e]);
        }
        store_v<V>(part[warp] + lane * V, acc);
        __syncthreads();
        if (threadIdx.x < 32 * V && c0 + (int)threadIdx.x < vdim) {
            float t = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; i++) t += part[i][threadIdx.x];
            out[(size_t)blockIdx.x * out_ld + blockIdx.y * vdim + c0 + threadIdx.x] = from_f<T>(t);
        }
        __syncthreads();
    }
}

// ------------------------------------------------------------------------------------------------ prompt rows (bf16)
// The hpg = H / G heads of K/V head g = blockIdx.x % G meet the same cached rows, so their (token, head) pairs are ONE list of query rows, pair f
// = (token f / hpg, head g hpg + f % hpg): a block of 8 warps takes LT_ROWS neighbours of the list (16 per warp) against tiles of LT_KEYS
// cached rows.  A tile is
// staged once, as bf16 [key][channel], and serves both products on the tensor pipe (mma.sync m16n8k16, f32 accumulators): ldmatrix gives
// its keys for the scores, ldmatrix.trans its first vdim channels as the values.  Two tiles in shared memory: the next one is loaded
// (DK <= 128: into registers, ahead of the products) while this one is used.  Mask, online softmax and normalisation in f32.  DK / DV:
// upper bounds of the row and of the value.  Blocks start with the last tokens, which see the most keys.
constexpr int LT_ROWS = 128, LT_KEYS = 64;
template <int DK> constexpr size_t row_tile_smem() { return (size_t)(LT_ROWS + 2 * LT_KEYS) * (DK + 8) * 2 + 2 * LT_KEYS * 4; }
// cap tanh(s / cap) through one exponential: 1 - 2 / (exp(2 s / cap) + 1), off by a few 1e-7 of cap
__device__ __forceinline__ float soft_cap_exp(float s, float two_log2e_over_cap, float cap) {
    return fmaf(-2.0f * cap, rcp_fast(ex2_fast(s * two_log2e_over_cap) + 1.0f), cap);
}
__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
template <int DK, int DV>
__global__ void __launch_bounds__(256) lp_row_tile_kernel(StepMeta sm, AttnGeom a, const float* __restrict__ qbuf, bf16* __restrict__ out) {
    constexpr int PITCH = DK + 8, NU = LT_KEYS * (DK / 4) / 256;
    constexpr bool AHEAD = DK <= 128;
    extern __shared__ __align__(16) uint8_t lt_sm[];
    bf16* Qs = reinterpret_cast<bf16*>(lt_sm);          // [LT_ROWS][PITCH]
    bf16* Ks = Qs + LT_ROWS * PITCH;                    // [2][LT_KEYS][PITCH]
    float* Fs = reinterpret_cast<float*>(Ks + 2 * LT_KEYS * PITCH);     // [2][LT_KEYS] factors of the rows (k_inv)
    const int run = blockIdx.y, g = blockIdx.x % a.G, bx = blockIdx.x / a.G, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int r0 = sm.run_start[run], len = sm.run_start[run + 1] - r0, p0 = sm.run_pos0[run];
    const int hpg = a.H / a.G, rows = len * hpg, nb = (rows + LT_ROWS - 1) / LT_ROWS;
    if (bx >= nb) return;
    const int f0 = (nb - 1 - bx) * LT_ROWS, D = a.dim, ldk = a.G * D;
    const float* cache = reinterpret_cast<const float*>(sm.run_kv[run] + a.kv_off) + g * D;
    const float* kinv = a.k_inv ? reinterpret_cast<const float*>(sm.run_kv[run] + a.kv_off) + (size_t)a.cap * ldk + g : nullptr;
    // pair f of the list: its place among the step's (row, head) pairs
    auto pair = [&](int f) { return (size_t)(r0 + f / hpg) * a.H + g * hpg + f % hpg; };
    for (int u = threadIdx.x; u < LT_ROWS * (DK / 4); u += 256) {
        const int f = u / (DK / 4), d = (u - f * (DK / 4)) * 4;
        const float4 v = (f0 + f < rows && d < D) ? *reinterpret_cast<const float4*>(qbuf + pair(f0 + f) * D + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        *reinterpret_cast<uint2*>(Qs + f * PITCH + d) = make_uint2(pack_bf2(v.x, v.y), pack_bf2(v.z, v.w));
    }
    const int last = p0 + min(f0 + LT_ROWS - 1, rows - 1) / hpg, lo = attn_lo(a, p0 + f0 / hpg);
    const int tiles = (last - lo) / LT_KEYS + 1;
    auto get = [&](int t, int u) {
        const int i = threadIdx.x + u * 256, key = i / (DK / 4), d = (i - key * (DK / 4)) * 4, j = lo + t * LT_KEYS + key;
        return (j <= last && d < D) ? *reinterpret_cast<const float4*>(cache + (size_t)j * ldk + d) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    auto put = [&](int t, int u, const float4& v) {
        const int i = threadIdx.x + u * 256, key = i / (DK / 4), d = (i - key * (DK / 4)) * 4;
        *reinterpret_cast<uint2*>(Ks + ((t & 1) * LT_KEYS + key) * PITCH + d) = make_uint2(pack_bf2(v.x, v.y), pack_bf2(v.z, v.w));
    };
    auto stage = [&](int t) {
#pragma unroll
        for (int u0 = 0; u0 < NU; u0 += 4) {
            float4 v[4];
#pragma unroll
            for (int u = 0; u < 4; u++) v[u] = get(t, u0 + u);
#pragma unroll
            for (int u = 0; u < 4; u++) put(t, u0 + u, v[u]);
        }
    };
    auto get_f = [&](int t) {         // (threads below LT_KEYS) the factor of a key of the tile
        const int j = lo + t * LT_KEYS + threadIdx.x;
        return (kinv && j <= last) ? kinv[(size_t)j * a.G] : 1.0f;
    };
    stage(0);
    if (kinv && threadIdx.x < LT_KEYS) Fs[threadIdx.x] = get_f(0);
    // this thread's two rows of the warp's 16, their positions, and the warp's first and last position
    const int fa = f0 + warp * 16 + gid, fb = fa + 8;
    const int ia = p0 + min(fa, rows - 1) / hpg, ib = p0 + min(fb, rows - 1) / hpg;
    const int w_first = p0 + min(f0 + warp * 16, rows - 1) / hpg, w_last = p0 + min(f0 + warp * 16 + 15, rows - 1) / hpg;
    const uint32_t q_addr = smem_u32(Qs + (warp * 16 + (lane & 15)) * PITCH + (lane >> 4) * 8);
    const uint32_t k_off = (uint32_t)(((lane & 7) + ((lane >> 4) << 3)) * PITCH + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t v_off = (uint32_t)(((lane & 7) + (((lane >> 3) & 1) << 3)) * PITCH + (lane >> 4) * 8) * 2;
    const float L2E = 1.4426950408889634f, sl = a.scale * L2E;      // scores in powers of two
    const float cap_in = a.softcap > 0.0f ? 2.0f * L2E / a.softcap * a.scale : 0.0f, cap_out = a.softcap * L2E;
    float o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; n++) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    {   // the extra term of the denominator (one of the four threads of a row counts it)
        float c;
        if (attn_sink(a, g * hpg + min(fa, rows - 1) % hpg, &c)) { m0 = c * L2E; l0 = tig == 0 ? 1.0f : 0.0f; }
        if (attn_sink(a, g * hpg + min(fb, rows - 1) % hpg, &c)) { m1 = c * L2E; l1 = tig == 0 ? 1.0f : 0.0f; }
    }
    __syncthreads();
    for (int t = 0; t < tiles; t++) {
        const int j0 = lo + t * LT_KEYS;
        float4 nx[AHEAD ? NU : 1];
        if (AHEAD && t + 1 < tiles) {
#pragma unroll
            for (int u = 0; u < NU; u++) nx[u % (AHEAD ? NU : 1)] = get(t + 1, u);
        }
        const float fn = (kinv && threadIdx.x < LT_KEYS && t + 1 < tiles) ? get_f(t + 1) : 1.0f;
        if (j0 <= w_last && j0 + LT_KEYS - 1 > w_first - a.window) {      // (some row of the warp sees some key of the tile)
            const uint32_t kt = smem_u32(Ks + (t & 1) * LT_KEYS * PITCH);
            float sc[LT_KEYS / 8][4];
#pragma unroll
            for (int n = 0; n < LT_KEYS / 8; n++) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.0f;
#pragma unroll
            for (int kb = 0; kb < DK / 16; kb++) {
                if (kb * 16 < D) {
                    uint32_t qa[4];
                    ldsm4(qa, q_addr + kb * 32);
#pragma unroll
                    for (int n = 0; n < LT_KEYS / 16; n++) {
                        uint32_t b[4];
                        ldsm4(b, kt + k_off + (uint32_t)(n * 16 * PITCH + kb * 16) * 2);
                        mma_bf16(sc[2 * n], qa, b[0], b[1]);
                        mma_bf16(sc[2 * n + 1], qa, b[2], b[3]);
                    }
                }
            }
            const bool all = j0 + LT_KEYS - 1 <= w_first && j0 > w_last - a.window;     // nothing of the tile is masked
            if (kinv) {
                const float* f = Fs + (t & 1) * LT_KEYS + 2 * tig;
#pragma unroll
                for (int n = 0; n < LT_KEYS / 8; n++) {
                    const float2 k = *reinterpret_cast<const float2*>(f + n * 8);
                    sc[n][0] *= k.x; sc[n][1] *= k.y; sc[n][2] *= k.x; sc[n][3] *= k.y;
                }
            }
            if (a.softcap > 0.0f) {
#pragma unroll
                for (int n = 0; n < LT_KEYS / 8; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) sc[n][e] = soft_cap_exp(sc[n][e], cap_in, cap_out);
            }
            const float mul = a.softcap > 0.0f ? 1.0f : sl;
            float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
            for (int n = 0; n < LT_KEYS / 8; n++) {
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int j = j0 + n * 8 + 2 * tig + (e & 1), i = (e & 2) ? ib : ia;
                    sc[n][e] = (all || (j <= i && i - j < a.window)) ? sc[n][e] * mul : -INFINITY;
                }
                x0 = fmaxf(x0, fmaxf(sc[n][0], sc[n][1]));
                x1 = fmaxf(x1, fmaxf(sc[n][2], sc[n][3]));
            }
            x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1));
            x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
            x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1));
            x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
            const float n0 = fmaxf(m0, x0), n1 = fmaxf(m1, x1);
            const float b0 = n0 == -INFINITY ? 0.0f : n0, b1 = n1 == -INFINITY ? 0.0f : n1;      // (a row without a visible key yet: all weights 0)
            const float c0 = ex2_fast(m0 - b0), c1 = ex2_fast(m1 - b1);
            m0 = n0;
            m1 = n1;
            float s0 = 0.0f, s1 = 0.0f;
            uint32_t pa[LT_KEYS / 16][4];
#pragma unroll
            for (int n = 0; n < LT_KEYS / 8; n++) {
                const float e0 = ex2_fast(sc[n][0] - b0), e1 = ex2_fast(sc[n][1] - b0), e2 = ex2_fast(sc[n][2] - b1), e3 = ex2_fast(sc[n][3] - b1);
                s0 += e0 + e1;
                s1 += e2 + e3;
                pa[n >> 1][(n & 1) * 2] = pack_bf2(e0, e1);
                pa[n >> 1][(n & 1) * 2 + 1] = pack_bf2(e2, e3);
            }
            l0 = l0 * c0 + s0;
            l1 = l1 * c1 + s1;
#pragma unroll
            for (int n = 0; n < DV / 8; n++) {
                o[n][0] *= c0; o[n][1] *= c0; o[n][2] *= c1; o[n][3] *= c1;
            }
#pragma unroll
            for (int n = 0; n < DV / 16; n++) {
                if (n * 16 < a.vdim) {
#pragma unroll
                    for (int k = 0; k < LT_KEYS / 16; k++) {
                        uint32_t b[4];
                        ldsm4_t(b, kt + v_off + (uint32_t)(k * 16 * PITCH + n * 16) * 2);
                        mma_bf16(o[2 * n], pa[k], b[0], b[1]);
                        mma_bf16(o[2 * n + 1], pa[k], b[2], b[3]);
                    }
                }
            }
        }
        if (t + 1 < tiles) {
            if (AHEAD) {
#pragma unroll
                for (int u = 0; u < NU; u++) put(t + 1, u, nx[u % (AHEAD ? NU : 1)]);
            } else stage(t + 1);
            if (kinv && threadIdx.x < LT_KEYS) Fs[((t + 1) & 1) * LT_KEYS + threadIdx.x] = fn;
        }
        __syncthreads();
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    const float v0 = 1.0f / l0, v1 = 1.0f / l1;
#pragma unroll
    for (int n = 0; n < DV / 8; n++) {
        const int c = n * 8 + 2 * tig;
        if (c < a.vdim) {        // (vdim is even: c + 1 < vdim)
            if (fa < rows) *reinterpret_cast<uint32_t*>(out + pair(fa) * a.vdim + c) = pack_bf2(o[n][0] * v0, o[n][1] * v0);
            if (fb < rows) *reinterpret_cast<uint32_t*>(out + pair(fb) * a.vdim + c) = pack_bf2(o[n][2] * v1, o[n][3] * v1);
        }
    }
}
