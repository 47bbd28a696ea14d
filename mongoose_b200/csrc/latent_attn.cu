// Latent attention on the CUDA cores: one token, and every token of 32-bit prompts (and of sizes that the
// tensor-core kernel does not take).  Three steps: queries folded through the key matrix, U_k^T q, so that they
// meet the cached rows themselves; attention over ranges of cached rows with an online softmax, a CTA for
// several heads at once because all heads read the same rows; the ranges joined and the weighted sum of
// latents taken through the value matrix.
#include <algorithm>

#include "layered_ops.cuh"

namespace mg {

namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ int token_pos(const LatentStep& a, int t) { return a.st ? a.st->pos : a.pos0 + t; }

// The pair (i, i + half) of a rotated part of `rot` values at position p.
__device__ __forceinline__ float rotated(const LatentAttn& A, const float* v, int p, int i) {
    const int half = A.rot / 2, k = i < half ? i : i - half;
    const float c = A.cos_tab[(size_t)p * half + k], s = A.sin_tab[(size_t)p * half + k];
    return i < half ? v[i] * c - v[i + half] * s : v[i] * c + v[i - half] * s;
}

// Normed latent and rotated key part of one token into the cache, by the whole CTA.
template <typename KT>
__device__ __forceinline__ void store_latent(const LatentAttn& A, const float* c, int pos, float* red) {
    KT* dst = static_cast<KT*>(A.cache) + (size_t)pos * A.row();
    float ss = 0.f;
    for (int i = threadIdx.x; i < A.rank; i += blockDim.x) ss = fmaf(c[i], c[i], ss);
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)A.rank + A.eps);
    for (int i = threadIdx.x; i < A.rank_s; i += blockDim.x) from_f32(i < A.rank ? c[i] * r * A.c_norm[i] : 0.f, dst + i);
    for (int i = threadIdx.x; i < A.rot_s; i += blockDim.x) from_f32(i < A.rot ? rotated(A, c + A.rank, pos, i) : 0.f, dst + A.rank_s + i);
}

constexpr int kFoldCols = 128;      // latent values per CTA: four per lane
constexpr int kFoldAhead = 16;      // rows of U_k a warp holds before the query is there

// CTA (head, 128 latent values) of one token: lanes over the values, warps over the head's dimensions.  The last
// CTA of a token stores its latent where `down` is given.
template <typename KT>
__global__ void __launch_bounds__(kThreads) latent_query_kernel(const LatentStep a) {
    __shared__ __align__(16) float part[kThreads / 32][kFoldCols];
    __shared__ float red[40];
    const LatentAttn& A = a.at;
    const int slices = (A.rank_s + kFoldCols - 1) / kFoldCols, t = blockIdx.y;
    const int h = blockIdx.x / slices, r0 = (blockIdx.x - h * slices) * kFoldCols;
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
    constexpr int nw = kThreads / 32;
    const bool fold = h < A.heads;
    const int r = r0 + lane * 4;
    const __nv_bfloat16* uk = A.uk + (size_t)h * A.dim_s * A.ld + r;
    uint2 w[kFoldAhead];
#pragma unroll
    for (int i = 0; i < kFoldAhead; i++) {
        const int d = wid + i * nw;
        w[i] = fold && r < A.rank_s && d < A.dim ? __ldg(reinterpret_cast<const uint2*>(uk + (size_t)d * A.ld)) : make_uint2(0u, 0u);
    }
    pdl_launch_dependents();
    pdl_wait();
    const int pos = token_pos(a, t);
    if (pos >= A.max_seq) return;
    if (!fold) {
        store_latent<KT>(A, a.down + A.q_rank, pos, red);
        return;
    }
    const float* q = a.q + ((size_t)t * A.heads + h) * A.qrow();
    float* qa = a.qa + ((size_t)t * A.heads + h) * A.row();
    float acc[4] = {};
    auto add = [&](uint2 u, float x) {
        acc[0] = fmaf(__uint_as_float(u.x << 16), x, acc[0]);
        acc[1] = fmaf(__uint_as_float(u.x & 0xffff0000u), x, acc[1]);
        acc[2] = fmaf(__uint_as_float(u.y << 16), x, acc[2]);
        acc[3] = fmaf(__uint_as_float(u.y & 0xffff0000u), x, acc[3]);
    };
#pragma unroll
    for (int i = 0; i < kFoldAhead; i++) {
        const int d = wid + i * nw;
        if (d < A.dim) add(w[i], q[d]);
    }
    for (int d = wid + kFoldAhead * nw; d < A.dim; d += nw)
        if (r < A.rank_s) add(__ldg(reinterpret_cast<const uint2*>(uk + (size_t)d * A.ld)), q[d]);
    *reinterpret_cast<float4*>(&part[wid][lane * 4]) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    __syncthreads();
    for (int i = threadIdx.x; i < kFoldCols; i += kThreads) {
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < nw; k++) v += part[k][i];
        if (r0 + i < A.rank_s) qa[r0 + i] = v * A.scale;
    }
    if (r0 == 0)
        for (int i = threadIdx.x; i < A.rot_s; i += kThreads) qa[A.rank_s + i] = i < A.rot ? rotated(A, q + A.dim_s, pos, i) * A.scale : 0.f;
}

// ---- attention over a range of cached rows ----
// Shared memory: rows [2][tile][row + 16 bytes], queries [group][row + 4], weights [tile][group4], then per head
// the running maximum, sum and this tile's correction.
template <typename KT>
struct Attend {
    int ks, qs, g4;
    KT* k;
    float *q, *w, *m, *l, *fix;
    __device__ __forceinline__ Attend(const LatentAttn& A, int group, int tile, float* base) {
        ks = A.row() + 16 / (int)sizeof(KT);
        qs = A.row() + 4;
        g4 = pad_to(group, 4);
        k = reinterpret_cast<KT*>(base);
        q = reinterpret_cast<float*>(k + 2 * (size_t)tile * ks);
        w = q + (size_t)group * qs;
        m = w + tile * g4;
        l = m + g4;
        fix = l + g4;
    }
};

// A thread's accumulators are four heads x two neighbouring latent values, EP such sets.
template <typename KT, int EP>
__global__ void __launch_bounds__(kThreads) latent_attend_kernel(const LatentStep a) {
    extern __shared__ __align__(16) float smem[];
    constexpr int CN = Chunk16<KT>::n;
    pdl_launch_dependents();
    pdl_wait();
    const LatentAttn& A = a.at;
    const int t = blockIdx.z, pos = token_pos(a, t), len = pos + 1, h0 = blockIdx.y * a.group, G = min(a.group, A.heads - h0);
    if (pos >= A.max_seq) return;
    int j0, j1;
    const int active = key_split(len, a.splits, a.tile, blockIdx.x, &j0, &j1);
    if ((int)blockIdx.x >= active) return;
    const Attend<KT> sm(A, a.group, a.tile, smem);
    const int row = A.row(), chunks = row / CN, tile = a.tile, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
    const KT* cache = static_cast<const KT*>(A.cache);
    auto load = [&](int buf, int j) {               // a warp per row; rows past the range are zero
        KT* dst = sm.k + (size_t)buf * tile * sm.ks;
        for (int p = wid; p < tile; p += kThreads / 32)
            for (int c = lane; c < chunks; c += 32) {
                if (j + p < j1) cp_async16(dst + p * sm.ks + c * CN, cache + (size_t)(j + p) * row + c * CN);
                else *reinterpret_cast<uint4*>(dst + p * sm.ks + c * CN) = make_uint4(0u, 0u, 0u, 0u);
            }
    };
    const float* qa = a.qa + ((size_t)t * A.heads + h0) * row;
    for (int h = wid; h < G; h += kThreads / 32)
        for (int c = lane * 4; c < row; c += 128) cp_async16(sm.q + h * sm.qs + c, qa + (size_t)h * row + c);
    load(0, j0);
    cp_async_commit();
    for (int i = threadIdx.x; i < sm.g4; i += kThreads) { sm.m[i] = -INFINITY; sm.l[i] = 0.f; sm.fix[i] = 1.f; }
    for (int i = threadIdx.x; i < tile * sm.g4; i += kThreads) sm.w[i] = 0.f;
    const int pairs = A.rank_s / 2, sets = sm.g4 / 4 * pairs;
    const int gh = (G + 1) / 2, units = gh * (tile / 2);
    int LS = 1;
    while (LS < 32 && 2 * LS * units <= kThreads) LS *= 2;
    const int sub = threadIdx.x & (LS - 1);
    float acc[EP][4][2] = {};
    int buf = 0;
    for (int j = j0; j < j1; j += tile, buf ^= 1) {
        if (j + tile < j1) load(buf ^ 1, j + tile);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const KT* K = sm.k + (size_t)buf * tile * sm.ks;
        const int keys = min(tile, j1 - j);
        // scores: LS lanes share two heads x two rows
        for (int u0 = 0; u0 < units; u0 += kThreads / LS) {
            const int u = u0 + threadIdx.x / LS;
            const bool in = u < units;
            const int p = in ? u / gh * 2 : 0, h = in ? (u - u / gh * gh) * 2 : 0, hb = min(h + 1, G - 1);
            const KT *ka = K + p * sm.ks, *kb = ka + sm.ks;
            const float *qa0 = sm.q + h * sm.qs, *qb0 = sm.q + hb * sm.qs;
            float s[2][2] = {};
#pragma unroll 2
            for (int c = in ? sub : chunks; c < chunks; c += LS) {
                float x[CN], y[CN];
                Chunk16<KT>::load(ka + c * CN, x);
                Chunk16<KT>::load(kb + c * CN, y);
#pragma unroll
                for (int i = 0; i < CN; i += 4) {
                    const float4 v = *reinterpret_cast<const float4*>(qa0 + c * CN + i), w = *reinterpret_cast<const float4*>(qb0 + c * CN + i);
                    const float vv[4] = {v.x, v.y, v.z, v.w}, ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                    for (int k = 0; k < 4; k++) {
                        s[0][0] = fmaf(vv[k], x[i + k], s[0][0]);
                        s[0][1] = fmaf(vv[k], y[i + k], s[0][1]);
                        s[1][0] = fmaf(ww[k], x[i + k], s[1][0]);
                        s[1][1] = fmaf(ww[k], y[i + k], s[1][1]);
                    }
                }
            }
            for (int o = LS / 2; o > 0; o >>= 1) {
                s[0][0] += __shfl_xor_sync(MG_FULL_MASK, s[0][0], o);
                s[0][1] += __shfl_xor_sync(MG_FULL_MASK, s[0][1], o);
                s[1][0] += __shfl_xor_sync(MG_FULL_MASK, s[1][0], o);
                s[1][1] += __shfl_xor_sync(MG_FULL_MASK, s[1][1], o);
            }
            if (in && sub == 0) {
                sm.w[p * sm.g4 + h] = s[0][0];
                sm.w[(p + 1) * sm.g4 + h] = s[0][1];
                if (h + 1 < G) {
                    sm.w[p * sm.g4 + h + 1] = s[1][0];
                    sm.w[(p + 1) * sm.g4 + h + 1] = s[1][1];
                }
            }
        }
        __syncthreads();
        for (int h = wid; h < G; h += kThreads / 32) {          // a warp per head, lanes over the tile's rows
            const float m0 = sm.m[h];
            float mx = m0;
            for (int p = lane; p < keys; p += 32) mx = fmaxf(mx, sm.w[p * sm.g4 + h]);
            mx = warp_max(mx);
            float sum = 0.f;
            for (int p = lane; p < tile; p += 32) {
                const float e = p < keys ? expf(sm.w[p * sm.g4 + h] - mx) : 0.f;
                sm.w[p * sm.g4 + h] = e;
                sum += e;
            }
            sum = warp_sum(sum);
            __syncwarp();
            if (lane == 0) {
                const float f = expf(m0 - mx);
                sm.fix[h] = f;
                sm.m[h] = mx;
                sm.l[h] = sm.l[h] * f + sum;
            }
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < EP; e++) {
            const int s = threadIdx.x + e * kThreads;
            if (s < sets) {
                const int hq = s / pairs * 4, pr = (s - s / pairs * pairs) * 2;
                const float4 f = *reinterpret_cast<const float4*>(sm.fix + hq);
                const float ff[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
                for (int i = 0; i < 4; i++) { acc[e][i][0] *= ff[i]; acc[e][i][1] *= ff[i]; }
#pragma unroll 4
                for (int p = 0; p < keys; p++) {
                    const float2 c = pair_f32(K + p * sm.ks + pr);
                    const float4 w = *reinterpret_cast<const float4*>(sm.w + p * sm.g4 + hq);
                    const float ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                    for (int i = 0; i < 4; i++) {
                        acc[e][i][0] = fmaf(ww[i], c.x, acc[e][i][0]);
                        acc[e][i][1] = fmaf(ww[i], c.y, acc[e][i][1]);
                    }
                }
            }
        }
        __syncthreads();
    }
    const size_t at = ((size_t)t * a.splits + blockIdx.x) * A.heads + h0;
#pragma unroll
    for (int e = 0; e < EP; e++) {
        const int s = threadIdx.x + e * kThreads;
        if (s >= sets) continue;
        const int hq = s / pairs * 4, pr = (s - s / pairs * pairs) * 2;
#pragma unroll
        for (int i = 0; i < 4; i++)
            if (hq + i < G) *reinterpret_cast<float2*>(a.part + (at + hq + i) * A.rank_s + pr) = make_float2(acc[e][i][0], acc[e][i][1]);
    }
    for (int h = threadIdx.x; h < G; h += kThreads) a.ml[at + h] = make_float2(sm.m[h], sm.l[h]);
}

constexpr int kValueRows = 32;      // value dimensions per CTA, four per warp
constexpr int kValueGroups = 8;     // groups of threads that share the ranges, at most

// CTA (head, 32 value dimensions) of one token: joins the ranges, then U_v times the weighted sum of latents.
template <typename OT>
__global__ void __launch_bounds__(kThreads) latent_value_kernel(const LatentStep a) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float red[40];
    const LatentAttn& A = a.at;
    float* o = smem;                                // [groups][ld], zero from rank_s on
    float* f = smem + kValueGroups * A.ld;          // [splits]
    const int slices = (A.vdim + kValueRows - 1) / kValueRows, t = blockIdx.y;
    const int h = blockIdx.x / slices, v0 = (blockIdx.x - h * slices) * kValueRows;
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
    constexpr int RW = kValueRows / (kThreads / 32), AHEAD = 2;
    const int chunks = A.ld / 8;
    const __nv_bfloat16* uv = A.uv + (size_t)h * A.vdim * A.ld;
    uint4 w[RW][AHEAD];
#pragma unroll
    for (int r = 0; r < RW; r++)
#pragma unroll
        for (int c = 0; c < AHEAD; c++) {
            const int v = v0 + wid * RW + r, ch = c * 32 + lane;
            w[r][c] = v < A.vdim && ch < chunks ? ld_stream16(uv + (size_t)v * A.ld + ch * 8) : make_uint4(0u, 0u, 0u, 0u);
        }
    pdl_launch_dependents();
    pdl_wait();
    const int len = token_pos(a, t) + 1;
    if (len > A.max_seq) return;
    int j0, j1;
    const int active = key_split(len, a.splits, a.tile, 0, &j0, &j1);
    const float2* ml = a.ml + (size_t)t * a.splits * A.heads + h;
    // four latent values per thread, the ranges dealt out to `rows` groups of threads
    const float* part = a.part + ((size_t)t * a.splits * A.heads + h) * A.rank_s;
    const size_t stride = (size_t)A.heads * A.rank_s;
    const int quads = A.ld / 4, rows = min(kThreads / min(quads, kThreads), kValueGroups), grp = threadIdx.x / min(quads, kThreads);
    {   // factors of the ranges
        float mx = -INFINITY, sum = 0.f;
        const float2 mine = (int)threadIdx.x < active ? ml[(size_t)threadIdx.x * A.heads] : make_float2(-INFINITY, 0.f);
        for (int s = threadIdx.x; s < active; s += kThreads) mx = fmaxf(mx, s < kThreads ? mine.x : ml[(size_t)s * A.heads].x);
        mx = block_max(mx, red);
        for (int s = threadIdx.x; s < active; s += kThreads) {
            const float2 p = s < kThreads ? mine : ml[(size_t)s * A.heads];
            f[s] = expf(p.x - mx);
            sum += f[s] * p.y;
        }
        const float inv = 1.0f / block_sum(sum, red);
        for (int s = threadIdx.x; s < active; s += kThreads) f[s] *= inv;
    }
    __syncthreads();
    if (grp < rows)
        for (int i = (threadIdx.x - grp * min(quads, kThreads)) * 4; i < A.ld; i += kThreads * 4) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i < A.rank_s) {
                constexpr int N = 16;               // ranges in flight
                for (int s0 = grp; s0 < active; s0 += N * rows) {
                    float4 p[N];
#pragma unroll
                    for (int q = 0; q < N; q++)
                        p[q] = s0 + q * rows < active ? *reinterpret_cast<const float4*>(part + (s0 + q * rows) * stride + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                    for (int q = 0; q < N; q++) {
                        const float w = s0 + q * rows < active ? f[s0 + q * rows] : 0.f;
                        v.x = fmaf(w, p[q].x, v.x); v.y = fmaf(w, p[q].y, v.y); v.z = fmaf(w, p[q].z, v.z); v.w = fmaf(w, p[q].w, v.w);
                    }
                }
            }
            *reinterpret_cast<float4*>(o + grp * A.ld + i) = v;
        }
    __syncthreads();
    for (int i = threadIdx.x; rows > 1 && i < A.ld; i += kThreads) {
        float v = o[i];
        for (int g = 1; g < rows; g++) v += o[g * A.ld + i];
        o[i] = v;
    }
    __syncthreads();
    auto dot = [&](uint4 u, int ch) {
        const float4 x = *reinterpret_cast<const float4*>(o + ch * 8), y = *reinterpret_cast<const float4*>(o + ch * 8 + 4);
        float s = __uint_as_float(u.x << 16) * x.x;
        s = fmaf(__uint_as_float(u.x & 0xffff0000u), x.y, s);
        s = fmaf(__uint_as_float(u.y << 16), x.z, s);
        s = fmaf(__uint_as_float(u.y & 0xffff0000u), x.w, s);
        s = fmaf(__uint_as_float(u.z << 16), y.x, s);
        s = fmaf(__uint_as_float(u.z & 0xffff0000u), y.y, s);
        s = fmaf(__uint_as_float(u.w << 16), y.z, s);
        return fmaf(__uint_as_float(u.w & 0xffff0000u), y.w, s);
    };
#pragma unroll
    for (int r = 0; r < RW; r++) {
        const int v = v0 + wid * RW + r;
        if (v >= A.vdim) continue;
        float s = 0.f;
#pragma unroll
        for (int c = 0; c < AHEAD; c++)
            if (c * 32 + lane < chunks) s += dot(w[r][c], c * 32 + lane);
        for (int ch = AHEAD * 32 + lane; ch < chunks; ch += 32) s += dot(ld_stream16(uv + (size_t)v * A.ld + ch * 8), ch);
        s = warp_sum(s);
        if (lane == 0) from_f32(s, static_cast<OT*>(a.out) + (size_t)t * a.ld_out + h * A.vdim + v);
    }
}

// One CTA per row of a portion.
template <typename AT>
__global__ void __launch_bounds__(kThreads) latent_rows_kernel(const LatentAttn A, const float* down, int ldd, int pos0, AT* act, int ld_act) {
    __shared__ float red[40];
    const float* q = down + (size_t)blockIdx.x * ldd;
    float ss = 0.f;
    for (int i = threadIdx.x; i < A.q_rank; i += kThreads) ss = fmaf(q[i], q[i], ss);
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)A.q_rank + A.eps);
    for (int i = threadIdx.x; i < A.q_rank; i += kThreads) from_f32(q[i] * r * A.q_norm[i], act + (size_t)blockIdx.x * ld_act + i);
    store_latent<AT>(A, q + A.q_rank, pos0 + blockIdx.x, red);
}

__global__ void __launch_bounds__(kThreads) latent_q_rows_kernel(const LatentAttn A, const float* q, int pos0, float scale, __nv_bfloat16* qh) {
    const int row = A.heads * A.qrow(), qr = A.qrow();
    const float* src = q + (size_t)blockIdx.x * row;
    __nv_bfloat16* dst = qh + (size_t)blockIdx.x * row;
    for (int i = threadIdx.x; i < row; i += kThreads) {
        const int d = i % qr - A.dim_s;
        float v = src[i];
        if (d >= 0) v = d < A.rot ? rotated(A, src + i - d, pos0 + blockIdx.x, d) : 0.f;
        dst[i] = __float2bfloat16_rn(v * scale);
    }
}

// Accumulator sets per thread (rounded up to an instance), 0 when one CTA cannot hold the heads.
int attend_sets(const LatentAttn& at, int group) {
    const int sets = pad_to(group, 4) / 4 * (at.rank_s / 2), ep = (sets + kThreads - 1) / kThreads;
    for (int p = 1; p <= 8; p *= 2)
        if (ep <= p) return p;
    return 0;
}

template <typename KT>
cudaError_t attend_for(const LatentStep& a, size_t smem, bool pdl, cudaStream_t s) {
    const dim3 grid(a.splits, (a.at.heads + a.group - 1) / a.group, a.tokens);
    auto run = [&](auto kern) {
        cudaError_t c = cudaFuncSetAttribute((const void*)kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        return c != cudaSuccess ? c : launch_pdl(kern, grid, kThreads, smem, pdl, s, a);
    };
    switch (attend_sets(a.at, a.group)) {
        case 1: return run(latent_attend_kernel<KT, 1>);
        case 2: return run(latent_attend_kernel<KT, 2>);
        case 4: return run(latent_attend_kernel<KT, 4>);
        case 8: return run(latent_attend_kernel<KT, 8>);
    }
    return cudaErrorInvalidValue;
}

}  // namespace

size_t latent_attend_smem(const LatentAttn& at, bool f32_cache, int* tile, int* group) {
    const size_t kt = f32_cache ? 4 : 2;
    // as many heads as fit 4 sets per thread, so that the cached rows are read by few CTAs
    for (int g = std::min(at.heads, 32);; g = (g + 1) / 2) {
        const int ep = attend_sets(at, g);
        if (ep && (ep <= 4 || g == 1))
            for (int t = 16; t >= 2; t /= 2) {
                const size_t b = 2 * (size_t)t * (at.row() * kt + 16) + ((size_t)g * (at.row() + 4) + (size_t)(t + 3) * pad_to(g, 4)) * sizeof(float);
                if (b <= 200 * 1024) { *tile = t; *group = g; return b; }
            }
        if (g == 1) return 0;
    }
}

cudaError_t launch_latent_query(const LatentStep& a, bool f32_cache, bool pdl, cudaStream_t s) {
    const dim3 grid(a.at.heads * ((a.at.rank_s + kFoldCols - 1) / kFoldCols) + (a.down ? 1 : 0), a.tokens);
    return f32_cache ? launch_pdl(latent_query_kernel<float>, grid, kThreads, 0, pdl, s, a)
                     : launch_pdl(latent_query_kernel<__nv_bfloat16>, grid, kThreads, 0, pdl, s, a);
}

cudaError_t launch_latent_attend(const LatentStep& a, bool f32_cache, bool pdl, cudaStream_t s) {
    int tile, group;
    const size_t smem = latent_attend_smem(a.at, f32_cache, &tile, &group);
    if (!smem || tile != a.tile || group != a.group) return cudaErrorInvalidValue;
    return f32_cache ? attend_for<float>(a, smem, pdl, s) : attend_for<__nv_bfloat16>(a, smem, pdl, s);
}

cudaError_t launch_latent_value(const LatentStep& a, bool f32_out, bool pdl, cudaStream_t s) {
    const dim3 grid(a.at.heads * ((a.at.vdim + kValueRows - 1) / kValueRows), a.tokens);
    const size_t smem = (size_t)(kValueGroups * a.at.ld + a.splits) * sizeof(float);
    if (smem > 48 * 1024) {
        cudaError_t c = cudaFuncSetAttribute(f32_out ? (const void*)latent_value_kernel<float> : (const void*)latent_value_kernel<__nv_bfloat16>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (c != cudaSuccess) return c;
    }
    return f32_out ? launch_pdl(latent_value_kernel<float>, grid, kThreads, smem, pdl, s, a)
                   : launch_pdl(latent_value_kernel<__nv_bfloat16>, grid, kThreads, smem, pdl, s, a);
}

cudaError_t launch_latent_rows(const LatentAttn& at, const float* down, int ldd, int pos0, int n, void* act, int ld_act, bool f32, cudaStream_t s) {
    if (f32) latent_rows_kernel<float><<<n, kThreads, 0, s>>>(at, down, ldd, pos0, (float*)act, ld_act);
    else latent_rows_kernel<__nv_bfloat16><<<n, kThreads, 0, s>>>(at, down, ldd, pos0, (__nv_bfloat16*)act, ld_act);
    return cudaGetLastError();
}

cudaError_t launch_latent_q_rows(const LatentAttn& at, const float* q, int pos0, int n, void* qh, cudaStream_t s) {
    latent_q_rows_kernel<<<n, kThreads, 0, s>>>(at, q, pos0, at.scale * 1.4426950408889634f, (__nv_bfloat16*)qh);
    return cudaGetLastError();
}

}  // namespace mg
