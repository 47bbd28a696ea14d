// Mixture of experts: the choice (the largest router logits, weights by a softmax over them, fp32), and the chosen
// experts.  One token streams the chosen experts' rows where they lie; a prompt's tokens are grouped by expert
// into row tiles of 128, each tile one expert's, and go through grouped products (gemm_tc, or launch_gemm_f32).
#include <algorithm>

#include "layered_ops.cuh"

namespace mg {

namespace {

constexpr int kThreads = 256;

// Order of floats as unsigned integers.
__device__ __forceinline__ unsigned ordered(float v) {
    const unsigned u = __float_as_uint(v);
    return u & 0x80000000u ? ~u : u | 0x80000000u;
}

// One warp: the `top` largest of z[0..experts) in falling order and the softmax over them.  z, sel and wt are shared
// memory.  Whatever z holds, the chosen indices are distinct and valid.
__device__ __forceinline__ void choose(const float* z, int experts, int top, int* sel, float* wt, int lane) {
    unsigned taken = 0;                     // of this lane's entries lane, lane + 32, ...
    float first = 0.f, sum = 0.f;
    for (int k = 0; k < top; k++) {
        int bi = -1;
        unsigned bv = 0;
        for (int i = lane, q = 0; i < experts; i += 32, q++) {
            const unsigned v = ordered(z[i]);
            if (!((taken >> q) & 1u) && (bi < 0 || v > bv)) { bi = i; bv = v; }
        }
        const unsigned best = __reduce_max_sync(MG_FULL_MASK, bi < 0 ? 0u : bv);
        const int from = __ffs(__ballot_sync(MG_FULL_MASK, bi >= 0 && bv == best)) - 1;
        bi = __shfl_sync(MG_FULL_MASK, bi, from);
        if ((bi & 31) == lane) taken |= 1u << (bi >> 5);
        const float v = z[bi];
        if (k == 0) first = v;
        const float e = expf(v - first);
        sum += e;
        if (lane == 0) { sel[k] = bi; wt[k] = e; }
    }
    __syncwarp();
    for (int k = lane; k < top; k += 32) wt[k] /= sum;
    __syncwarp();
}
static_assert(kMaxExperts <= 32 * 32, "a lane marks its entries in 32 bits");

// Choice of one token, by the whole CTA (every CTA for itself).  zs: `experts` floats.
__device__ __forceinline__ void choose_cta(const Moe& m, const float* router, float* zs, int* sel, float* wt) {
    for (int i = threadIdx.x; i < m.experts; i += blockDim.x) zs[i] = router[i] + m.bias[i];
    __syncthreads();
    if (threadIdx.x < 32) choose(zs, m.experts, m.top, sel, wt, threadIdx.x);
    __syncthreads();
}

// The vector that the down matrices read: per chosen expert silu(gate row . h) * (up row . h) times its weight, then the
// shared expert's inner vector times its gate; parts are padded like the matrices' rows.  A warp per (expert, row).
__global__ void __launch_bounds__(kThreads) moe_up_kernel(const MoeStep a) {
    extern __shared__ __align__(16) float smem[];
    __shared__ int sel[kMaxTop];
    __shared__ float wt[kMaxTop];
    const Moe& m = a.moe;
    float* hs = smem;                       // [ldw]
    float* zs = smem + m.ldw;               // [experts]
    pdl_launch_dependents();
    pdl_wait();
    for (int i = threadIdx.x * 4; i < m.ldw; i += kThreads * 4) cp_async16(hs + i, a.h + i);
    cp_async_commit();
    choose_cta(m, a.router, zs, sel, wt);
    if (blockIdx.x == 0)
        for (int k = threadIdx.x; k < m.top; k += kThreads) a.sel[k] = sel[k];
    cp_async_wait<0>();
    __syncthreads();
    const int lane = threadIdx.x & 31, nw = gridDim.x * (kThreads / 32), chunks = m.ldw / 8, items = m.top * m.ff;
    for (int it = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5); it < items; it += nw) {
        const int k = it / m.ff, f = it - k * m.ff;
        const size_t row = (size_t)sel[k] * m.ff + f;
        const uint4* g = reinterpret_cast<const uint4*>(m.gate + row * m.ldw * 2);
        const uint4* u = reinterpret_cast<const uint4*>(m.up + row * m.ldw * 2);
        float sg = 0.f, su = 0.f;
        for (int c0 = 0; c0 < chunks; c0 += 128) {
            uint4 wg[4], wu[4];
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const int c = c0 + i * 32 + lane;
                wg[i] = c < chunks ? ld_stream16(g + c) : make_uint4(0u, 0u, 0u, 0u);
                wu[i] = c < chunks ? ld_stream16(u + c) : make_uint4(0u, 0u, 0u, 0u);
            }
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const int c = c0 + i * 32 + lane;
                if (c < chunks) {
                    const float4 x[2] = {*reinterpret_cast<const float4*>(hs + c * 8), *reinterpret_cast<const float4*>(hs + c * 8 + 4)};
                    sg += Chunk<FMT_BF16>::dot(wg[i], x);
                    su += Chunk<FMT_BF16>::dot(wu[i], x);
                }
            }
        }
        sg = warp_sum(sg);
        su = warp_sum(su);
        if (lane == 0) a.mid[k * m.ffs + f] = silu(sg) * su * wt[k];
    }
    if (m.shared_ff) {
        const float *g = a.router + m.sg_col() + 1, *u = g + m.shared_ff;
        for (int i = blockIdx.x * kThreads + threadIdx.x; i < m.shared_ff; i += gridDim.x * kThreads)
            a.mid[m.top * m.ffs + i] = silu(g[i]) * u[i] * sigmoid(a.router[m.sg_col()]);
    }
}

// out = the chosen experts' down matrices and the shared one, side by side, times that vector.  A CTA takes R rows at
// a time, its warps share their columns, and the first rows' weights are on the way before the vector is there.
template <int R>
__global__ void __launch_bounds__(kThreads) moe_down_kernel(const MoeStep a) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float part[2][kThreads / 32][R];
    __shared__ int sel[kMaxTop];
    constexpr int AHEAD = 3;
    const Moe& m = a.moe;
    float* xs = smem;                                   // [top * ffs + shared_ffs]
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
    const int per = m.ffs / 8, own = m.top * per, chunks = own + m.shared_ffs / 8;
    pdl_launch_dependents();
    pdl_wait();
    for (int i = threadIdx.x * 4; i < chunks * 8; i += kThreads * 4) cp_async16(xs + i, a.mid + i);
    cp_async_commit();
    for (int k = threadIdx.x; k < m.top; k += kThreads) sel[k] = a.sel[k];
    __syncthreads();
    auto load = [&](int c, int r0, uint4 (&w)[R]) {
        const int k = c / per;
#pragma unroll
        for (int r = 0; r < R; r++) {
            const size_t row = min(r0 + r, m.width - 1);
            w[r] = c >= chunks ? make_uint4(0u, 0u, 0u, 0u)
                 : c < own ? ld_stream16(m.down + (((size_t)sel[k] * m.width + row) * per + (c - k * per)) * 16)
                           : ld_stream16(m.shared_down + (row * (m.shared_ffs / 8) + (c - own)) * 16);
        }
    };
    uint4 w[AHEAD][R];
    int r0 = blockIdx.x * R;
#pragma unroll
    for (int i = 0; i < AHEAD; i++) load(threadIdx.x + i * kThreads, r0, w[i]);
    cp_async_wait<0>();
    __syncthreads();
    for (int buf = 0; r0 < m.width; r0 += gridDim.x * R, buf ^= 1) {
        float acc[R] = {};
        auto use = [&](int c, const uint4 (&v)[R]) {
            if (c < chunks) {
                const float4 x[2] = {*reinterpret_cast<const float4*>(xs + c * 8), *reinterpret_cast<const float4*>(xs + c * 8 + 4)};
#pragma unroll
                for (int r = 0; r < R; r++) acc[r] += Chunk<FMT_BF16>::dot(v[r], x);
            }
        };
        const int next = r0 + gridDim.x * R;
#pragma unroll
        for (int i = 0; i < AHEAD; i++) use(threadIdx.x + i * kThreads, w[i]);
        for (int c = threadIdx.x + AHEAD * kThreads; c < chunks; c += AHEAD * kThreads) {
#pragma unroll
            for (int i = 0; i < AHEAD; i++) load(c + i * kThreads, r0, w[i]);
#pragma unroll
            for (int i = 0; i < AHEAD; i++) use(c + i * kThreads, w[i]);
        }
        if (next < m.width) {
#pragma unroll
            for (int i = 0; i < AHEAD; i++) load(threadIdx.x + i * kThreads, next, w[i]);
        }
#pragma unroll
        for (int r = 0; r < R; r++) {
            const float v = warp_sum(acc[r]);
            if (lane == 0) part[buf][wid][r] = v;
        }
        __syncthreads();
        if (threadIdx.x < R && r0 + threadIdx.x < m.width) {
            float v = 0.f;
#pragma unroll
            for (int q = 0; q < kThreads / 32; q++) v += part[buf][q][threadIdx.x];
            a.out[r0 + threadIdx.x] = v;
        }
    }
}

// ---- prompts ----

// A warp per token: choice, and the token's place among those of its expert.
__global__ void __launch_bounds__(kThreads) moe_choose_kernel(const Moe m, const float* router, int ldr, int slices, int n, MoeRows w) {
    extern __shared__ __align__(16) float smem[];
    __shared__ int sel[kThreads / 32][kMaxTop];
    __shared__ float wt[kThreads / 32][kMaxTop];
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * (kThreads / 32) + wid;
    if (t >= n) return;
    float* z = smem + wid * m.experts;
    for (int i = lane; i < m.experts + (m.shared_ff ? 1 : 0); i += 32) {
        float v = 0.f;
        for (int s = 0; s < slices; s++) v += router[((size_t)s * n + t) * ldr + i];
        if (i < m.experts) z[i] = v + m.bias[i];
        else w.shared_gate[t] = sigmoid(v);
    }
    __syncwarp();
    choose(z, m.experts, m.top, sel[wid], wt[wid], lane);
    for (int k = lane; k < m.top; k += 32) {
        const int e = sel[wid][k];
        w.sel[(size_t)t * m.top + k] = e;
        w.weight[(size_t)t * m.top + k] = wt[wid][k];
        w.slot[(size_t)t * m.top + k] = atomicAdd(w.count + e, 1);      // which place a token gets does not change its result
    }
}

// One CTA: first row of every expert (whole tiles of 128), the expert of every tile; clears the counts.
__global__ void __launch_bounds__(1024) moe_plan_kernel(const Moe m, MoeRows w) {
    __shared__ int tiles[kMaxExperts], first[kMaxExperts + 1];
    for (int e = threadIdx.x; e < m.experts; e += blockDim.x) {
        tiles[e] = (w.count[e] + 127) / 128;
        w.count[e] = 0;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int at = 0;
        for (int e = 0; e < m.experts; e++) { first[e] = at; at += tiles[e]; }
        first[m.experts] = at;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < m.experts; e += blockDim.x) {
        w.first[e] = first[e] * 128;
        for (int i = first[e]; i < first[e + 1] && i < w.tiles; i++) w.group[i] = e;
    }
    for (int i = first[m.experts] + threadIdx.x; i < w.tiles; i += blockDim.x) w.group[i] = -1;
}

// A CTA per token: its row to its place in every chosen expert's group; slot becomes the grouped row.
__global__ void __launch_bounds__(128) moe_gather_kernel(const Moe m, const uint4* act, int units, MoeRows w) {
    const size_t t = blockIdx.x;
    for (int k = 0; k < m.top; k++) {
        const size_t at = t * m.top + k;
        const int row = w.first[w.sel[at]] + w.slot[at];
        uint4* dst = static_cast<uint4*>(w.x) + (size_t)row * units;
        for (int i = threadIdx.x; i < units; i += 128) dst[i] = act[t * units + i];
    }
}

template <typename AT, int V>
__global__ void __launch_bounds__(kThreads) moe_combine_kernel(const Moe m, MoeRows w, float* z) {
    __shared__ float wt[kMaxTop];
    __shared__ int row[kMaxTop];
    const size_t t = blockIdx.x;
    for (int k = threadIdx.x; k < m.top; k += kThreads) {
        wt[k] = w.weight[t * m.top + k];
        row[k] = w.first[w.sel[t * m.top + k]] + w.slot[t * m.top + k];
    }
    __syncthreads();
    const AT* y = static_cast<const AT*>(w.y);
    const float sg = m.shared_ff ? w.shared_gate[t] : 0.f;
    float* out = z + t * m.width;
    for (int i = threadIdx.x * V; i < m.width; i += kThreads * V) {
        float v[V] = {};
        if (m.shared_ff) {
            load_values<V>(out + i, v);
#pragma unroll
            for (int q = 0; q < V; q++) v[q] *= sg;
        }
#pragma unroll 4
        for (int k = 0; k < m.top; k++) {
            float e[V];
            load_values<V>(y + (size_t)row[k] * m.width + i, e);
#pragma unroll
            for (int q = 0; q < V; q++) v[q] = fmaf(wt[k], e[q], v[q]);
        }
        store_values<V>(v, out + i);
    }
}

constexpr int kDownRows = 4;

}  // namespace

size_t moe_step_smem(const Moe& m) { return (size_t)std::max(m.ldw + m.experts, m.top * m.ffs + m.shared_ffs) * sizeof(float); }

cudaError_t moe_step_attrs(size_t bytes) {
    cudaError_t c = cudaFuncSetAttribute((const void*)moe_up_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    return c != cudaSuccess ? c : cudaFuncSetAttribute((const void*)moe_down_kernel<kDownRows>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

cudaError_t launch_moe_up(const MoeStep& a, int sms, bool pdl, cudaStream_t s) {
    const int grid = std::min((a.moe.top * a.moe.ff + 7) / 8, 2 * sms);
    return launch_pdl(moe_up_kernel, grid, kThreads, (size_t)(a.moe.ldw + a.moe.experts) * sizeof(float), pdl, s, a);
}

cudaError_t launch_moe_down(const MoeStep& a, int sms, bool pdl, cudaStream_t s) {
    const Moe& m = a.moe;
    const size_t smem = (size_t)(m.top * m.ffs + m.shared_ffs) * sizeof(float);
    const int per_sm = std::max(1, std::min(2, (int)(220 * 1024 / (smem + 2048))));     // CTAs that share an SM
    const int grid = std::min((m.width + kDownRows - 1) / kDownRows, per_sm * sms);
    return launch_pdl(moe_down_kernel<kDownRows>, grid, kThreads, smem, pdl, s, a);
}

cudaError_t launch_moe_route(const Moe& m, const float* router, int ldr, int slices, int n, const void* act, bool f32, const MoeRows& w, cudaStream_t s) {
    moe_choose_kernel<<<(n + 7) / 8, kThreads, (size_t)8 * m.experts * sizeof(float), s>>>(m, router, ldr, slices, n, w);
    moe_plan_kernel<<<1, 1024, 0, s>>>(m, w);
    moe_gather_kernel<<<n, 128, 0, s>>>(m, (const uint4*)act, m.ldw * (f32 ? 4 : 2) / 16, w);
    return cudaGetLastError();
}

cudaError_t launch_moe_combine(const Moe& m, int n, const MoeRows& w, float* z, bool f32, cudaStream_t s) {
    const bool quads = m.width % 4 == 0;
    if (f32 && quads) moe_combine_kernel<float, 4><<<n, kThreads, 0, s>>>(m, w, z);
    else if (f32) moe_combine_kernel<float, 1><<<n, kThreads, 0, s>>>(m, w, z);
    else if (quads) moe_combine_kernel<__nv_bfloat16, 4><<<n, kThreads, 0, s>>>(m, w, z);
    else moe_combine_kernel<__nv_bfloat16, 1><<<n, kThreads, 0, s>>>(m, w, z);
    return cudaGetLastError();
}

}  // namespace mg
