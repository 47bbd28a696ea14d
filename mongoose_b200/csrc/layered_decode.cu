// One token of a layer-described model: bf16 instances of the phase kernels, and the mixer step, in
// which the attention branch (split over keys) and the matrix-memory branch run side by side.
#include "kernel_table.h"
#include "layered_ops.cuh"

namespace mg {

phase_fn_t layered_phase(int epi, int R) {
    switch (epi) {
        case EPI_GELU:
            return R == 4 ? phase_kernel<FMT_BF16, EPI_GELU, 4, 2> : R == 2 ? phase_kernel<FMT_BF16, EPI_GELU, 2, 4> : phase_kernel<FMT_BF16, EPI_GELU, 1, 8>;
        case EPI_LOGITS: return phase_kernel<FMT_BF16, EPI_LOGITS, 4, 2>;
        default:
            return R == 4 ? phase_kernel<FMT_BF16, EPI_STORE, 4, 2> : R == 2 ? phase_kernel<FMT_BF16, EPI_STORE, 2, 4> : phase_kernel<FMT_BF16, EPI_STORE, 1, 8>;
    }
}

phase_pair_fn_t layered_phase_pair(int R) {
    return R == 4 ? phase_pair_kernel<FMT_BF16, EPI_STORE, 4, 2> : R == 2 ? phase_pair_kernel<FMT_BF16, EPI_STORE, 2, 4> : phase_pair_kernel<FMT_BF16, EPI_STORE, 1, 8>;
}

phase_parts_fn_t layered_phase_parts(int R) {
    return R == 4 ? phase_parts_kernel<FMT_BF16, EPI_STORE, 4, 2> : R == 2 ? phase_parts_kernel<FMT_BF16, EPI_STORE, 2, 4> : phase_parts_kernel<FMT_BF16, EPI_STORE, 1, 8>;
}

namespace {

constexpr int kStateRows = 16;      // rows of the state a warp holds at a time

// One token of the matrix memory: CTA (head, slice of 32 value columns); lanes over columns, warps over
// the rows of the state.  Every slice forms the head's normaliser; slice 0 stores it into the other
// parity slot, so no slice reads what another writes.
__device__ __forceinline__ void mem_step(const MixerStep& a, int cta, float* smem) {
    const MatMem& M = a.mem;
    const int head = cta / a.vslices, slice = cta % a.vslices;
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    float* red = smem;                      // 40
    float* part = smem + 40;                // nw * 32
    float* ks = part + nw * 32;             // dim
    float* qs = ks + M.dim;                 // dim
    const int pos = a.st->pos;
    const bool fresh = pos == 0;
    const float* row = a.proj;
    const int v = slice * 32 + lane;
    float* S = M.S + (size_t)head * M.dim * M.vdim + v;
    // the state's rows come first: nothing they wait for is computed here
    float s0[kStateRows];
    auto load_rows = [&](int d0) {
#pragma unroll
        for (int i = 0; i < kStateRows; i++) {
            const int d = d0 + wid + i * nw;
            s0[i] = !fresh && v < M.vdim && d < M.dim ? S[(size_t)d * M.vdim] : 0.f;
        }
    };
    load_rows(0);
    const float vv = v < M.vdim ? row[a.c.mv + head * M.vdim + v] : 0.f;
    const float ig = soft_cap(row[a.c.mi + head] + M.i_bias[head], M.cap);
    const float fg = log_sigmoid(soft_cap(row[a.c.mf + head] + M.f_bias[head], M.cap));
    const int cur = pos & 1;
    const float m0 = fresh ? 0.f : M.m[cur * M.heads + head];
    const float m1 = fmaxf(fg + m0, ig);
    const float keep = expf(fg + m0 - m1), add = expf(ig - m1);
    const float qscale = 1.0f / sqrtf((float)M.dim);
    float nq = 0.f;
    for (int d = threadIdx.x; d < M.dim; d += blockDim.x) {
        const float k = row[a.c.mk + head * M.dim + d], q = row[a.c.mq + head * M.dim + d] * qscale;
        ks[d] = k * add;
        qs[d] = q;
        const float n0 = fresh ? 0.f : M.nrm[((size_t)cur * M.heads + head) * M.dim + d];
        const float n1 = keep * n0 + add * k;
        if (slice == 0) M.nrm[((size_t)(cur ^ 1) * M.heads + head) * M.dim + d] = n1;
        nq = fmaf(n1, q, nq);
    }
    nq = block_sum(nq, red);                // its barriers publish ks and qs
    if (slice == 0 && threadIdx.x == 0) M.m[(cur ^ 1) * M.heads + head] = m1;
    float acc = 0.f;
    for (int d0 = 0; d0 < M.dim; d0 += kStateRows * nw) {
        if (d0 > 0) load_rows(d0);
#pragma unroll
        for (int i = 0; i < kStateRows; i++) {
            const int d = d0 + wid + i * nw;
            if (v < M.vdim && d < M.dim) {
                const float s1 = fmaf(ks[d], vv, keep * s0[i]);
                S[(size_t)d * M.vdim] = s1;
                acc = fmaf(s1, qs[d], acc);
            }
        }
    }
    part[wid * 32 + lane] = acc;
    __syncthreads();
    if (wid == 0 && v < M.vdim) {
        float o = 0.f;
        for (int w = 0; w < nw; w++) o += part[w * 32 + lane];
        a.mem_o[head * M.vdim + v] = o / (fmaxf(fabsf(nq), expf(-m1)) + 1e-6f);
    }
}

template <typename KT, int EP>
__global__ void __launch_bounds__(kAttnThreads) mixer_step_kernel(const MixerStep a) {
    extern __shared__ __align__(16) float smem[];
    pdl_launch_dependents();
    pdl_wait();
    if ((int)blockIdx.x < a.n_mem) {
        mem_step(a, blockIdx.x, smem);
        return;
    }
    const GateAttn& A = a.at;
    const int pos = a.st->pos, len = pos + 1;
    if (pos >= A.max_seq) return;
    const int split = blockIdx.x - a.n_mem;
    int j0, j1;
    const int active = key_split(len, a.splits, a.tile, split, &j0, &j1);
    if (split >= active) return;
    const AttnSmem<KT> sm(A, 1, a.tile, smem);
    // this token's query, and its key where this CTA's range ends with it
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const float temp = query_temp(A, pos);
    norm_queries(A, a.proj + a.c.q, temp, sm.q, sm.qs);
    if (j1 == len)
        for (int c = wid; c < A.kv_heads; c += nw) store_key<KT>(A, a.proj + a.c.k + c * A.dim, pos, c, lane);
    sm.load_tables(A);
    __syncthreads();                        // the cache row above is read back by this CTA only
    float acc[1][EP][2] = {};
    attend<KT, 1, EP>(A, sm, pos, j0, j1, a.tile, acc);
#pragma unroll
    for (int p = 0; p < EP; p++) {
        const int e = 2 * (threadIdx.x + p * kAttnThreads);
        if (e < A.heads * A.dim_s)
            *reinterpret_cast<float2*>(a.part + (size_t)split * A.heads * A.dim_s + e) = make_float2(acc[0][p][0], acc[0][p][1]);
    }
}

constexpr int kJoinCols = 32, kJoinParts = 8;      // outputs per CTA, threads that share one output's splits

// Joins the key splits, and norms and gates the memory's outputs (one CTA per memory head).
__global__ void __launch_bounds__(kJoinCols * kJoinParts) mixer_join_kernel(const MixerStep a) {
    __shared__ float red[40];
    pdl_launch_dependents();
    pdl_wait();
    const MatMem& M = a.mem;
    const int nm = a.n_mem ? M.heads : 0;
    if ((int)blockIdx.x < nm) {
        const int head = blockIdx.x;
        const float* o = a.mem_o + head * M.vdim;
        float ss = 0.f;
        for (int v = threadIdx.x; v < M.vdim; v += blockDim.x) ss = fmaf(o[v], o[v], ss);
        const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)M.vdim + M.eps);
        for (int v = threadIdx.x; v < M.vdim; v += blockDim.x) {
            const int c = head * M.vdim + v;
            a.mem_y[c] = o[v] * r * M.norm[c] * sigmoid(a.proj[a.c.mg + c]);
        }
        return;
    }
    const GateAttn& A = a.at;
    const int col = threadIdx.x % kJoinCols, grp = threadIdx.x / kJoinCols;
    const int e = (blockIdx.x - nm) * kJoinCols + col;
    const bool ok = e < A.heads * A.dim;
    int j0, j1;
    const int active = key_split(a.st->pos + 1, a.splits, a.tile, 0, &j0, &j1);
    const int src = ok ? e / A.dim * A.dim_s + e % A.dim : 0;
    const size_t stride = (size_t)A.heads * A.dim_s;
    float v = 0.f;
    if (ok) {
#pragma unroll 8
        for (int s = grp; s < active; s += kJoinParts) v += a.part[s * stride + src];
    }
    __shared__ float sum[kJoinParts][kJoinCols];
    sum[grp][col] = v;
    __syncthreads();
    if (grp == 0 && ok) {
#pragma unroll
        for (int g = 1; g < kJoinParts; g++) v += sum[g][col];
        a.attn_out[e] = v;
    }
}

__global__ void __launch_bounds__(256) resolve_kernel(const ResolveArgs a) {
    extern __shared__ __align__(16) float smem[];
    pdl_launch_dependents();
    pdl_wait();
    stage_layered(a.p, smem, smem + a.p.K, false);
    for (int i = threadIdx.x; i < a.p.k_valid; i += blockDim.x) a.out[i] = smem[i];
}

template <typename KT>
cudaError_t step_for(const MixerStep& a, size_t smem, bool pdl, cudaStream_t s) {
    const int ep = attn_pairs(a.at);
    const int grid = a.n_mem + a.splits;
    auto run = [&](auto kern) {
        cudaError_t c = cudaFuncSetAttribute((const void*)kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        return c != cudaSuccess ? c : launch_pdl(kern, grid, kAttnThreads, smem, pdl, s, a);
    };
    switch (ep) {
        case 1: return run(mixer_step_kernel<KT, 1>);
        case 2: return run(mixer_step_kernel<KT, 2>);
        case 4: return run(mixer_step_kernel<KT, 4>);
        case 8: return run(mixer_step_kernel<KT, 8>);
        case 16: return run(mixer_step_kernel<KT, 16>);
    }
    return cudaErrorInvalidValue;
}

}  // namespace

cudaError_t layered_phase_smem(size_t bytes) {
    for (int R = 1; R <= 4; R *= 2) {
        for (int epi : {EPI_STORE, EPI_GELU, EPI_LOGITS}) {
            cudaError_t c = cudaFuncSetAttribute((const void*)layered_phase(epi, R), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
            if (c != cudaSuccess) return c;
        }
        for (const void* f : {(const void*)layered_phase_pair(R), (const void*)layered_phase_parts(R)}) {
            cudaError_t c = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
            if (c != cudaSuccess) return c;
        }
    }
    return cudaSuccess;
}

size_t mixer_step_smem(const GateAttn& at, const MatMem& mem, bool f32_cache, int* tile) {
    const size_t need_mem = (40 + kAttnThreads + 2 * (size_t)mem.dim) * sizeof(float);
    const size_t need = attn_smem(at, 1, f32_cache ? 4 : 2, 8, tile);
    return need == 0 ? 0 : need > need_mem ? need : need_mem;
}

cudaError_t launch_mixer_step(const MixerStep& a, bool f32_cache, bool pdl, cudaStream_t s) {
    int tile;
    const size_t smem = mixer_step_smem(a.at, a.mem, f32_cache, &tile);
    return f32_cache ? step_for<float>(a, smem, pdl, s) : step_for<__nv_bfloat16>(a, smem, pdl, s);
}

cudaError_t launch_mixer_join(const MixerStep& a, bool pdl, cudaStream_t s) {
    const int nm = a.n_mem ? a.mem.heads : 0;
    return launch_pdl(mixer_join_kernel, nm + (a.at.heads * a.at.dim + kJoinCols - 1) / kJoinCols, kJoinCols * kJoinParts, 0, pdl, s, a);
}

cudaError_t launch_resolve(const ResolveArgs& a, bool pdl, cudaStream_t s) {
    const size_t smem = ((size_t)a.p.K + 72) * sizeof(float);
    cudaError_t c = cudaFuncSetAttribute((const void*)resolve_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return c != cudaSuccess ? c : launch_pdl(resolve_kernel, 1, 256, smem, pdl, s, a);
}

}  // namespace mg
