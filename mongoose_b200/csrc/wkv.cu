// Linear recurrence with a decay per key channel, S <- diag(w) S + k v^T, o = (S_before + diag(u) k v^T)^T r, in
// fp32.  The columns of a head's state (value channels) never meet, so a prompt runs the recurrence itself,
// token by token, with the columns of all heads spread over the GPU: no chunk's cumulative decay is ever formed,
// and decays of any strength are exact.
#include "layered_ops.cuh"

namespace mg {

namespace {

constexpr int kStepThreads = 256;
constexpr int kStepRows = 16;       // rows of the state a warp holds at a time

// One token: a CTA per head, lanes over value channels, warps over key channels.
__global__ void __launch_bounds__(kStepThreads) wkv_step_kernel(const WkvStep a) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float red[40];
    const Wkv& M = a.wk;
    const int D = M.dim, n = M.heads * D, c0 = blockIdx.x * D, rk = pad_to(M.rank, 8);
    float *r = smem, *k = r + D, *w = k + D, *v = w + D, *u = v + D, *inner = smem + pad_to(5 * D, 4);
    float* part = inner + rk;               // [warps][D]
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
    constexpr int nw = kStepThreads / 32;
    for (int i = threadIdx.x; i < D; i += kStepThreads) u[i] = M.u[c0 + i];
    pdl_launch_dependents();
    pdl_wait();
    const bool fresh = a.st->pos == 0;
    float* S = M.S + (size_t)blockIdx.x * D * D;
    float s0[kStepRows];
    auto load_rows = [&](int k0, int col) {
#pragma unroll
        for (int i = 0; i < kStepRows; i++) {
            const int d = k0 + wid + i * nw;
            s0[i] = !fresh && col < D && d < D ? S[(size_t)d * D + col] : 0.f;
        }
    };
    load_rows(0, lane);
    for (int i = threadIdx.x; i < D; i += kStepThreads) { r[i] = a.row[c0 + i]; k[i] = a.row[n + c0 + i]; v[i] = a.row[2 * n + c0 + i]; }
    for (int i = threadIdx.x; i < rk; i += kStepThreads) inner[i] = i < M.rank ? tanhf(a.row[4 * (size_t)n + i]) : 0.f;
    __syncthreads();
    // decays: four threads per channel
    const int sub = threadIdx.x & 3;
    for (int d0 = 0; d0 < D; d0 += kStepThreads / 4) {
        const int d = d0 + (threadIdx.x >> 2);
        float z = 0.f;
        if (d < D) {
            const __nv_bfloat16* wp = M.w2 + (size_t)(c0 + d) * M.ld2;
            for (int c = sub * 8; c < rk; c += 32) {
                float x[8];
                Chunk16<__nv_bfloat16>::load(wp + c, x);
#pragma unroll
                for (int i = 0; i < 8; i++) z = fmaf(x[i], inner[c + i], z);
            }
        }
        z += __shfl_xor_sync(MG_FULL_MASK, z, 1);
        z += __shfl_xor_sync(MG_FULL_MASK, z, 2);
        if (sub == 0 && d < D) w[d] = expf(-expf(z + M.w0[c0 + d]));
    }
    __syncthreads();
    for (int v0 = 0; v0 < D; v0 += 32) {
        const int col = v0 + lane;
        const float vv = col < D ? v[col] : 0.f;
        float o = 0.f;
        for (int k0 = 0; k0 < D; k0 += kStepRows * nw) {
            if (v0 > 0 || k0 > 0) load_rows(k0, col);
#pragma unroll
            for (int i = 0; i < kStepRows; i++) {
                const int d = k0 + wid + i * nw;
                if (d < D) {
                    const float kv = k[d] * vv;
                    o = fmaf(fmaf(u[d], kv, s0[i]), r[d], o);
                    if (col < D) S[(size_t)d * D + col] = fmaf(w[d], s0[i], kv);
                }
            }
        }
        if (col < D) part[wid * D + col] = o;
    }
    __syncthreads();
    float ss = 0.f;
    for (int i = threadIdx.x; i < D; i += kStepThreads) {
        float o = 0.f;
#pragma unroll
        for (int q = 0; q < nw; q++) o += part[q * D + i];
        part[i] = o;                        // row 0 of this column is read by this thread only
        ss = fmaf(o, o, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)D + M.eps);
    for (int i = threadIdx.x; i < D; i += kStepThreads)
        a.y[c0 + i] = part[i] * inv * M.norm[c0 + i] * silu(a.row[3 * (size_t)n + c0 + i]);
}

template <typename AT>
__global__ void __launch_bounds__(256) wkv_mix_kernel(const float* h, const float* prev, const float* m0, const float* m1, const float* m2,
                                                      const float* m3, const float* m4, int pos0, int width, AT* act, int ld_act,
                                                      long long stride) {
    const int t = blockIdx.x;
    const float* cur = h + (size_t)t * width;
    const float* before = t > 0 ? cur - width : prev + (size_t)(pos0 & 1) * width;
    const bool none = t == 0 && pos0 == 0;
    const float* mu[5] = {m0, m1, m2, m3, m4};
    for (int i = threadIdx.x; i < width; i += 256) {
        const float x = cur[i], d = (none ? 0.f : before[i]) - x;
#pragma unroll
        for (int j = 0; j < 5; j++) from_f32(fmaf(d, mu[j][i], x), act + j * stride + (size_t)t * ld_act + i);
    }
}

// ---- prompts ----
constexpr int kScanThreads = 128;

// KS lanes share a column of the state, KPT key channels each: lane j holds channels 4 (j + q KS) .. + 3.  Tokens
// come through shared memory in tiles; sums over key channels of KS tokens are reduced at once, which leaves
// lane j with token j's output.
template <int KPT, int KS>
struct Scan {
    static constexpr int cols = kScanThreads / KS;      // value channels per CTA
    static constexpr int rows = KPT * KS;               // key channels, padded
};

// A token in shared memory: r, k, w padded to `rows`, then the CTA's value channels.
template <int KPT, int KS>
__global__ void __launch_bounds__(kScanThreads) wkv_scan_kernel(const Wkv M, const float* proj, int ldp, const float* decay, int pos0, int n,
                                                                int tile, float* out) {
    extern __shared__ __align__(16) float smem[];
    using G = Scan<KPT, KS>;
    constexpr int Q = KPT / 4;
    const int D = M.dim, nh = M.heads * D, h = blockIdx.x, v0 = blockIdx.y * G::cols;
    const int sub = threadIdx.x % KS, col = threadIdx.x / KS, v = v0 + col;
    constexpr int per = 3 * G::rows + (G::cols + 3) / 4 * 4;
    const int cols = min(G::cols, D - v0);
    // the padding is zero and stays so
    for (int i = threadIdx.x; i < 2 * tile * per; i += kScanThreads) smem[i] = 0.f;
    __syncthreads();
    const bool wide = ((D | ldp) & 3) == 0;
    auto load = [&](int buf, int t0) {
        const int T = min(tile, n - t0);
        float* dst = smem + (size_t)buf * tile * per;
        const int step = wide ? 4 : 1, units = D / step;
        for (int i = threadIdx.x; i < T * units; i += kScanThreads) {
            const int t = i / units, c = (i - t * units) * step;
            const float* row = proj + (size_t)(t0 + t) * ldp + h * D + c;
            const float* dw = decay + (size_t)(t0 + t) * nh + h * D + c;
            float* to = dst + t * per + c;
            if (wide) {
                cp_async16(to, row);
                cp_async16(to + G::rows, row + nh);
                cp_async16(to + 2 * G::rows, dw);
            } else {
                cp_async4(to, row);
                cp_async4(to + G::rows, row + nh);
                cp_async4(to + 2 * G::rows, dw);
            }
        }
        for (int i = threadIdx.x; i < T * cols; i += kScanThreads) {
            const int t = i / cols, c = i - t * cols;
            cp_async4(dst + t * per + 3 * G::rows + c, proj + (size_t)(t0 + t) * ldp + 2 * (size_t)nh + h * D + v0 + c);
        }
    };
    load(0, 0);
    cp_async_commit();
    float S[KPT], u[KPT];
#pragma unroll
    for (int i = 0; i < KPT; i++) {
        const int d = 4 * (sub + i / 4 * KS) + i % 4;
        const bool in = d < D && v < D;
        u[i] = d < D ? M.u[h * D + d] : 0.f;
        S[i] = in && pos0 > 0 ? M.S[((size_t)h * D + d) * D + v] : 0.f;
    }
    int buf = 0;
    for (int t0 = 0; t0 < n; t0 += tile, buf ^= 1) {
        if (t0 + tile < n) load(buf ^ 1, t0 + tile);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const float* base = smem + (size_t)buf * tile * per;
        const int T = min(tile, n - t0);
        for (int g = 0; g < T; g += KS) {
            float o[KS];
#pragma unroll
            for (int j = 0; j < KS; j++) {
                o[j] = 0.f;
                if (g + j < T) {
                    const float* p = base + (g + j) * per + 4 * sub;
                    const float vv = base[(g + j) * per + 3 * G::rows + col];
#pragma unroll
                    for (int q = 0; q < Q; q++) {
                        const float4 r4 = *reinterpret_cast<const float4*>(p + 4 * q * KS), k4 = *reinterpret_cast<const float4*>(p + G::rows + 4 * q * KS),
                                     w4 = *reinterpret_cast<const float4*>(p + 2 * G::rows + 4 * q * KS);
                        const float rr[4] = {r4.x, r4.y, r4.z, r4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w}, ww[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            const float kv = kk[i] * vv;
                            o[j] = fmaf(fmaf(u[4 * q + i], kv, S[4 * q + i]), rr[i], o[j]);
                            S[4 * q + i] = fmaf(ww[i], S[4 * q + i], kv);
                        }
                    }
                }
            }
            // halves exchange until lane `sub` holds token `sub`'s sum
#pragma unroll
            for (int m = KS / 2; m > 0; m >>= 1) {
                const bool up = (sub & m) != 0;
#pragma unroll
                for (int j = 0; j < m; j++) {
                    const float give = up ? o[j] : o[j + m], keep = up ? o[j + m] : o[j];
                    o[j] = keep + __shfl_xor_sync(MG_FULL_MASK, give, m);
                }
            }
            if (g + sub < T && v < D) out[(size_t)(t0 + g + sub) * nh + h * D + v] = o[0];
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < KPT; i++) {
        const int d = 4 * (sub + i / 4 * KS) + i % 4;
        if (d < D && v < D) M.S[((size_t)h * D + d) * D + v] = S[i];
    }
}

template <int KPT, int KS>
cudaError_t scan_for(const Wkv& wk, const float* proj, int ldp, const float* decay, int pos0, int n, float* out, cudaStream_t s) {
    using G = Scan<KPT, KS>;
    constexpr int per = 3 * G::rows + (G::cols + 3) / 4 * 4;
    int tile = 32;
    while (tile > KS && 2 * (size_t)tile * per * sizeof(float) > 100 * 1024) tile /= 2;
    const size_t smem = 2 * (size_t)tile * per * sizeof(float);
    static cudaError_t attr = cudaFuncSetAttribute((const void*)wkv_scan_kernel<KPT, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (attr != cudaSuccess) return attr;
    wkv_scan_kernel<KPT, KS><<<dim3(wk.heads, (wk.dim + G::cols - 1) / G::cols), kScanThreads, smem, s>>>(wk, proj, ldp, decay, pos0, n, tile, out);
    return cudaGetLastError();
}

}  // namespace

size_t wkv_step_smem(const Wkv& wk) { return ((size_t)pad_to(5 * wk.dim, 4) + pad_to(wk.rank, 8) + (size_t)kStepThreads / 32 * wk.dim) * sizeof(float); }

cudaError_t launch_wkv_step(const WkvStep& a, bool pdl, cudaStream_t s) {
    return launch_pdl(wkv_step_kernel, a.wk.heads, kStepThreads, wkv_step_smem(a.wk), pdl, s, a);
}

cudaError_t launch_wkv_mix(const float* h, const float* prev, const float* const mu[5], int pos0, int n, int width, void* act, int ld_act,
                           long long act_stride, bool f32, cudaStream_t s) {
    if (f32) wkv_mix_kernel<float><<<n, 256, 0, s>>>(h, prev, mu[0], mu[1], mu[2], mu[3], mu[4], pos0, width, (float*)act, ld_act, act_stride);
    else wkv_mix_kernel<__nv_bfloat16><<<n, 256, 0, s>>>(h, prev, mu[0], mu[1], mu[2], mu[3], mu[4], pos0, width, (__nv_bfloat16*)act, ld_act, act_stride);
    return cudaGetLastError();
}

bool wkv_rows_fits(const Wkv& wk) { return wk.dim <= 512; }

cudaError_t launch_wkv_rows(const Wkv& wk, const float* proj, int ldp, const float* decay, int pos0, int n, float* out, cudaStream_t s) {
    if (wk.dim <= 32) return scan_for<8, 4>(wk, proj, ldp, decay, pos0, n, out, s);
    if (wk.dim <= 64) return scan_for<8, 8>(wk, proj, ldp, decay, pos0, n, out, s);
    if (wk.dim <= 128) return scan_for<8, 16>(wk, proj, ldp, decay, pos0, n, out, s);
    if (wk.dim <= 256) return scan_for<16, 16>(wk, proj, ldp, decay, pos0, n, out, s);
    if (wk.dim <= 512) return scan_for<32, 16>(wk, proj, ldp, decay, pos0, n, out, s);
    return cudaErrorInvalidValue;
}

}  // namespace mg
