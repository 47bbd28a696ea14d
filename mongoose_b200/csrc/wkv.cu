// Linear recurrence with a decay per key channel, S <- diag(w) S + k v^T, o = (S_before + diag(u) k v^T)^T r, in
// fp32.  The columns of a head's state (value channels) never meet, so a prompt runs the recurrence itself,
// token by token, with the columns of all heads spread over the GPU: no chunk's cumulative decay is ever formed,
// and decays of any strength are exact.
#include "layered_ops.cuh"

namespace mg {

namespace {

constexpr int kStepThreads = 256;
constexpr int kStepRows = 8;        // rows of the state a warp holds at a time, two columns per lane

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
    // weights first: they wait for nothing
    const int sub = threadIdx.x & 3, d_of = threadIdx.x >> 2;
    constexpr int kAhead = 2;
    uint4 w2[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; i++) {
        const int c = (sub + 4 * i) * 8;
        w2[i] = d_of < D && c < rk ? __ldg(reinterpret_cast<const uint4*>(M.w2 + (size_t)(c0 + d_of) * M.ld2 + c)) : make_uint4(0u, 0u, 0u, 0u);
    }
    const float w0 = d_of < D ? M.w0[c0 + d_of] : 0.f;
    for (int i = threadIdx.x; i < D; i += kStepThreads) u[i] = M.u[c0 + i];
    pdl_launch_dependents();
    pdl_wait();
    const bool fresh = a.st->pos == 0;
    float* S = M.S + (size_t)blockIdx.x * D * D;
    float s0[kStepRows][2];
    auto load_rows = [&](int k0, int col) {
#pragma unroll
        for (int i = 0; i < kStepRows; i++) {
            const int d = k0 + wid + i * nw;
            s0[i][0] = !fresh && col < D && d < D ? S[(size_t)d * D + col] : 0.f;
            s0[i][1] = !fresh && col + 32 < D && d < D ? S[(size_t)d * D + col + 32] : 0.f;
        }
    };
    load_rows(0, lane);
    for (int i = threadIdx.x; i < D; i += kStepThreads) { r[i] = a.row[c0 + i]; k[i] = a.row[n + c0 + i]; v[i] = a.row[2 * n + c0 + i]; }
    for (int i = threadIdx.x; i < rk; i += kStepThreads) inner[i] = i < M.rank ? tanhf(a.row[4 * (size_t)n + i]) : 0.f;
    __syncthreads();
    // decays: four threads per channel
    for (int d0 = 0; d0 < D; d0 += kStepThreads / 4) {
        const int d = d0 + d_of;
        float z = 0.f;
        if (d < D) {
            const __nv_bfloat16* wp = M.w2 + (size_t)(c0 + d) * M.ld2;
#pragma unroll
            for (int i = 0; i < kAhead; i++) {
                const int c = (sub + 4 * i) * 8;
                if (c < rk) {
                    if (d0 > 0) w2[i] = __ldg(reinterpret_cast<const uint4*>(wp + c));
                    const float4 x[2] = {*reinterpret_cast<const float4*>(inner + c), *reinterpret_cast<const float4*>(inner + c + 4)};
                    z += Chunk<FMT_BF16>::dot(w2[i], x);
                }
            }
            for (int c = (sub + 4 * kAhead) * 8; c < rk; c += 32) {
                const float4 x[2] = {*reinterpret_cast<const float4*>(inner + c), *reinterpret_cast<const float4*>(inner + c + 4)};
                z += Chunk<FMT_BF16>::dot(__ldg(reinterpret_cast<const uint4*>(wp + c)), x);
            }
        }
        z += __shfl_xor_sync(MG_FULL_MASK, z, 1);
        z += __shfl_xor_sync(MG_FULL_MASK, z, 2);
        if (sub == 0 && d < D) w[d] = expf(-expf(z + (d0 > 0 ? M.w0[c0 + d] : w0)));
    }
    __syncthreads();
    for (int v0 = 0; v0 < D; v0 += 64) {
        const int col = v0 + lane;
        const float va = col < D ? v[col] : 0.f, vb = col + 32 < D ? v[col + 32] : 0.f;
        float oa = 0.f, ob = 0.f;
        for (int k0 = 0; k0 < D; k0 += kStepRows * nw) {
            if (v0 > 0 || k0 > 0) load_rows(k0, col);
#pragma unroll
            for (int i = 0; i < kStepRows; i++) {
                const int d = k0 + wid + i * nw;
                if (d < D) {
                    const float ka = k[d] * va, kb = k[d] * vb;
                    oa = fmaf(fmaf(u[d], ka, s0[i][0]), r[d], oa);
                    ob = fmaf(fmaf(u[d], kb, s0[i][1]), r[d], ob);
                    if (col < D) S[(size_t)d * D + col] = fmaf(w[d], s0[i][0], ka);
                    if (col + 32 < D) S[(size_t)d * D + col + 32] = fmaf(w[d], s0[i][1], kb);
                }
            }
        }
        if (col < D) part[wid * D + col] = oa;
        if (col + 32 < D) part[wid * D + col + 32] = ob;
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

// V values per thread and step (4 where rows are whole quads).
template <typename AT, int V>
__global__ void __launch_bounds__(256) wkv_mix_kernel(const float* h, const float* prev, const float* m0, const float* m1, const float* m2,
                                                      const float* m3, const float* m4, int pos0, int width, AT* act, int ld_act,
                                                      long long stride) {
    const int t = blockIdx.x;
    const float* cur = h + (size_t)t * width;
    const float* before = t > 0 ? cur - width : prev + (size_t)(pos0 & 1) * width;
    const bool none = t == 0 && pos0 == 0;
    const float* mu[5] = {m0, m1, m2, m3, m4};
    for (int i = threadIdx.x * V; i < width; i += 256 * V) {
        float x[V], d[V];
        load_values<V>(cur + i, x);
        if (none) {
#pragma unroll
            for (int q = 0; q < V; q++) d[q] = 0.f;
        } else {
            load_values<V>(before + i, d);
        }
#pragma unroll
        for (int j = 0; j < 5; j++) {
            float m[V];
            load_values<V>(mu[j] + i, m);
#pragma unroll
            for (int q = 0; q < V; q++) m[q] = fmaf(d[q] - x[q], m[q], x[q]);
            store_values<V>(m, act + j * stride + (size_t)t * ld_act + i);
        }
    }
}

// act[t] = [high, low]: tanh of the decay's inner projection, the sum of `slices` slabs, as two bf16 parts (16 bits of
// mantissa together), each padded to ld / 2, so that a product of bf16 operands keeps it.
__global__ void __launch_bounds__(256) wkv_inner_kernel(const float* inner, int ldp, int slices, int rank, int n, __nv_bfloat16* act, int ld) {
    const int i = blockIdx.x * 256 + threadIdx.x, t = i / rank, c = i - t * rank;
    if (t >= n) return;
    float v = 0.f;
    for (int s = 0; s < slices; s++) v += inner[((size_t)s * n + t) * ldp + c];
    v = tanhf(v);
    const __nv_bfloat16 high = __float2bfloat16_rn(v);
    act[(size_t)t * ld + c] = high;
    act[(size_t)t * ld + ld / 2 + c] = __float2bfloat16_rn(v - __bfloat162float(high));
}

// ---- prompts ----
constexpr int kScanWarps = 8, kScanThreads = kScanWarps * 32;
constexpr int kScanTile = 32;       // tokens of a tile in shared memory
constexpr int kScanStages = 3;

constexpr int kScanCols = 2;        // value channels per warp
constexpr int kScanGroup = 16;      // tokens whose sums are reduced together

// A lane's N key channels as pairs: neighbouring ones, quads 32 lanes apart where N > 4.
template <int N>
__device__ __forceinline__ void lds_pairs(const float* p, int lane, unsigned long long (&o)[N / 2]) {
    if constexpr (N == 2) {
        o[0] = *reinterpret_cast<const unsigned long long*>(p + 2 * lane);
    } else {
#pragma unroll
        for (int q = 0; q < N / 4; q++) {
            const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p + 4 * (lane + 32 * q));
            o[2 * q] = v.x; o[2 * q + 1] = v.y;
        }
    }
}
template <int KPT>
__device__ __forceinline__ int scan_channel(int lane, int i) { return KPT == 2 ? 2 * lane + i : 4 * (lane + i / 4 * 32) + i % 4; }

// A warp owns kScanCols columns of a head's state (value channels), its lanes KPT key channels each, two at a time in
// packed arithmetic.  Tokens come through shared memory in tiles: r, k, w padded to 32 KPT channels, then the
// CTA's value channels.  A sum over key channels is one over lanes; those of several tokens are reduced at once
// by halving exchanges, which spread tokens and columns over the lanes.
template <int KPT>
struct Scan {
    static constexpr int cols = kScanCols * kScanWarps;     // value channels per CTA
    static constexpr int rows = 32 * KPT, per = 3 * rows + cols, P = KPT / 2;
    static constexpr size_t smem(int tile) { return kScanStages * (size_t)tile * per * sizeof(float); }
    static constexpr int tile = smem(kScanTile) <= 200 * 1024 ? kScanTile : kScanTile / 2;
    static_assert(tile % kScanGroup == 0 && smem(tile) <= 227 * 1024, "a tile holds whole groups");
};

template <int KPT>
__global__ void __launch_bounds__(kScanThreads) wkv_scan_kernel(const Wkv M, const float* proj, int ldp, const float* decay, int pos0, int n,
                                                                float* out) {
    extern __shared__ __align__(16) float smem[];
    using G = Scan<KPT>;
    constexpr int rows = G::rows, per = G::per, P = G::P, tile = G::tile, NO = kScanGroup * kScanCols;
    const int D = M.dim, nh = M.heads * D, h = blockIdx.x, v0 = blockIdx.y * G::cols;
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, vw = v0 + wid * kScanCols;
    const int cols = min(G::cols, D - v0);
    // the padding is zero and stays so
    for (int i = threadIdx.x; i < kScanStages * tile * per; i += kScanThreads) smem[i] = 0.f;
    __syncthreads();
    // a thread copies piece `c` of every `step`-th token from `first` on; quads where rows are whole quads
    const int wide = ((D | ldp) & 3) == 0 ? 4 : 1;
    auto pieces = [&](int count, int& first, int& c, int& step) {
        if (count > kScanThreads) count = kScanThreads;             // the rest in further rounds over c
        step = kScanThreads / count;
        first = threadIdx.x / count;
        c = (threadIdx.x - first * count) * wide;
        if (first >= step) first = tile;
    };
    int f1, c1, s1, f2, c2, s2;
    pieces(D / wide, f1, c1, s1);
    pieces(cols / wide, f2, c2, s2);
    const float* row0 = proj + h * D;
    const float* dec0 = decay + h * D;
    auto load = [&](int i) {
        const int t0 = i * tile, T = min(tile, n - t0);
        float* dst = smem + (size_t)(i % kScanStages) * tile * per;
        auto copy = [&](float* to, const float* from) {
            if (wide == 4) cp_async16(to, from);
            else cp_async4(to, from);
        };
        for (int t = f1; t < T; t += s1)
            for (int c = c1; c < D; c += kScanThreads * wide) {
                const float* row = row0 + (size_t)(t0 + t) * ldp + c;
                copy(dst + t * per + c, row);
                copy(dst + t * per + rows + c, row + nh);
                copy(dst + t * per + 2 * rows + c, dec0 + (size_t)(t0 + t) * nh + c);
            }
        for (int t = f2; t < T; t += s2) copy(dst + t * per + 3 * rows + c2, row0 + (size_t)(t0 + t) * ldp + 2 * (size_t)nh + v0 + c2);
        cp_async_commit();
    };
    for (int i = 0; i < kScanStages - 1; i++) load(i);
    unsigned long long S[kScanCols][P], u[P];
#pragma unroll
    for (int i = 0; i < P; i++) {
        const int d = scan_channel<KPT>(lane, 2 * i);       // and the next
        u[i] = pack2(d < D ? M.u[h * D + d] : 0.f, d + 1 < D ? M.u[h * D + d + 1] : 0.f);
#pragma unroll
        for (int c = 0; c < kScanCols; c++) {
            const float* s = M.S + ((size_t)h * D + d) * D + vw + c;
            const bool in = vw + c < D && pos0 > 0;
            S[c][i] = pack2(in && d < D ? s[0] : 0.f, in && d + 1 < D ? s[D] : 0.f);
        }
    }
    struct Token {
        unsigned long long r[P], k[P], w[P];
        float v[kScanCols];
    };
    auto fetch = [&](const float* p, Token& x) {
        lds_pairs<KPT>(p, lane, x.r);
        lds_pairs<KPT>(p + rows, lane, x.k);
        lds_pairs<KPT>(p + 2 * rows, lane, x.w);
        const float* v = p + 3 * rows + wid * kScanCols;
#pragma unroll
        for (int c = 0; c < kScanCols; c += 2) {
            const float2 t = *reinterpret_cast<const float2*>(v + c);
            x.v[c] = t.x; x.v[c + 1] = t.y;
        }
    };
    auto step = [&](const Token& x, float* o) {
#pragma unroll
        for (int c = 0; c < kScanCols; c++) {
            const unsigned long long v = pack2(x.v[c], x.v[c]);
            unsigned long long sum = 0ull;
#pragma unroll
            for (int i = 0; i < P; i++) {
                const unsigned long long kv = mul2(x.k[i], v);
                const unsigned long long t = fma2(u[i], kv, S[c][i]);
                sum = i ? fma2(t, x.r[i], sum) : mul2(t, x.r[i]);
                S[c][i] = fma2(x.w[i], S[c][i], kv);
            }
            o[c] = lo(sum) + hi(sum);
        }
    };
    const int tiles = (n + tile - 1) / tile;
    for (int it = 0; it < tiles; it++) {
        const int t0 = it * tile, T = min(tile, n - t0);
        load(it + kScanStages - 1);
        cp_async_wait<kScanStages - 1>();
        __syncthreads();
        const float* base = smem + (size_t)(it % kScanStages) * tile * per;
        for (int g = 0; g < T; g += kScanGroup) {
            float o[NO];
            if (g + kScanGroup <= T) {
                constexpr int AHEAD = KPT == 2 ? 4 : 1;     // tokens held before they are needed
                Token x[AHEAD];
#pragma unroll
                for (int j = 0; j < AHEAD; j++) fetch(base + (g + j) * per, x[j]);
#pragma unroll
                for (int j = 0; j < kScanGroup; j++) {
                    const Token now = x[j % AHEAD];
                    if (j + AHEAD < kScanGroup) fetch(base + (g + j + AHEAD) * per, x[j % AHEAD]);
                    step(now, o + j * kScanCols);
                }
            } else {
#pragma unroll
                for (int j = 0; j < kScanGroup; j++)
                    if (g + j < T) {
                        Token x;
                        fetch(base + (g + j) * per, x);
                        step(x, o + j * kScanCols);
                    }
            }
            constexpr int L = 32 / NO;              // lanes that end with the same sum
#pragma unroll
            for (int m = NO / 2; m > 0; m >>= 1) {
                const bool up = (lane & (L * m)) != 0;
#pragma unroll
                for (int j = 0; j < m; j++) {
                    const float give = up ? o[j] : o[j + m], keep = up ? o[j + m] : o[j];
                    o[j] = keep + __shfl_xor_sync(MG_FULL_MASK, give, L * m);
                }
            }
#pragma unroll
            for (int m = L / 2; m > 0; m >>= 1) o[0] += __shfl_xor_sync(MG_FULL_MASK, o[0], m);
            const int t = g + lane / L / kScanCols, v = vw + lane / L % kScanCols;
            if (lane % L == 0 && t < T && v < D) out[(size_t)(t0 + t) * nh + h * D + v] = o[0];
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < P; i++) {
        const int d = scan_channel<KPT>(lane, 2 * i);
#pragma unroll
        for (int c = 0; c < kScanCols; c++) {
            float* s = M.S + ((size_t)h * D + d) * D + vw + c;
            if (vw + c < D && d < D) s[0] = lo(S[c][i]);
            if (vw + c < D && d + 1 < D) s[D] = hi(S[c][i]);
        }
    }
}

template <int KPT>
cudaError_t scan_for(const Wkv& wk, const float* proj, int ldp, const float* decay, int pos0, int n, float* out, cudaStream_t s) {
    using G = Scan<KPT>;
    constexpr size_t smem = G::smem(G::tile);
    static cudaError_t attr = cudaFuncSetAttribute((const void*)wkv_scan_kernel<KPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (attr != cudaSuccess) return attr;
    wkv_scan_kernel<KPT><<<dim3(wk.heads, (wk.dim + G::cols - 1) / G::cols), kScanThreads, smem, s>>>(wk, proj, ldp, decay, pos0, n, out);
    return cudaGetLastError();
}

template <typename AT>
cudaError_t mix_for(const float* h, const float* prev, const float* const mu[5], int pos0, int n, int width, AT* act, int ld_act, long long stride,
                    cudaStream_t s) {
    if (width % 4 == 0) wkv_mix_kernel<AT, 4><<<n, 256, 0, s>>>(h, prev, mu[0], mu[1], mu[2], mu[3], mu[4], pos0, width, act, ld_act, stride);
    else wkv_mix_kernel<AT, 1><<<n, 256, 0, s>>>(h, prev, mu[0], mu[1], mu[2], mu[3], mu[4], pos0, width, act, ld_act, stride);
    return cudaGetLastError();
}

}  // namespace

size_t wkv_step_smem(const Wkv& wk) { return ((size_t)pad_to(5 * wk.dim, 4) + pad_to(wk.rank, 8) + (size_t)kStepThreads / 32 * wk.dim) * sizeof(float); }

cudaError_t launch_wkv_step(const WkvStep& a, bool pdl, cudaStream_t s) {
    return launch_pdl(wkv_step_kernel, a.wk.heads, kStepThreads, wkv_step_smem(a.wk), pdl, s, a);
}

cudaError_t launch_wkv_mix(const float* h, const float* prev, const float* const mu[5], int pos0, int n, int width, void* act, int ld_act,
                           long long act_stride, bool f32, cudaStream_t s) {
    return f32 ? mix_for(h, prev, mu, pos0, n, width, (float*)act, ld_act, act_stride, s)
               : mix_for(h, prev, mu, pos0, n, width, (__nv_bfloat16*)act, ld_act, act_stride, s);
}

cudaError_t launch_wkv_inner(const float* inner, int ldp, int slices, int rank, int n, void* act, int ld, cudaStream_t s) {
    wkv_inner_kernel<<<(n * rank + 255) / 256, 256, 0, s>>>(inner, ldp, slices, rank, n, (__nv_bfloat16*)act, ld);
    return cudaGetLastError();
}

bool wkv_rows_fits(const Wkv& wk) { return wk.dim <= 256; }

cudaError_t launch_wkv_rows(const Wkv& wk, const float* proj, int ldp, const float* decay, int pos0, int n, float* out, cudaStream_t s) {
    if (wk.dim <= 64) return scan_for<2>(wk, proj, ldp, decay, pos0, n, out, s);
    if (wk.dim <= 128) return scan_for<4>(wk, proj, ldp, decay, pos0, n, out, s);
    if (wk.dim <= 256) return scan_for<8>(wk, proj, ldp, decay, pos0, n, out, s);
    return cudaErrorInvalidValue;
}

}  // namespace mg
