// Latent attention over a portion of a prompt, on the tensor cores.
//
// Keys and values of every position so far are formed from the cached latents by two products; the value
// product has the value matrix on the left, so that values come out transposed, as the second product of
// attention wants them.  Then a CTA owns 128 queries of one head and walks the keys in tiles of 64: scores
// S = Q K^T into one of two TMEM buffers, softmax on four warps (a thread owns a query row), weights as bf16
// into shared memory, O += P V in TMEM.  A score's operands are the head's unrotated part and the rotated part
// that all heads share, side by side in shared memory, so nothing is concatenated in memory.  O is rescaled
// only when a row's maximum has grown by more than 2^8 since its reference was set; until then the larger
// weights are exact in bf16's range and the sum in fp32.
#include <algorithm>

#include "gemm_tc.h"
#include "layered_ops.cuh"
#include "umma.cuh"

namespace mg {

namespace {

constexpr int kThreads = 192;       // TMA warp, MMA warp, 4 softmax warps
constexpr int kKeys = 64;           // keys per tile
constexpr float kGrow = 8.0f;       // log2 of the growth that a row's reference tolerates

struct FlashArgs {
    CUtensorMap qn, qr, kn, kr, v;
    int pos0, n;                    // queries 0 .. n - 1 at positions pos0 + row
    int dim_s, rot_s, vdim;
    int cn, cr;                     // 64-column steps of the unrotated and the rotated part
    int vp;                         // vdim padded to 16
    int stages;
    int tmem_cols;
    __nv_bfloat16* out;             // [n][ld_out], head h at columns h * vdim
    int ld_out;
    int* status;
};

__host__ __device__ inline int k_bytes(int chunks) { return chunks * kKeys * 128; }
__host__ __device__ inline int v_bytes(int vp) { return vp * 128; }
__host__ __device__ inline int q_bytes(int chunks) { return chunks * 128 * 128; }
constexpr int kPBytes = 128 * 128;

__device__ __forceinline__ float exp2_fast(float t) {
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(t));
    return e;
}

__global__ void __launch_bounds__(kThreads, 2) latent_flash_kernel(const __grid_constant__ FlashArgs a) {
    extern __shared__ uint8_t raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>(((uintptr_t)raw + 1023) & ~(uintptr_t)1023);
    const int chunks = a.cn + a.cr, NS = a.stages;
    // every part is a multiple of 1024 bytes (vp * 128 is rounded up)
    const int kb = k_bytes(chunks), vb = pad_to(v_bytes(a.vp), 1024);
    uint8_t* Q = base;
    uint8_t* P = Q + q_bytes(chunks);
    uint8_t* Ks = P + kPBytes;
    uint8_t* Vs = Ks + NS * kb;
    uint64_t* bars = reinterpret_cast<uint64_t*>(Vs + NS * vb);
    uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = bars + 3, *v_full = bars + 5, *v_empty = bars + 7, *s_full = bars + 9,
             *s_empty = bars + 11, *p_full = bars + 13;
    uint32_t* tmem_base = reinterpret_cast<uint32_t*>(bars + 14);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y, row0 = (gridDim.x - 1 - blockIdx.x) * 128;        // the longest rows first
    const int last = min(a.n - 1, row0 + 127);
    const int len = a.pos0 + a.n;
    const int tiles = (a.pos0 + last) / kKeys + 1;

    if (threadIdx.x == 0) {
        for (int i = 0; i < 13; i++) bar_init(bars + i, i >= 11 ? 4 : 1);
        bar_init(p_full, 4);
        bar_init_fence();
        tma_prefetch_map(&a.qn); tma_prefetch_map(&a.qr); tma_prefetch_map(&a.kn); tma_prefetch_map(&a.kr); tma_prefetch_map(&a.v);
    }
    if (warp == 1) tmem_alloc(tmem_base, a.tmem_cols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_base, S0 = tmem, O = tmem + 2 * kKeys;

    if (warp == 0) {
        if (lane == 0) {
            bar_expect(q_full, q_bytes(chunks));
            for (int c = 0; c < a.cn; c++) tma_load_3d(Q + c * 128 * 128, &a.qn, c * 64, h, row0, q_full);
            for (int c = 0; c < a.cr; c++) tma_load_3d(Q + (a.cn + c) * 128 * 128, &a.qr, c * 64, h, row0, q_full);
            int ki = 0, vi = 0;
            for (int j = 0; j < tiles; j++) {
                const int s = j % NS, use = j / NS;
                if (use > 0 && !bar_wait(k_empty + s, (use - 1) & 1, a.status)) break;
                bar_expect(k_full + s, kb);
                uint8_t* st = Ks + s * kb;
                for (int c = 0; c < a.cn; c++) tma_load_3d(st + c * kKeys * 128, &a.kn, c * 64, h, j * kKeys, k_full + s);
                for (int c = 0; c < a.cr; c++) tma_load_3d(st + (a.cn + c) * kKeys * 128, &a.kr, c * 64, j * kKeys, 0, k_full + s);
                ki = j + 1;
                if (use > 0 && !bar_wait(v_empty + s, (use - 1) & 1, a.status)) break;
                bar_expect(v_full + s, v_bytes(a.vp));
                tma_load_3d(Vs + s * vb, &a.v, j * kKeys, 0, h, v_full + s);
                vi = j + 1;
            }
            // no copy may be in flight when the CTA leaves
            bar_wait(q_full, 0, a.status);
            for (int i = max(0, ki - NS); i < ki; i++) bar_wait(k_full + i % NS, (i / NS) & 1, a.status);
            for (int i = max(0, vi - NS); i < vi; i++) bar_wait(v_full + i % NS, (i / NS) & 1, a.status);
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            auto scores = [&](int j) {
                const int s = j % NS, b = j & 1;
                if (!bar_wait(k_full + s, (j / NS) & 1, a.status)) return false;
                if (j >= 2 && !bar_wait(s_empty + b, (j / 2 - 1) & 1, a.status)) return false;
                tc_fence_after();
                for (int c = 0; c < chunks; c++) {
                    const uint64_t da = tile_desc(Q + c * 128 * 128), db = tile_desc(Ks + s * kb + c * kKeys * 128);
#pragma unroll
                    for (int k = 0; k < 4; k++) mma_bf16(S0 + b * kKeys, da + 2 * k, db + 2 * k, mma_desc(kKeys), c > 0 || k > 0);
                }
                mma_commit(k_empty + s);
                mma_commit(s_full + b);
                return true;
            };
            bool ok = bar_wait(q_full, 0, a.status) && scores(0);
            for (int j = 0; j < tiles && ok; j++) {
                if (j + 1 < tiles && !(ok = scores(j + 1))) break;
                const int s = j % NS;
                ok = bar_wait(p_full, j & 1, a.status) && bar_wait(v_full + s, (j / NS) & 1, a.status);
                if (!ok) break;
                tc_fence_after();
                const uint64_t da = tile_desc(P), db = tile_desc(Vs + s * vb);
                const uint32_t desc = mma_desc(a.vp);
#pragma unroll
                for (int k = 0; k < 4; k++) mma_bf16(O, da + 2 * k, db + 2 * k, desc, j > 0 || k > 0);
                mma_commit(v_empty + s);
            }
        }
        __syncwarp();
    } else {
        const int quarter = warp & 3, r = quarter * 32 + lane;
        const uint32_t mine = (uint32_t)(quarter * 32) << 16;
        const int row = row0 + r, pos = min(a.pos0 + row, len - 1);
        float ref = -INFINITY, sum = 0.f;
        bool ok = true;
        for (int j = 0; j < tiles; j++) {
            const int b = j & 1;
            ok = __all_sync(0xffffffffu, bar_wait(s_full + b, (j / 2) & 1, a.status));
            if (!ok) break;
            tc_fence_after();
            float s[2][32];
            tmem_load32(S0 + mine + b * kKeys, s[0]);
            tmem_load32(S0 + mine + b * kKeys + 32, s[1]);
            tc_fence_before();
            __syncwarp();
            if (lane == 0) bar_arrive(s_empty + b);
            const int seen = pos - j * kKeys + 1;       // keys of this tile that the row sees
            if (__any_sync(0xffffffffu, seen < kKeys)) {
#pragma unroll
                for (int i = 0; i < kKeys; i++)
                    if (i >= seen) s[i >> 5][i & 31] = -INFINITY;
            }
            float mx = s[0][0];
#pragma unroll
            for (int i = 1; i < kKeys; i++) mx = fmaxf(mx, s[i >> 5][i & 31]);
            // P and O are free once the last tile's product is done
            if (j > 0) {
                ok = __all_sync(0xffffffffu, bar_wait(v_empty + (j - 1) % NS, ((j - 1) / NS) & 1, a.status));
                if (!ok) break;
                tc_fence_after();
            }
            if (j == 0) {
                ref = mx;                               // key 0 is in this tile and seen by every row
            } else if (__any_sync(0xffffffffu, mx > ref + kGrow)) {
                const float up = fmaxf(mx, ref), f = exp2_fast(ref - up);
                ref = up;
                sum *= f;
                for (int c = 0; c < a.vp; c += 32) {
                    float o[32];
                    tmem_load32(O + mine + c, o);
#pragma unroll
                    for (int i = 0; i < 32; i++) o[i] *= f;
                    tmem_store32(O + mine + c, o);
                }
            }
#pragma unroll
            for (int c = 0; c < 8; c++) {
                uint32_t w[4];
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const int k = c * 8 + i * 2;
                    const float x = exp2_fast(s[k >> 5][k & 31] - ref), y = exp2_fast(s[(k + 1) >> 5][(k + 1) & 31] - ref);
                    sum += x + y;
                    const __nv_bfloat162 p = __floats2bfloat162_rn(x, y);
                    w[i] = *reinterpret_cast<const uint32_t*>(&p);
                }
                *reinterpret_cast<uint4*>(P + r * 128 + ((c ^ (r & 7)) << 4)) = make_uint4(w[0], w[1], w[2], w[3]);
            }
            async_proxy_fence();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) bar_arrive(p_full);
        }
        if (ok) ok = __all_sync(0xffffffffu, bar_wait(v_empty + (tiles - 1) % NS, ((tiles - 1) / NS) & 1, a.status));
        if (ok) {
            tc_fence_after();
            const float inv = 1.0f / sum;
            __nv_bfloat16* out = a.out + (size_t)row * a.ld_out + h * a.vdim;
            const bool pair = ((a.vdim | a.ld_out) & 1) == 0;
            for (int c = 0; c < a.vdim; c += 32) {
                float o[32];
                tmem_load32(O + mine + c, o);
                if (row < a.n) {
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        if (pair) {
                            if (c + i < a.vdim) *reinterpret_cast<__nv_bfloat162*>(out + c + i) = __floats2bfloat162_rn(o[i] * inv, o[i + 1] * inv);
                        } else {
                            if (c + i < a.vdim) out[c + i] = __float2bfloat16_rn(o[i] * inv);
                            if (c + i + 1 < a.vdim) out[c + i + 1] = __float2bfloat16_rn(o[i + 1] * inv);
                        }
                    }
                }
                __syncwarp();
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    tc_fence_after();
    if (warp == 1) tmem_free(tmem, a.tmem_cols);
}

struct Geometry {
    int cn, cr, vp, stages, tmem_cols;
    size_t smem;
};

// Two stages where two CTAs still share an SM, or where they do not in any case.
Geometry geometry(const LatentAttn& at) {
    Geometry g{};
    g.cn = (at.dim_s + 63) / 64; g.cr = (at.rot_s + 63) / 64; g.vp = pad_to(at.vdim, 16);
    // columns are read and rescaled in steps of 32
    const int cols = 2 * kKeys + pad_to(at.vdim, 32);
    g.tmem_cols = cols <= 256 ? 256 : 512;
    auto bytes = [&](int st) {
        return (size_t)q_bytes(g.cn + g.cr) + kPBytes + (size_t)st * (k_bytes(g.cn + g.cr) + pad_to(v_bytes(g.vp), 1024)) + 1024 + 256;
    };
    const size_t two = 113 * 1024, one = 226 * 1024;
    g.stages = g.tmem_cols == 256 && bytes(2) <= two ? 2 : g.tmem_cols == 256 && bytes(1) <= two ? 1 : bytes(2) <= one ? 2 : 1;
    g.smem = bytes(g.stages);
    return g;
}

}  // namespace

bool latent_attn_tc_fits(const LatentAttn& at) {
    return at.vdim <= 256 && at.dim_s <= 256 && at.rot_s <= 256 && geometry(at).smem <= 226 * 1024;
}

cudaError_t launch_latent_attn_tc(const LatentAttn& at, const void* qh, int pos0, int n, void* keys, void* vt, int ldv, void* out, int ld_out,
                                  int* status, int* launches, cudaStream_t s) {
    const int len = pos0 + n;
    GemmTC g{};
    g.batch = 1; g.b_group = 1; g.causal_pos0 = -1; g.k = at.ld; g.mode = GEMM_BF16; g.status = status;
    // keys[len][heads * dim_s] = c U_k^T
    g.m = len; g.n = at.heads * at.dim_s; g.bn = g.n > 64 ? 128 : 64; g.out = keys; g.ldc = g.n;
    if (!make_tile_map(&g.a, at.cache, at.rank_s, at.max_seq, 1, at.row(), (long long)at.max_seq * at.row(), 128) ||
        !make_tile_map(&g.b, at.uk, at.ld, g.n, 1, at.ld, (long long)g.n * at.ld, g.bn))
        return cudaErrorInvalidValue;
    cudaError_t c = launch_gemm_tc(g, s);
    if (c != cudaSuccess) return c;
    // vt[heads * vdim][len] = U_v c^T
    g.m = at.heads * at.vdim; g.n = len; g.bn = len > 64 ? 128 : 64; g.out = vt; g.ldc = ldv;
    if (!make_tile_map(&g.a, at.uv, at.ld, g.m, 1, at.ld, (long long)g.m * at.ld, 128) ||
        !make_tile_map(&g.b, at.cache, at.rank_s, at.max_seq, 1, at.row(), (long long)at.max_seq * at.row(), g.bn))
        return cudaErrorInvalidValue;
    if ((c = launch_gemm_tc(g, s)) != cudaSuccess) return c;

    const Geometry geo = geometry(at);
    FlashArgs f{};
    f.pos0 = pos0; f.n = n; f.dim_s = at.dim_s; f.rot_s = at.rot_s; f.vdim = at.vdim; f.cn = geo.cn; f.cr = geo.cr; f.vp = geo.vp;
    f.stages = geo.stages; f.tmem_cols = geo.tmem_cols; f.out = (__nv_bfloat16*)out; f.ld_out = ld_out; f.status = status;
    const int qr = at.qrow();
    const __nv_bfloat16* q = (const __nv_bfloat16*)qh;
    // rows past the portion (queries) and past the last position (keys and values) read as zero
    if (!make_head_map(&f.qn, q, at.dim_s, at.heads, n, qr, (long long)at.heads * qr, 128) ||
        !make_head_map(&f.qr, q + at.dim_s, at.rot_s, at.heads, n, qr, (long long)at.heads * qr, 128) ||
        !make_head_map(&f.kn, keys, at.dim_s, at.heads, len, at.dim_s, (long long)at.heads * at.dim_s, kKeys) ||
        !make_tile_map(&f.kr, (const __nv_bfloat16*)at.cache + at.rank_s, at.rot_s, len, 1, at.row(), (long long)at.max_seq * at.row(), kKeys) ||
        !make_tile_map(&f.v, vt, len, at.vdim, at.heads, ldv, (long long)at.vdim * ldv, geo.vp))
        return cudaErrorInvalidValue;
    static cudaError_t attr = cudaFuncSetAttribute((const void*)latent_flash_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (attr != cudaSuccess) return attr;
    latent_flash_kernel<<<dim3((n + 127) / 128, at.heads), kThreads, geo.smem, s>>>(f);
    *launches += 3;
    return cudaGetLastError();
}

}  // namespace mg
