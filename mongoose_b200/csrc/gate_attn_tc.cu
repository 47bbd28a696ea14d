// Sigmoid attention with mixed heads over a portion of a prompt, on the tensor cores.
//
// Mixing couples every head at every (query, key) pair, so a CTA owns a tile of 128 queries x BN keys for
// ALL heads: each head's scores land in their own TMEM columns (heads x BN <= 512), then a thread reads
// one query row's scores of all heads for four keys at a time, forms the sigmoids in fp32, and the mixed
// weights are written as bf16.  Up to 8 heads are mixed in registers (packed fma.rn.f32x2).  With more
// heads the mixing is a small product per key, mix[h][query] = sum_g T[h][g] w[g][query]: T is bf16 as
// stored, and the fp32 weights go in as two bf16 parts, high and low (16 bits of mantissa together), in
// two rounds of mma.sync over the same accumulator; their operand layout is what the TMEM rows give
// after one pass through shared memory.  The product with the raw keys is a
// batched gemm_tc over heads (its causal bound skips the zero part), against keys transposed once per
// call.  Queries go in blocks, so that the weights of a block stay within the workspace.
#include <algorithm>

#include "gemm_tc.h"
#include "layered_ops.cuh"
#include "umma.cuh"

namespace mg {

namespace {

constexpr int kThreads = 320;       // TMA warp, MMA warp, 8 epilogue warps

struct ScoreArgs {
    CUtensorMap q, k;               // [rows][heads][dim_s] in boxes of 128 rows; [max_seq][kv][dim_s] in boxes of BN rows
    GateAttn at;
    int row0, rows, pos0;           // queries [row0, row0 + rows) of the portion, at positions pos0 + row
    int ldp;                        // columns of a weight row (a multiple of 64)
    long long head_stride;          // elements between heads of the weights
    __nv_bfloat16* w;               // [heads][.][ldp]
    int* status;
};

template <int HP>
struct Geo {
    static constexpr bool tensor_mix = HP >= 16;
    static constexpr int bn = HP <= 8 ? 32 : 16;
    static constexpr int cols = HP * bn < 32 ? 32 : HP * bn;
    static constexpr int per_sm = cols <= 256 ? 2 : 1;
    static constexpr int stages = HP == 32 ? 8 : HP == 16 ? 5 : 4;
    static constexpr int stage = 128 * 128 + bn * 128;
    static constexpr int ring = stages * stage;
    // the epilogue's operand rows take the ring's place: per warp 4 keys x 32 queries x {high, low}
    static constexpr int point = HP * 2 + 16;               // bytes of a row of bf16 weights, padded against conflicts
    static constexpr int part = 4 * 32 * point;
    static constexpr int mix_bytes = tensor_mix ? 8 * 2 * part : 0;
    static constexpr int body = ring > mix_bytes ? ring : mix_bytes;
    static constexpr int talk_bytes = tensor_mix ? 0 : 8 * HP * HP;    // mixing pairs {t, t}
    static constexpr int bytes = body + 1024 + 256 + talk_bytes + (2 * HP + bn * HP) * 4;
};

// 1 / (1 + 2^t)
__device__ __forceinline__ float sigmoid_of_exp2(float t) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(t));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
    return r;
}
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t bf16_pair(float a, float b) {
    const __nv_bfloat162 p = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&p);
}

template <int HP>
__global__ void __launch_bounds__(kThreads, Geo<HP>::per_sm) gate_scores_kernel(const __grid_constant__ ScoreArgs a) {
    using G = Geo<HP>;
    constexpr int BN = G::bn, kStages = G::stages;
    const GateAttn& A = a.at;
    const int tile_row = blockIdx.y * 128, j0 = blockIdx.x * BN;
    const int tile_rows = min(128, a.rows - tile_row);
    // the product reads whole steps of 64 columns up to the last query of the row tile
    if (j0 >= pad_to(a.pos0 + a.row0 + tile_row + tile_rows, 64)) return;

    extern __shared__ uint8_t raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>(((uintptr_t)raw + 1023) & ~(uintptr_t)1023);
    uint64_t* full = reinterpret_cast<uint64_t*>(base + G::body);
    uint64_t* empty = full + kStages;
    uint64_t* done = empty + kStages;
    uint32_t* tmem_base = reinterpret_cast<uint32_t*>(done + 1);
    ulonglong2* talk = reinterpret_cast<ulonglong2*>(base + G::body + 256);     // [h][g / 2]: {t, t} of two g
    float2* line = reinterpret_cast<float2*>(base + G::body + 256 + G::talk_bytes);  // per head: slope, -bias, in units of log2 e
    float* kr = reinterpret_cast<float*>(line + HP);                            // [head][key]: -1 / rms of the key, likewise
    static_assert((2 * kStages + 1) * 8 + 4 <= 256, "barriers fit their place");

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int H = A.heads, group = H / A.kv_heads;
    const int kb = (A.dim_s + 63) / 64, steps = H * kb;

    if (threadIdx.x == 0) {
        for (int i = 0; i < kStages; i++) { bar_init(full + i, 1); bar_init(empty + i, 1); }
        bar_init(done, 1);
        bar_init_fence();
        tma_prefetch_map(&a.q);
        tma_prefetch_map(&a.k);
    }
    if (warp == 1) tmem_alloc(tmem_base, G::cols);
    constexpr float kLog2e = 1.4426950408889634f;
    if constexpr (!G::tensor_mix) {
        for (int i = threadIdx.x; i < HP * HP / 2; i += kThreads) {
            const int h = i / (HP / 2), g = 2 * (i % (HP / 2));
            const float t0 = h < H && g < H ? A.talk[h * H + g] : 0.f, t1 = h < H && g + 1 < H ? A.talk[h * H + g + 1] : 0.f;
            talk[i] = make_ulonglong2(pack2(t0, t0), pack2(t1, t1));
        }
    }
    for (int i = threadIdx.x; i < HP; i += kThreads)
        line[i] = i < H ? make_float2(A.slopes[i] * kLog2e, -A.head_bias[i] * kLog2e) : make_float2(0.f, 0.f);
    const int len = a.pos0 + a.row0 + a.rows;       // keys the block's queries can see
    for (int i = threadIdx.x; i < BN * HP; i += kThreads) {
        const int p = i % BN, h = i / BN;
        kr[i] = h < H && j0 + p < len ? -kLog2e * A.cache_r[(size_t)(j0 + p) * A.kv_heads + h / group] : 0.f;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t acc = *tmem_base;

    if (warp == 0) {
        if (lane == 0) {
            int issued = 0;
            for (int i = 0; i < steps; i++) {
                const int s = i % kStages, use = i / kStages, h = i / kb, x = (i - h * kb) * 64;
                if (use > 0 && !bar_wait(empty + s, (use - 1) & 1, a.status)) break;
                bar_expect(full + s, G::stage);
                uint8_t* st = base + s * G::stage;
                tma_load_3d(st, &a.q, x, h, a.row0 + tile_row, full + s);
                tma_load_3d(st + 128 * 128, &a.k, x, h / group, j0, full + s);
                issued = i + 1;
            }
            for (int i = max(0, issued - kStages); i < issued; i++) bar_wait(full + i % kStages, (i / kStages) & 1, a.status);
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            for (int i = 0; i < steps; i++) {
                const int s = i % kStages, h = i / kb;
                if (!bar_wait(full + s, (i / kStages) & 1, a.status)) break;
                tc_fence_after();
                const uint64_t da = tile_desc(base + s * G::stage), db = tile_desc(base + s * G::stage + 128 * 128);
#pragma unroll
                for (int k = 0; k < 4; k++) mma_bf16(acc + h * BN, da + 2 * k, db + 2 * k, mma_desc(BN), i > h * kb || k > 0);
                mma_commit(empty + s);
            }
            mma_commit(done);
        }
        __syncwarp();
    } else {
        // mixing matrix as MMA operands: rows h, columns g
        constexpr int MT = HP >= 16 ? HP / 16 : 1;
        uint32_t ta[MT][MT][4];
        if constexpr (G::tensor_mix) {
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int k = 0; k < MT; k++)
#pragma unroll
                    for (int r = 0; r < 4; r++) {
                        const int h = m * 16 + (lane >> 2) + (r & 1) * 8, g = k * 16 + (lane & 3) * 2 + (r >> 1) * 8;
                        ta[m][k][r] = bf16_pair(h < H && g < H ? A.talk[h * H + g] : 0.f, h < H && g + 1 < H ? A.talk[h * H + g + 1] : 0.f);
                    }
        }
        const bool ok = __all_sync(0xffffffffu, bar_wait(done, 0, a.status));
        tc_fence_after();
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        const int row = tile_row + quarter * 32 + lane;
        const int pos = a.pos0 + a.row0 + row;
        uint8_t* mine = base + (warp - 2) * 2 * G::part;
        if (ok) {
#pragma unroll 1
            for (int c = half * (BN / 2); c < (half + 1) * (BN / 2); c += 4) {
                constexpr int GB = HP < 8 ? HP : 8;         // heads per round of loads
                unsigned long long w[G::tensor_mix ? 1 : HP][2];
                const float dist = (float)(pos - (j0 + c));
#pragma unroll
                for (int g0 = 0; g0 < HP; g0 += GB) {
                    uint32_t s[GB][4];
                    float v[GB][4];
#pragma unroll
                    for (int g = 0; g < GB; g++)
                        if (g0 + g < H) tmem_load4_async(acc + ((uint32_t)(quarter * 32) << 16) + (g0 + g) * BN + c, s[g]);
                    tmem_wait_load();
#pragma unroll
                    for (int g = 0; g < GB; g++) {
                        const float2 ln = line[g0 + g];
                        const float4 k4 = *reinterpret_cast<const float4*>(kr + (g0 + g) * BN + c);
                        const float kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            const float t = fmaf(__uint_as_float(s[g][i]), kk[i], fmaf(ln.x, dist - (float)i, ln.y));
                            v[g][i] = g0 + g < H && dist >= (float)i ? sigmoid_of_exp2(t) : 0.f;
                        }
                    }
                    if constexpr (G::tensor_mix) {
                        // eight heads are 16 bytes of a point's row, as bf16 and what bf16 leaves over
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            uint32_t hi4[4], lo4[4];
#pragma unroll
                            for (int g = 0; g < GB; g += 2) {
                                const uint32_t p = bf16_pair(v[g][i], v[g + 1][i]);
                                hi4[g / 2] = p;
                                lo4[g / 2] = bf16_pair(v[g][i] - __uint_as_float(p << 16), v[g + 1][i] - __uint_as_float(p & 0xffff0000u));
                            }
                            uint8_t* row_at = mine + (i * 32 + lane) * G::point + g0 * 2;
                            *reinterpret_cast<uint4*>(row_at) = make_uint4(hi4[0], hi4[1], hi4[2], hi4[3]);
                            *reinterpret_cast<uint4*>(row_at + G::part) = make_uint4(lo4[0], lo4[1], lo4[2], lo4[3]);
                        }
                    } else {
#pragma unroll
                        for (int g = 0; g < GB; g++) {
                            w[g0 + g][0] = pack2(v[g][0], v[g][1]);
                            w[g0 + g][1] = pack2(v[g][2], v[g][3]);
                        }
                    }
                }
                if constexpr (G::tensor_mix) {
                    __syncwarp();
#pragma unroll 1
                    for (int nt = 0; nt < 4; nt++) {            // eight queries at a time
                        float o[MT][4][4] = {};                 // [h tile][key][accumulator]
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            uint32_t bh[4], bl[4];
                            if constexpr (MT == 2) {
                                const uint32_t at = smem_addr(mine) + (i * 32 + nt * 8 + (lane & 7)) * G::point + (lane >> 3) * 16;
                                ldmatrix4(bh, at);
                                ldmatrix4(bl, at + G::part);
                            } else {                            // high columns 0-7, 8-15, then low
                                uint32_t b4[4];
                                ldmatrix4(b4, smem_addr(mine) + (i * 32 + nt * 8 + (lane & 7)) * G::point + ((lane >> 3) & 1) * 16 + (lane >> 4) * G::part);
                                bh[0] = b4[0]; bh[1] = b4[1]; bl[0] = b4[2]; bl[1] = b4[3];
                            }
#pragma unroll
                            for (int m = 0; m < MT; m++)
#pragma unroll
                                for (int k = 0; k < MT; k++) {
                                    mma_16816(o[m][i], ta[m][k], bh[2 * k], bh[2 * k + 1]);
                                    mma_16816(o[m][i], ta[m][k], bl[2 * k], bl[2 * k + 1]);
                                }
                        }
#pragma unroll
                        for (int m = 0; m < MT; m++)
#pragma unroll
                            for (int r = 0; r < 4; r++) {
                                const int h = m * 16 + (lane >> 2) + (r >> 1) * 8;
                                const int q = tile_row + quarter * 32 + nt * 8 + (lane & 3) * 2 + (r & 1);
                                if (h < H && q < a.rows)
                                    *reinterpret_cast<uint2*>(a.w + h * a.head_stride + (long long)q * a.ldp + j0 + c) =
                                        make_uint2(bf16_pair(o[m][0][r], o[m][1][r]), bf16_pair(o[m][2][r], o[m][3][r]));
                            }
                    }
                    __syncwarp();                               // the rows are free again
                } else {
                    __nv_bfloat16* out = a.w + (long long)row * a.ldp + j0 + c;
#pragma unroll 2
                    for (int h = 0; h < H; h++) {
                        unsigned long long m0 = 0ull, m1 = 0ull;
#pragma unroll
                        for (int g = 0; g < HP; g += 2) {
                            const ulonglong2 t = talk[h * (HP / 2) + g / 2];
                            m0 = fma2(t.x, w[g][0], m0);
                            m1 = fma2(t.x, w[g][1], m1);
                            m0 = fma2(t.y, w[g + 1][0], m0);
                            m1 = fma2(t.y, w[g + 1][1], m1);
                        }
                        if (row < a.rows)
                            *reinterpret_cast<uint2*>(out + h * a.head_stride) = make_uint2(bf16_pair(lo(m0), hi(m0)), bf16_pair(lo(m1), hi(m1)));
                    }
                }
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    tc_fence_after();
    if (warp == 1) tmem_free(acc, G::cols);
}

// cache [len][kv][dim_s] -> vt [kv][dim][ldv], zero from len to ldv
__global__ void __launch_bounds__(256) key_transpose_kernel(const __nv_bfloat16* cache, int kv_heads, int dim, int dim_s, int len, int ldv,
                                                            __nv_bfloat16* vt) {
    __shared__ __nv_bfloat16 t[32][34];
    const int p0 = blockIdx.x * 32, d0 = blockIdx.y * 32, c = blockIdx.z, x = threadIdx.x & 31, y = threadIdx.x >> 5;
    for (int i = y; i < 32; i += 8)
        t[i][x] = p0 + i < len && d0 + x < dim ? cache[((size_t)(p0 + i) * kv_heads + c) * dim_s + d0 + x] : __float2bfloat16_rn(0.f);
    __syncthreads();
    for (int i = y; i < 32; i += 8)
        if (d0 + i < dim && p0 + x < ldv) vt[((size_t)c * dim + d0 + i) * ldv + p0 + x] = t[x][i];
}

template <int HP>
cudaError_t scores(const ScoreArgs& a, cudaStream_t s) {
    using G = Geo<HP>;
    static cudaError_t attr = cudaFuncSetAttribute((const void*)gate_scores_kernel<HP>, cudaFuncAttributeMaxDynamicSharedMemorySize, G::bytes);
    if (attr != cudaSuccess) return attr;
    gate_scores_kernel<HP><<<dim3(pad_to(a.pos0 + a.row0 + a.rows, 64) / G::bn, (a.rows + 127) / 128), kThreads, G::bytes, s>>>(a);
    return cudaGetLastError();
}

}  // namespace

bool gate_attn_tc_fits(const GateAttn& at) { return at.heads <= 32; }

int gate_attn_tc_rows(const GateAttn& at, int max_seq, int max_rows, size_t budget) {
    const size_t per = (size_t)at.heads * pad_to(max_seq, 64) * 2;
    int rows = (int)std::min<size_t>(budget / per, (size_t)pad_to(max_rows, 128)) / 128 * 128;
    return rows < 128 ? 128 : rows;
}

cudaError_t launch_gate_attn_tc(const GateAttn& at, const void* qh, int pos0, int n, int max_rows, void* weights, int block_rows, void* vt,
                                void* out, int ld_out, int* status, int* launches, cudaStream_t s) {
    const int len = pos0 + n, ldv = pad_to(len, 64);
    key_transpose_kernel<<<dim3(ldv / 32, (at.dim + 31) / 32, at.kv_heads), 256, 0, s>>>((const __nv_bfloat16*)at.cache, at.kv_heads, at.dim,
                                                                                       at.dim_s, len, ldv, (__nv_bfloat16*)vt);
    *launches += 1;
    const int hp = at.heads <= 4 ? 4 : at.heads <= 8 ? 8 : at.heads <= 16 ? 16 : 32;
    ScoreArgs a{};
    a.at = at; a.pos0 = pos0; a.w = (__nv_bfloat16*)weights; a.status = status;
    if (!make_head_map(&a.q, qh, at.dim_s, at.heads, max_rows, at.dim_s, (long long)at.heads * at.dim_s, 128) ||
        !make_head_map(&a.k, at.cache, at.dim_s, at.kv_heads, at.max_seq, at.dim_s, (long long)at.kv_heads * at.dim_s, hp <= 8 ? 32 : 16))
        return cudaErrorInvalidValue;
    GemmTC g{};
    g.bn = at.dim > 64 ? 128 : 64;
    g.n = at.dim; g.batch = at.heads; g.b_group = at.heads / at.kv_heads; g.ldc = ld_out; g.batch_c = at.dim; g.mode = GEMM_BF16; g.status = status;
    if (!make_tile_map(&g.b, vt, ldv, at.dim, at.kv_heads, ldv, (long long)at.dim * ldv, g.bn)) return cudaErrorInvalidValue;
    for (int q0 = 0; q0 < n; q0 += block_rows) {
        const int rows = std::min(block_rows, n - q0);
        a.row0 = q0; a.rows = rows; a.ldp = pad_to(pos0 + q0 + rows, 64); a.head_stride = (long long)block_rows * a.ldp;
        cudaError_t c = hp == 4 ? scores<4>(a, s) : hp == 8 ? scores<8>(a, s) : hp == 16 ? scores<16>(a, s) : scores<32>(a, s);
        if (c != cudaSuccess) return c;
        if (!make_tile_map(&g.a, weights, a.ldp, block_rows, at.heads, a.ldp, a.head_stride, 128)) return cudaErrorInvalidValue;
        g.m = rows; g.k = a.ldp; g.causal_pos0 = pos0 + q0;
        g.out = (__nv_bfloat16*)out + (size_t)q0 * ld_out;
        if ((c = launch_gemm_tc(g, s)) != cudaSuccess) return c;
        *launches += 2;
    }
    return cudaSuccess;
}

}  // namespace mg
