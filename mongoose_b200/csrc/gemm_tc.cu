// out = A B^T for bf16 A [m][k] and B [n][k], fp32 accumulation: one 128 x BN tile per CTA.  Warp 0 streams both
// operands with TMA into a ring of 64-column stages, one thread of warp 1 issues tcgen05.mma into TMEM,
// warps 2-5 read the accumulator back and store it row by row through shared memory.  Two CTAs share an
// SM, so one's epilogue runs under the other's products; where there are fewer tiles than SMs, a CTA has the
// SM to itself and a ring deep enough to cover the latency of its copies.
#include "gemm_tc.h"
#include "layered_ops.cuh"
#include "umma.cuh"

namespace mg {

namespace {

constexpr int kThreads = 192;
constexpr int kShallow = 3;
constexpr int deep(int bn) { return bn == 64 ? 8 : 6; }

// gelu for results that are rounded to bf16: tanh from one fast exponential
__device__ __forceinline__ float gelu_tanh_fast(float z) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return z - z * __fdividef(1.0f, 1.0f + __expf(2.0f * u));
}

__device__ __forceinline__ float silu_fast(float z) { return z * __fdividef(1.0f, 1.0f + __expf(-z)); }

template <int BN, int kStages>
struct Smem {
    static constexpr int a_bytes = 128 * 128, b_bytes = BN * 128, stage = a_bytes + b_bytes;
    static constexpr int bytes = kStages * stage + 1024 + 256;      // + alignment + barriers
};

template <int BN, int kStages>
__global__ void __launch_bounds__(kThreads, kStages == kShallow ? 2 : 1) gemm_tc_kernel(const __grid_constant__ GemmTC g) {
    extern __shared__ uint8_t raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>(((uintptr_t)raw + 1023) & ~(uintptr_t)1023);
    uint64_t* full = reinterpret_cast<uint64_t*>(base + kStages * Smem<BN, kStages>::stage);
    uint64_t* empty = full + kStages;
    uint64_t* done = empty + kStages;
    uint32_t* tmem_base = reinterpret_cast<uint32_t*>(done + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool dual = BN == 128 && g.mode == GEMM_SILU_BF16;
    const int col0 = blockIdx.x * (dual ? 64 : BN), row0 = blockIdx.y * 128, z = blockIdx.z;
    int zb = z / g.b_group;
    if (g.group) {
        zb = g.group[blockIdx.y];
        if (zb < 0) return;
    }
    int kt = (g.k + 63) / 64;
    if (g.causal_pos0 >= 0) kt = min(kt, (g.causal_pos0 + min(row0 + 128, g.m) + 63) / 64);

    if (threadIdx.x == 0) {
        for (int i = 0; i < kStages; i++) { bar_init(full + i, 1); bar_init(empty + i, 1); }
        bar_init(done, 1);
        bar_init_fence();
        tma_prefetch_map(&g.a);
        tma_prefetch_map(&g.b);
        if (dual) tma_prefetch_map(&g.b2);
    }
    if (warp == 1) tmem_alloc(tmem_base, BN);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t acc = *tmem_base;

    if (warp == 0) {
        if (lane == 0) {
            int issued = 0;
            for (int i = 0; i < kt; i++) {
                const int s = i % kStages, use = i / kStages;
                if (use > 0 && !bar_wait(empty + s, (use - 1) & 1, g.status)) break;
                bar_expect(full + s, Smem<BN, kStages>::stage);
                uint8_t* st = base + s * Smem<BN, kStages>::stage;
                tma_load_3d(st, &g.a, i * 64, row0, z, full + s);
                tma_load_3d(st + Smem<BN, kStages>::a_bytes, &g.b, (g.b_steps ? i % g.b_steps : i) * 64, col0, zb, full + s);
                if (dual) tma_load_3d(st + Smem<BN, kStages>::a_bytes + 64 * 128, &g.b2, i * 64, col0, zb, full + s);
                issued = i + 1;
            }
            // no copy may be in flight when the CTA leaves
            for (int i = max(0, issued - kStages); i < issued; i++) bar_wait(full + i % kStages, (i / kStages) & 1, g.status);
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            bool ok = true;
            for (int i = 0; i < kt && ok; i++) {
                const int s = i % kStages;
                ok = bar_wait(full + s, (i / kStages) & 1, g.status);
                if (!ok) break;
                tc_fence_after();
                const uint64_t da = tile_desc(base + s * Smem<BN, kStages>::stage), db = tile_desc(base + s * Smem<BN, kStages>::stage + Smem<BN, kStages>::a_bytes);
#pragma unroll
                for (int k = 0; k < 4; k++) mma_bf16(acc, da + 2 * k, db + 2 * k, mma_desc(BN), i > 0 || k > 0);
                mma_commit(empty + s);
            }
            mma_commit(done);
        }
        __syncwarp();
    } else {
        const bool ok = __all_sync(0xffffffffu, bar_wait(done, 0, g.status));
        tc_fence_after();
        const int quarter = warp & 3;
        float* tile = reinterpret_cast<float*>(base) + quarter * 32 * 33;     // every stage has been consumed
        if (ok) {
#pragma unroll 1
            for (int c = 0; c < (dual ? 64 : BN); c += 32) {
                float v[32];
                tmem_load32(acc + ((uint32_t)(quarter * 32) << 16) + c, v);
                if (dual) {
                    float u[32];
                    tmem_load32(acc + ((uint32_t)(quarter * 32) << 16) + 64 + c, u);
#pragma unroll
                    for (int i = 0; i < 32; i++) v[i] = silu_fast(v[i]) * u[i];
                }
#pragma unroll
                for (int i = 0; i < 32; i++) tile[lane * 33 + i] = v[i];
                __syncwarp();
                if (g.mode == GEMM_F32 || g.mode == GEMM_DECAY_F32) {
                    const int col = col0 + c + lane;
                    float* out = static_cast<float*>(g.out) + z * g.batch_c + col;
                    const float bias = g.mode == GEMM_DECAY_F32 && col < g.n ? g.bias[col] : 0.f;
#pragma unroll 8
                    for (int r = 0; r < 32; r++) {
                        const int row = row0 + quarter * 32 + r;
                        float x = tile[r * 33 + lane];
                        if (g.mode == GEMM_DECAY_F32) x = expf(-expf(x + bias));
                        if (row < g.m && col < g.n) out[row * g.ldc] = x;
                    }
                } else {                            // two columns per lane, two rows at a time
                    const int col = col0 + c + 2 * (lane & 15);
                    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(g.out) + z * g.batch_c + col;
                    const bool pair = (reinterpret_cast<uintptr_t>(out) & 3) == 0 && (g.ldc & 1) == 0 && col + 1 < g.n;
#pragma unroll 4
                    for (int r = lane >> 4; r < 32; r += 2) {
                        const int row = row0 + quarter * 32 + r;
                        float x = tile[r * 33 + 2 * (lane & 15)], y = tile[r * 33 + 2 * (lane & 15) + 1];
                        if (g.mode == GEMM_GELU_BF16) { x = gelu_tanh_fast(x); y = gelu_tanh_fast(y); }
                        if (row >= g.m) break;
                        if (pair) {
                            *reinterpret_cast<__nv_bfloat162*>(out + row * g.ldc) = __floats2bfloat162_rn(x, y);
                        } else {
                            if (col < g.n) out[row * g.ldc] = __float2bfloat16_rn(x);
                            if (col + 1 < g.n) out[row * g.ldc + 1] = __float2bfloat16_rn(y);
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
    if (warp == 1) tmem_free(acc, BN);
}

typedef CUresult (*encode_fn_t)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

encode_fn_t encode_fn() {
    static encode_fn_t fn = [] {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) p = nullptr;
        return (encode_fn_t)p;
    }();
    return fn;
}

bool encode(CUtensorMap* map, const void* base, const cuuint64_t dims[3], const cuuint64_t strides[2], const cuuint32_t box[3]) {
    const cuuint32_t ones[3] = {1, 1, 1};
    encode_fn_t fn = encode_fn();
    return fn && fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, ones,
                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                    CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int BN, int kStages>
cudaError_t run(const GemmTC& g, dim3 grid, cudaStream_t s) {
    constexpr int bytes = Smem<BN, kStages>::bytes;
    static cudaError_t attr = cudaFuncSetAttribute((const void*)gemm_tc_kernel<BN, kStages>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (attr != cudaSuccess) return attr;
    gemm_tc_kernel<BN, kStages><<<grid, kThreads, bytes, s>>>(g);
    return cudaGetLastError();
}

int sm_count() {
    static const int n = [] {
        int dev = 0, v = 0;
        return cudaGetDevice(&dev) == cudaSuccess && cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev) == cudaSuccess ? v : 0;
    }();
    return n;
}

template <int BN>
cudaError_t run(const GemmTC& g, cudaStream_t s) {
    const int cols = g.mode == GEMM_SILU_BF16 ? 64 : BN;
    const dim3 grid((g.n + cols - 1) / cols, (g.m + 127) / 128, g.batch);
    const bool few = (long long)grid.x * grid.y * grid.z <= sm_count() && g.k > kShallow * 64;
    return few ? run<BN, deep(BN)>(g, grid, s) : run<BN, kShallow>(g, grid, s);
}

}  // namespace

bool make_tile_map(CUtensorMap* map, const void* base, int k, int rows, int batch, long long row_stride, long long batch_stride, int box_rows) {
    const cuuint64_t dims[3] = {(cuuint64_t)k, (cuuint64_t)rows, (cuuint64_t)batch};
    const cuuint64_t strides[2] = {(cuuint64_t)row_stride * 2, (cuuint64_t)batch_stride * 2};
    const cuuint32_t box[3] = {64, (cuuint32_t)box_rows, 1};
    return encode(map, base, dims, strides, box);
}

bool make_head_map(CUtensorMap* map, const void* base, int k, int batch, int rows, long long batch_stride, long long row_stride, int box_rows) {
    const cuuint64_t dims[3] = {(cuuint64_t)k, (cuuint64_t)batch, (cuuint64_t)rows};
    const cuuint64_t strides[2] = {(cuuint64_t)batch_stride * 2, (cuuint64_t)row_stride * 2};
    const cuuint32_t box[3] = {64, 1, (cuuint32_t)box_rows};
    return encode(map, base, dims, strides, box);
}

cudaError_t launch_gemm_tc(const GemmTC& g, cudaStream_t s) {
    if (g.bn == 64 && g.mode != GEMM_SILU_BF16) return run<64>(g, s);
    if (g.bn == 128) return run<128>(g, s);
    return cudaErrorInvalidValue;
}

}  // namespace mg
