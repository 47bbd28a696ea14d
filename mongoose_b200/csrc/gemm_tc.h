// bf16 matrix products on the tensor cores (gemm_tc.cu).
#pragma once

#include <cuda.h>
#include <cuda_runtime.h>

namespace mg {

enum : int { GEMM_F32 = 0, GEMM_BF16 = 1, GEMM_GELU_BF16 = 2,
             GEMM_SILU_BF16 = 3,        // two matrices on one input: silu(A B^T) * (A B2^T)
             GEMM_DECAY_F32 = 4 };      // exp(-exp(A B^T + bias))

// A 3-D bf16 tensor [batch][rows][k] seen by TMA in boxes of box_rows x 64 columns (128-byte swizzle); the
// part of a box outside the tensor reads as zero.  Strides in elements, multiples of 8.
bool make_tile_map(CUtensorMap* map, const void* base, int k, int rows, int batch, long long row_stride, long long batch_stride,
                   int box_rows);
// The same with the batch index in the middle: box of 64 columns x 1 x box_rows over [rows][batch][k].
bool make_head_map(CUtensorMap* map, const void* base, int k, int batch, int rows, long long batch_stride, long long row_stride,
                   int box_rows);

struct GemmTC {
    CUtensorMap a, b;       // a: boxes of 128 rows; b: boxes of `bn` rows (64 for GEMM_SILU_BF16)
    CUtensorMap b2;         // GEMM_SILU_BF16: the second matrix, boxes of 64 rows
    int bn;                 // 64 or 128; GEMM_SILU_BF16: 128, n in steps of 64
    int m, n, k;            // out[m][n], k columns (rounded up to 64 inside)
    int b_steps;            // > 0: b has this many steps of 64 columns, a several times as many: a = [a1 a2 ..] multiplies [b b ..]
    const float* bias;      // [n], GEMM_DECAY_F32
    int batch, b_group;     // batch z multiplies a's batch z with b's batch z / b_group
    const int* group;       // not NULL: row tile y multiplies b's batch group[y]; -1: the tile is empty
    int causal_pos0;        // >= 0: row r only needs columns k <= causal_pos0 + r (the rest of a is zero)
    void* out;              // fp32 or bf16
    long long ldc, batch_c; // elements
    int mode;
    int* status;
};
cudaError_t launch_gemm_tc(const GemmTC& g, cudaStream_t s);

}  // namespace mg
