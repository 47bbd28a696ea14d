// Launchers of the kernels that serve layer-described models (mg_create_layered).  One entry per
// mechanism, every size and constant an argument; the kernels themselves are in layered_decode.cu (one
// token), layered_prefill.cu (portions of a prompt), gate_attn_tc.cu and gemm_tc.cu (bf16 tensor cores).
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "decode_kernels.cuh"

namespace mg {

constexpr int kMemChunk = 64;       // tokens per chunk of the matrix memory's chunked form

__host__ __device__ inline int pad_to(int n, int m) { return (n + m - 1) / m * m; }

// Attention whose weights are sigmoids (no normalisation over keys), whose heads' weights are mixed by a
// matrix, and whose values are the raw keys: one cache row per position serves scores and values.
struct GateAttn {
    int heads, kv_heads, dim, dim_s;    // dim_s: dim padded to a multiple of 8 (stored rows)
    float scale;
    float temp_coef;                    // query temperature 1 + coef * ln(floor((p + 1) / every) + 1)
    int temp_every;
    const float* q_norm;                // [dim]
    const float* k_norm;                // [dim]
    const float* talk;                  // [heads][heads]
    const float* head_bias;             // [heads]
    const float* slopes;                // [heads]
    float eps;
    void* cache;                        // [max_seq][kv_heads][dim_s] raw keys, bf16 or fp32
    float* cache_r;                     // [max_seq][kv_heads] 1 / rms of the stored key
    int max_seq;
};

// Matrix memory (one [dim][vdim] state per head) with exponential input and forget gates.
struct MatMem {
    int heads, dim, vdim;
    float cap, eps;
    const float *i_bias, *f_bias;       // [heads]
    const float* norm;                  // [heads * vdim]
    float* S;                           // [heads][dim][vdim]
    float* nrm;                         // [2][heads][dim]: the slot of parity p holds the state before position p
    float* m;                           // [2][heads]
};

// Columns of a projection row (the mixers' input matrices stacked into one).
struct ProjCols {
    int q, k, mq, mk, mv, mg, mi, mf, total;
};

// ---- one token (layered_decode.cu) -------------------------------------------------------------
phase_fn_t layered_phase(int epi, int R);
typedef void (*phase_pair_fn_t)(const PhaseArgs, const PhaseArgs, int);
phase_pair_fn_t layered_phase_pair(int R);

// Largest dynamic shared memory the phase kernels may be launched with.
cudaError_t layered_phase_smem(size_t bytes);

struct MixerStep {
    GateAttn at;
    MatMem mem;
    ProjCols c;
    const float* proj;      // one projection row
    const StepState* st;
    int n_mem;              // CTAs of the memory part (0: no such branch)
    int vslices;            // value slices of 32 columns per head
    int splits;             // CTAs of the attention part
    int tile;               // keys per shared-memory tile
    float* part;            // [splits][heads * dim_s]
    float* mem_o;           // [heads * vdim] raw outputs
    float* attn_out;        // [heads * dim]
    float* mem_y;           // [heads * vdim] normed and gated
};
// Shared memory of the step (0: the sizes do not fit), and its tile.
size_t mixer_step_smem(const GateAttn& at, const MatMem& mem, bool f32_cache, int* tile);
cudaError_t launch_mixer_step(const MixerStep& a, bool f32_cache, bool pdl, cudaStream_t s);
cudaError_t launch_mixer_join(const MixerStep& a, bool pdl, cudaStream_t s);

struct ResolveArgs {            // the pending residual update of a step that ends between layers
    PhaseArgs p;                // its prologue fields
    float* out;
};
cudaError_t launch_resolve(const ResolveArgs& a, bool pdl, cudaStream_t s);

// ---- portions of a prompt (layered_prefill.cu) -----------------------------------------------------
// `act` buffers hold bf16 or fp32 (f32 = true) rows padded to a multiple of 64 with zeros.
cudaError_t launch_embed_rows(const WeightView& embed, int ld_embed, const float* pos_tab, const int* tokens, int pos0, int n,
                              int width, float* x, void* act, int ld_act, bool f32, cudaStream_t s);
// out[n][ldc] = A[n][K] W[rows][K]^T, fp32 accumulation on the CUDA cores (32-bit mode)
cudaError_t launch_gemm_f32(const float* A, int lda, const uint8_t* W, int ldw, float* out, int ldc, int n, int rows, int K,
                            bool gelu, cudaStream_t s);
// queries: normed, times temperature, score scale and key-norm weight; keys: raw rows into the cache
cudaError_t launch_qk_rows(const GateAttn& at, const float* proj, int ldp, int q_col, int k_col, int pos0, int n, void* qh,
                           bool f32, cudaStream_t s);
cudaError_t launch_gate_attn_rows(const GateAttn& at, const void* qh, int pos0, int n, void* out, int ld_out, bool f32,
                                  cudaStream_t s);
size_t gate_attn_rows_smem(const GateAttn& at, bool f32, int* tile);
// The same on the tensor cores (bf16 only, gate_attn_tc.cu): `weights` holds block_rows rows of every head
// (gate_attn_tc_rows of them fit `budget`), `vt` the keys transposed; qh has max_rows rows.
bool gate_attn_tc_fits(const GateAttn& at);
int gate_attn_tc_rows(const GateAttn& at, int max_seq, int max_rows, size_t budget);
cudaError_t launch_gate_attn_tc(const GateAttn& at, const void* qh, int pos0, int n, int max_rows, void* weights, int block_rows, void* vt,
                                void* out, int ld_out, int* status, int* launches, cudaStream_t s);
// x += norm(z) or x += norm(half the sum of two normed branches); act = x
cudaError_t launch_post_rows(float* x, const float* z0, const float* z1, const float* w0, const float* w1, const float* post_w,
                             float eps, int n, int width, void* act, int ld_act, bool f32, cudaStream_t s);
// act[r] = norm(x[rows[r]]), weight around zero
cudaError_t launch_last_norm_rows(const float* x, const int* rows, const float* w, float eps, int n, int width, void* act,
                                  int ld_act, bool f32, cudaStream_t s);

struct MemRows {                // workspace of the chunked memory for up to n tokens
    double* b;                  // [heads][n] log-forget sum inside the chunk
    float* ig;                  // [heads][n] log input gate
    float* mm;                  // [heads][n] running maximum
    float* g;                   // [heads][chunks] decay of the state over a chunk
    float* m0;                  // [heads] the maximum before the portion
    float* U;                   // [chunks][heads][dim][vdim]
    float* nU;                  // [chunks][heads][dim]
    float* o;                   // [n][heads * vdim]
};
cudaError_t launch_mem_rows(const MatMem& mem, const ProjCols& c, const float* proj, int ldp, int pos0, int n, const MemRows& w,
                            void* act, int ld_act, bool f32, cudaStream_t s);

}  // namespace mg
