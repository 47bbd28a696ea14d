// Launchers of the kernels that serve layer-described models (mg_create_layered).  One entry per
// mechanism, every size and constant an argument; the kernels themselves are in layered_decode.cu (one
// token), layered_prefill.cu (portions of a prompt), latent_attn.cu, wkv.cu and moe.cu (both), gate_attn_tc.cu,
// latent_attn_tc.cu and gemm_tc.cu (bf16 tensor cores).
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

// Softmax attention over a cached latent c (rank values) and a rotated key part shared by the heads.  A head's
// unrotated key is U_k c and its value U_v c, so q . (U_k c) = (U_k^T q) . c: one token, and 32-bit mode, score
// the cached rows themselves with U_k^T q and apply U_v to the weighted sum of rows; bf16 prompts form keys and
// values.  Parts of a row are padded to multiples of 8 with zeros.
struct LatentAttn {
    int heads, dim, rot, vdim, rank, q_rank;
    int dim_s, rot_s, rank_s;
    float scale, eps;
    const float *q_norm, *c_norm;       // [q_rank], [rank]
    const float *cos_tab, *sin_tab;     // [max_seq][rot / 2]
    const __nv_bfloat16 *uk, *uv;       // [heads * dim_s][ld], [heads * vdim][ld]
    int ld;                             // rank padded to a multiple of 64
    void* cache;                        // [max_seq][rank_s + rot_s] bf16 or fp32
    int max_seq;
    __host__ __device__ int row() const { return rank_s + rot_s; }      // a cached row
    __host__ __device__ int qrow() const { return dim_s + rot_s; }      // a head's query
};

// Linear recurrence with a decay per key channel.
struct Wkv {
    int heads, dim, rank;               // rank of the decay's projection
    float eps;
    const __nv_bfloat16* w2;            // [heads * dim][ld2]
    int ld2;
    const float *w0, *u, *norm;         // [heads * dim]
    float* S;                           // [heads][dim key channels][dim value channels]
};

// Mixture of experts: `top` of `experts` gated feed-forwards of inner width ff, and a shared one.
struct Moe {
    int experts, top, ff, shared_ff, width;
    int ffs, shared_ffs;                // padded to multiples of 64
    const float* bias;                  // [experts]
    const uint8_t *gate, *up, *down;    // bf16 [experts * ff][ldw], [experts * ff][ldw], [experts * width][ffs]
    const uint8_t* shared_down;         // [width][shared_ffs]
    int ldw;
    // a router row: logits, the shared expert's gate, then (one token) its gate and up projections
    __host__ __device__ int sg_col() const { return experts; }
};
constexpr int kMaxExperts = 1024, kMaxTop = 64;

// ---- one token (layered_decode.cu) -------------------------------------------------------------
phase_fn_t layered_phase(int epi, int R);
typedef void (*phase_pair_fn_t)(const PhaseArgs, const PhaseArgs, int);
phase_pair_fn_t layered_phase_pair(int R);

typedef void (*phase_parts_fn_t)(const PhaseArgs, const PhaseParts);
phase_parts_fn_t layered_phase_parts(int R);

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

// ---- latent attention (latent_attn.cu) ----
// Work on tokens one after the other in memory: one token at st->pos, or `tokens` of them from pos0 (st NULL).
struct LatentStep {
    LatentAttn at;
    const StepState* st;
    int pos0, tokens;
    const float* q;             // [tokens][heads * qrow] queries, not yet rotated
    const float* down;          // one token: [q_rank + rank + rot], its latent and rotated part go into the cache
    float* qa;                  // [tokens][heads][row]: U_k^T q and the rotated part, times scale
    int splits, tile, group;    // key ranges; keys per tile; heads per CTA
    float* part;                // [tokens][splits][heads][rank_s]
    float2* ml;                 // [tokens][splits][heads] maximum and sum of the range
    void* out;                  // [tokens][ld_out]
    int ld_out;
};
// Tile and heads per CTA of the attention over cached rows; 0: the sizes do not fit.
size_t latent_attend_smem(const LatentAttn& at, bool f32_cache, int* tile, int* group);
cudaError_t launch_latent_query(const LatentStep& a, bool f32_cache, bool pdl, cudaStream_t s);
cudaError_t launch_latent_attend(const LatentStep& a, bool f32_cache, bool pdl, cudaStream_t s);
cudaError_t launch_latent_value(const LatentStep& a, bool f32_out, bool pdl, cudaStream_t s);
// rows of a portion: act = normed query latent; normed latent and rotated key part into the cache
cudaError_t launch_latent_rows(const LatentAttn& at, const float* down, int ldd, int pos0, int n, void* act, int ld_act, bool f32, cudaStream_t s);
// rows of a portion: qh = queries with their rotated part rotated, times scale * log2 e (bf16)
cudaError_t launch_latent_q_rows(const LatentAttn& at, const float* q, int pos0, int n, void* qh, cudaStream_t s);
// bf16 prompts on the tensor cores (latent_attn_tc.cu): keys [max_seq][heads * dim_s] and values, transposed,
// [heads * vdim][ldv] of positions [0, pos0 + n) are formed from the cache, then attention in tiles of 128 queries.
bool latent_attn_tc_fits(const LatentAttn& at);
cudaError_t launch_latent_attn_tc(const LatentAttn& at, const void* qh, int pos0, int n, void* keys, void* vt, int ldv, void* out, int ld_out,
                                  int* status, int* launches, cudaStream_t s);

// ---- linear recurrence (wkv.cu) ----
struct WkvStep {
    Wkv wk;
    const float* row;           // r, k, v, g [heads * dim] each, then the decay's inner projection [rank]
    const StepState* st;
    float* y;                   // [heads * dim]
};
cudaError_t launch_wkv_step(const WkvStep& a, bool pdl, cudaStream_t s);
size_t wkv_step_smem(const Wkv& wk);
// act[j][r] = the mix of row r and the one before it (prev before the first) with mu[j]
cudaError_t launch_wkv_mix(const float* h, const float* prev, const float* const mu[5], int pos0, int n, int width, void* act, int ld_act,
                           long long act_stride, bool f32, cudaStream_t s);
// act[n][ld] = tanh of the decay's inner projection (the sum of `slices` slabs [n][ldp]) as two bf16 parts
cudaError_t launch_wkv_inner(const float* inner, int ldp, int slices, int rank, int n, void* act, int ld, cudaStream_t s);
bool wkv_rows_fits(const Wkv& wk);
// proj rows as WkvStep's, decays [n][heads * dim]; out [n][heads * dim] raw outputs
cudaError_t launch_wkv_rows(const Wkv& wk, const float* proj, int ldp, const float* decay, int pos0, int n, float* out, cudaStream_t s);

// ---- mixture of experts (moe.cu) ----
struct MoeStep {
    Moe moe;
    const float* router;        // one router row
    const float* h;             // [ldw] normed, zero from width on
    int* sel;                   // [top] the choice, made by launch_moe_up's kernel
    float* mid;                 // [top * ffs + shared_ffs] inner vectors of the chosen experts and the shared one
    float* out;                 // [width]
};
size_t moe_step_smem(const Moe& m);
cudaError_t moe_step_attrs(size_t bytes);
cudaError_t launch_moe_up(const MoeStep& a, int sms, bool pdl, cudaStream_t s);
cudaError_t launch_moe_down(const MoeStep& a, int sms, bool pdl, cudaStream_t s);
struct MoeRows {                // workspace of a portion
    int *sel, *slot;            // [n][top] chosen expert, its row among the grouped rows
    float* weight;              // [n][top]
    float* shared_gate;         // [n]
    int* count;                 // [experts], zero between calls
    int* first;                 // [experts + 1] first grouped row of an expert
    int* group;                 // [tiles] expert of every 128 grouped rows, -1: none
    int tiles;
    void* x;                    // [tiles * 128][ldw] grouped inputs
    void* y;                    // [tiles * 128][width] grouped outputs, bf16 or fp32
};
inline int moe_tiles(const Moe& m, int n) { return (int)(((long long)n * m.top + 127) / 128) + m.experts; }
// choice, grouping, the grouped inputs and the shared expert's gate; the router rows are the sum of `slices` slabs
// [n][ldr]
cudaError_t launch_moe_route(const Moe& m, const float* router, int ldr, int slices, int n, const void* act, bool f32, const MoeRows& w, cudaStream_t s);
// z = weighted sum of the grouped rows (+ z times the shared expert's gate)
cudaError_t launch_moe_combine(const Moe& m, int n, const MoeRows& w, float* z, bool f32, cudaStream_t s);

// ---- portions of a prompt (layered_prefill.cu) -----------------------------------------------------
// `act` buffers hold bf16 or fp32 (f32 = true) rows padded to a multiple of 64 with zeros.
cudaError_t launch_embed_rows(const WeightView& embed, int ld_embed, const float* pos_tab, const int* tokens, int pos0, int n,
                              int width, float* x, void* act, int ld_act, bool f32, cudaStream_t s);
// out[n][ldc] = A[n][K] W[rows][K]^T, fp32 on the CUDA cores (32-bit mode, and what is 32-bit in every mode)
enum : int { F32_STORE = 0, F32_GELU = 1,
             F32_SILU_MUL = 2,      // silu(aux) * the product
             F32_DECAY = 3 };       // exp(-exp(tanh(A) W^T + bias))
struct GemmF32 {
    const float* A;
    int lda;
    const uint8_t* W;
    int ldw;
    float* out;
    int ldc, n, rows, K, epi;
    const float* aux;               // [n][ldc]
    const float* bias;              // [rows]
    const int* group;               // per 128 rows of A: which of the stacked matrices (-1: none); NULL: one matrix
    long long group_stride;         // elements between the stacked matrices
};
cudaError_t launch_gemm_f32(const GemmF32& g, cudaStream_t s);
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
// act[r] = norm(x[rows[r]]) of the kind NORM_*
cudaError_t launch_last_norm_rows(const float* x, const int* rows, const float* w, int kind, float eps, int n, int width, void* act,
                                  int ld_act, bool f32, cudaStream_t s);
// x += mult * ls * z (where z is given); then act (or h, 32-bit rows without padding) = norm(x), or, where cat is
// given, act = [x, cat]
struct PrenormRows {
    float* x;
    const float *z, *ls;
    float mult;
    const float* norm_w;            // NULL: no norm, act = x where given
    int kind;
    float eps;
    int n, width;
    void* act;
    int ld_act;
    float* h;
    const float* cat;
};
cudaError_t launch_prenorm_rows(const PrenormRows& a, bool f32, cudaStream_t s);
// act[t] = unit rms per head of o[t] (a norm weight over all heads) times a gate
enum : int { GATE_SIGMOID = 0, GATE_SILU = 1 };
cudaError_t launch_head_norm_rows(int heads, int vdim, float eps, const float* norm, const float* gate, int ldg, int gate_kind, int n,
                                  const float* o, void* act, int ld_act, bool f32, cudaStream_t s);

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
