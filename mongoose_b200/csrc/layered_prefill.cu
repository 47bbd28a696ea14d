// Portions of a prompt of a layer-described model: row-wise kernels, the 32-bit matrix product, attention on
// the CUDA cores (32-bit mode and head counts the tensor-core kernel does not take), and the matrix
// memory in chunked form: every chunk's contribution in parallel, one pass over the chunks, then every
// chunk's outputs in parallel.
#include "layered_ops.cuh"

namespace mg {

namespace {

template <typename AT>
__global__ void __launch_bounds__(256) embed_rows_kernel(WeightView embed, int ld_embed, const float* pos_tab, const int* tokens,
                                                         int pos0, int width, float* x, AT* act, int ld_act) {
    const int r = blockIdx.x, token = tokens[r];
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = embed_value(embed, FMT_BF16, ld_embed, token, i) + (pos_tab ? pos_tab[(size_t)(pos0 + r) * width + i] : 0.f);
        x[(size_t)r * width + i] = v;
        from_f32(v, act + (size_t)r * ld_act + i);
    }
}

// 64 x 64 tile, 16 columns of K per step, 4 x 4 outputs per thread.  W's rows are padded with zeros to a multiple
// of 16 at least; A's columns from K on are not read.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32 g) {
    __shared__ __align__(16) float As[16][68], Ws[16][68];
    const int r0 = blockIdx.y * 64, c0 = blockIdx.x * 64;
    const __nv_bfloat16* W = reinterpret_cast<const __nv_bfloat16*>(g.W);
    if (g.group) {
        const int e = g.group[r0 / 128];
        if (e < 0) return;
        W += e * g.group_stride;
    }
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < g.K; k0 += 16) {
        float a4[4] = {0.f, 0.f, 0.f, 0.f};
        float2 w0 = make_float2(0.f, 0.f), w1 = w0;
        if (r0 + lr < g.n) {
            const float* ap = g.A + (size_t)(r0 + lr) * g.lda + k0 + lk;
            if (k0 + lk + 4 <= g.K) {
                const float4 av = *reinterpret_cast<const float4*>(ap);
                a4[0] = av.x; a4[1] = av.y; a4[2] = av.z; a4[3] = av.w;
            } else {
                for (int i = 0; i < 4; i++)
                    if (k0 + lk + i < g.K) a4[i] = ap[i];
            }
            if (g.epi == F32_DECAY)
                for (int i = 0; i < 4; i++) a4[i] = tanhf(a4[i]);
        }
        if (c0 + lr < g.rows) {
            const __nv_bfloat16* wp = W + (size_t)(c0 + lr) * g.ldw + k0 + lk;
            w0 = pair_f32(wp);
            w1 = pair_f32(wp + 2);
        }
        As[lk][lr] = a4[0]; As[lk + 1][lr] = a4[1]; As[lk + 2][lr] = a4[2]; As[lk + 3][lr] = a4[3];
        Ws[lk][lr] = w0.x; Ws[lk + 1][lr] = w0.y; Ws[lk + 2][lr] = w1.x; Ws[lk + 3][lr] = w1.y;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; k++) {
            const float4 a = *reinterpret_cast<const float4*>(&As[k][ty * 4]), w = *reinterpret_cast<const float4*>(&Ws[k][tx * 4]);
            const float aa[4] = {a.x, a.y, a.z, a.w}, ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(aa[i], ww[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int r = r0 + ty * 4 + i, c = c0 + tx * 4 + j;
            if (r >= g.n || c >= g.rows) continue;
            float v = acc[i][j];
            if (g.epi == F32_GELU) v = gelu_tanh(v);
            else if (g.epi == F32_SILU_MUL) v *= silu(g.aux[(size_t)r * g.ldc + c]);
            else if (g.epi == F32_DECAY) v = expf(-expf(v + g.bias[c]));
            g.out[(size_t)r * g.ldc + c] = v;
        }
}

// One warp per (token, query head or key head).
template <typename AT>
__global__ void __launch_bounds__(256) qk_rows_kernel(GateAttn A, const float* proj, int ldp, int q_col, int k_col, int pos0, int n,
                                                      AT* qh) {
    const int w = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    const int per = A.heads + A.kv_heads, t = w / per, h = w - t * per;
    if (t >= n) return;
    const float* row = proj + (size_t)t * ldp;
    if (h < A.heads)
        norm_query(A, row + q_col + h * A.dim, query_temp(A, pos0 + t), qh + ((size_t)t * A.heads + h) * A.dim_s, lane);
    else
        store_key<AT>(A, row + k_col + (h - A.heads) * A.dim, pos0 + t, h - A.heads, lane);
}

template <typename KT, int NQ, int EP>
__global__ void __launch_bounds__(kAttnThreads) gate_attn_rows_kernel(GateAttn A, const KT* qh, int pos0, int n, int tile, KT* out,
                                                                      int ld_out) {
    extern __shared__ __align__(16) float smem[];
    const AttnSmem<KT> sm(A, NQ, tile, smem);
    const int t0 = (gridDim.x - 1 - blockIdx.x) * NQ;      // the longest rows first
    const int row = A.heads * A.dim_s;
    for (int i = threadIdx.x; i < NQ * row; i += kAttnThreads)
        sm.q[i / A.dim_s * sm.qs + i % A.dim_s] = t0 + i / row < n ? to_f32(qh[(size_t)t0 * row + i]) : 0.f;
    sm.load_tables(A);
    __syncthreads();
    const int last = min(t0 + NQ, n) - 1;
    float acc[NQ][EP][2] = {};
    attend<KT, NQ, EP>(A, sm, pos0 + t0, 0, pos0 + last + 1, tile, acc);
#pragma unroll
    for (int e = 0; e < EP; e++) {
        const int el = 2 * (threadIdx.x + e * kAttnThreads);
        if (el >= row) continue;
        const int h = el / A.dim_s, d = el - h * A.dim_s;
#pragma unroll
        for (int q = 0; q < NQ; q++) {
            if (t0 + q > last) continue;
            KT* o = out + (size_t)(t0 + q) * ld_out + h * A.dim + d;
            if (d < A.dim) from_f32(acc[q][e][0], o);
            if (d + 1 < A.dim) from_f32(acc[q][e][1], o + 1);
        }
    }
}

template <typename AT>
__global__ void __launch_bounds__(256) post_rows_kernel(float* x, const float* z0, const float* z1, const float* w0, const float* w1,
                                                        const float* post_w, float eps, int width, AT* act, int ld_act) {
    extern __shared__ __align__(16) float y[];
    __shared__ float red[40];
    const size_t r = blockIdx.x;
    const float inv = 1.0f / (float)width;
    const float *a = z0 + r * width, *b = z1 ? z1 + r * width : nullptr;
    float ra = 1.f, rb = 0.f, ss = 0.f;
    if (b) {
        float s0 = 0.f, s1 = 0.f;
        for (int i = threadIdx.x; i < width; i += blockDim.x) { s0 = fmaf(a[i], a[i], s0); s1 = fmaf(b[i], b[i], s1); }
        ra = 0.5f / sqrtf(block_sum(s0, red) * inv + eps);
        rb = 0.5f / sqrtf(block_sum(s1, red) * inv + eps);
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = b ? a[i] * ra * w0[i] + b[i] * rb * w1[i] : a[i];
        y[i] = v;
        ss = fmaf(v, v, ss);
    }
    const float rr = 1.0f / sqrtf(block_sum(ss, red) * inv + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = x[r * width + i] + y[i] * rr * (1.0f + post_w[i]);
        x[r * width + i] = v;
        from_f32(v, act + r * ld_act + i);
    }
}

// Mean and 1 / sqrt(spread + eps) of row y for a norm of the given kind; a thread reads V values at a time, those
// it would write in a loop of the same shape.
template <int V>
__device__ __forceinline__ float2 row_norm(const float* y, int kind, float eps, int width, float* red) {
    const float inv = 1.0f / (float)width;
    float s = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V];
        load_values<V>(y + i, v);
#pragma unroll
        for (int q = 0; q < V; q++) s += kind == NORM_LAYER ? v[q] : v[q] * v[q];
    }
    s = block_sum(s, red) * inv;
    if (kind != NORM_LAYER) return make_float2(0.f, 1.0f / sqrtf(s + eps));
    float d = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V];
        load_values<V>(y + i, v);
#pragma unroll
        for (int q = 0; q < V; q++) d = fmaf(v[q] - s, v[q] - s, d);
    }
    return make_float2(s, 1.0f / sqrtf(block_sum(d, red) * inv + eps));
}

template <typename AT>
__global__ void __launch_bounds__(256) last_norm_rows_kernel(const float* x, const int* rows, const float* w, int kind, float eps, int width,
                                                             AT* act, int ld_act) {
    __shared__ float red[40];
    const float* a = x + (size_t)rows[blockIdx.x] * width;
    const float2 n = row_norm<1>(a, kind, eps, width, red);
    const float one = kind == NORM_RMS_AROUND_ZERO ? 1.0f : 0.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) from_f32((a[i] - n.x) * n.y * (one + w[i]), act + (size_t)blockIdx.x * ld_act + i);
}

template <typename AT, int V>
__global__ void __launch_bounds__(256) prenorm_rows_kernel(const PrenormRows a) {
    extern __shared__ __align__(16) float y[];
    __shared__ float red[40];
    const int W = a.width, step = 256 * V;
    const size_t r = blockIdx.x;
    float* x = a.x + r * W;
    AT* act = static_cast<AT*>(a.act) + r * a.ld_act;
    for (int i = threadIdx.x * V; i < W; i += step) {
        float v[V];
        load_values<V>(x + i, v);
        if (a.z) {
            float z[V], ls[V];
            load_values<V>(a.z + r * W + i, z);
            load_values<V>(a.ls + i, ls);
#pragma unroll
            for (int q = 0; q < V; q++) v[q] += a.mult * (ls[q] * z[q]);
            store_values<V>(v, x + i);
        }
        if (a.norm_w) store_values<V>(v, y + i);
        else if (a.act) store_values<V>(v, act + i);
        if (a.cat) {
            load_values<V>(a.cat + r * W + i, v);
            store_values<V>(v, act + W + i);
        }
    }
    if (!a.norm_w) return;
    const float2 n = row_norm<V>(y, a.kind, a.eps, W, red);
    const float one = a.kind == NORM_RMS_AROUND_ZERO ? 1.0f : 0.0f;
    for (int i = threadIdx.x * V; i < W; i += step) {
        float v[V], w[V];
        load_values<V>(y + i, v);
        load_values<V>(a.norm_w + i, w);
#pragma unroll
        for (int q = 0; q < V; q++) v[q] = (v[q] - n.x) * n.y * (one + w[q]);
        if (a.h) store_values<V>(v, a.h + r * W + i);
        else store_values<V>(v, act + i);
    }
}

// ---------------------------------------------------------------------
// Matrix memory in chunks of kMemChunk tokens.
// ---------------------------------------------------------------------

// One CTA per head, one warp per chunk: gates, the log-forget sum inside each chunk, and the running maximum
// m_t = max(f_t + m_{t-1}, i_t) as a scan of the maps m -> max(m + f, i): within halves of a chunk by
// shuffles, across the chunks through shared memory.
constexpr int kGateWarps = 32;

__global__ void __launch_bounds__(kGateWarps * 32) mem_gates_kernel(MatMem M, int i_col, int f_col, const float* proj, int ldp, int pos0,
                                                                    int n, MemRows w) {
    static_assert(kMemChunk == 64, "a warp holds a chunk as two tokens per lane");
    __shared__ double sum_f[kGateWarps];
    __shared__ float top_i[kGateWarps], m_end;
    const int h = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float m = pos0 == 0 ? 0.f : M.m[(pos0 & 1) * M.heads + h];      // before the chunks of this pass
    if (threadIdx.x == 0) w.m0[h] = m;
    const float ib = M.i_bias[h], fb = M.f_bias[h];
    for (int c0 = 0; c0 * kMemChunk < n; c0 += kGateWarps) {
        const int t0 = (c0 + warp) * kMemChunk;
        float ig[2], mi[2];
        double b[2];
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const int t = t0 + 32 * k + lane;
            ig[k] = -INFINITY;                      // tokens past n change nothing: f = 0, i = -inf
            float fg = 0.f;
            if (t < n) {
                ig[k] = soft_cap(proj[(size_t)t * ldp + i_col + h] + ib, M.cap);
                fg = log_sigmoid(soft_cap(proj[(size_t)t * ldp + f_col + h] + fb, M.cap));
            }
            b[k] = (double)fg;
            mi[k] = ig[k];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double pb = __shfl_up_sync(MG_FULL_MASK, b[k], o);
                const float pm = __shfl_up_sync(MG_FULL_MASK, mi[k], o);
                if (lane >= o) { mi[k] = fmaxf((float)((double)pm + b[k]), mi[k]); b[k] += pb; }
            }
        }
        const double b0 = __shfl_sync(MG_FULL_MASK, b[0], 31);
        const float i0 = __shfl_sync(MG_FULL_MASK, mi[0], 31);
        mi[1] = fmaxf((float)((double)i0 + b[1]), mi[1]);
        b[1] += b0;
        __syncthreads();                            // the last pass's sums have been read
        if (lane == 31) { sum_f[warp] = b[1]; top_i[warp] = mi[1]; }
        __syncthreads();
        float before = m;
        for (int c = 0; c < warp; c++) before = fmaxf((float)((double)before + sum_f[c]), top_i[c]);
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const int t = t0 + 32 * k + lane;
            const float mt = fmaxf((float)((double)before + b[k]), mi[k]);
            if (t < n) {
                w.b[(size_t)h * n + t] = b[k];
                w.ig[(size_t)h * n + t] = ig[k];
                w.mm[(size_t)h * n + t] = mt;
            }
            if (k == 1 && lane == 31) {
                if (t0 < n) w.g[(size_t)h * ((n + kMemChunk - 1) / kMemChunk) + c0 + warp] = expf((float)b[1] + before - mt);
                if (warp == kGateWarps - 1) m_end = mt;
            }
        }
        __syncthreads();
        m = m_end;
    }
    if (threadIdx.x == 0) M.m[((pos0 + n) & 1) * M.heads + h] = m;
}

// Running maximum before token t0 of the portion (the state's own slot may be overwritten by now).
__device__ __forceinline__ float mem_before(const MemRows& w, int h, int n, int t0) {
    return t0 > 0 ? w.mm[(size_t)h * n + t0 - 1] : w.m0[h];
}

// U[chunk][head] = sum over the chunk of exp(b_T - b_s + i_s - m_T) k_s v_s^T, a 64 x 64 tile per CTA.
__global__ void __launch_bounds__(256) mem_chunk_kernel(MatMem M, int k_col, int v_col, const float* proj, int ldp, int n, int vtiles,
                                                        MemRows w) {
    __shared__ __align__(16) float Ks[kMemChunk][68], Vs[kMemChunk][68];
    const int ch = blockIdx.x, h = blockIdx.y, d0 = blockIdx.z / vtiles * 64, v0 = blockIdx.z % vtiles * 64;
    const int t0 = ch * kMemChunk, T = min(kMemChunk, n - t0);
    const double bT = w.b[(size_t)h * n + t0 + T - 1];
    const float mT = w.mm[(size_t)h * n + t0 + T - 1];
    for (int i = threadIdx.x; i < kMemChunk * 64; i += 256) {
        const int s = i >> 6, c = i & 63;
        float k = 0.f, v = 0.f;
        if (s < T) {
            const float* row = proj + (size_t)(t0 + s) * ldp;
            if (d0 + c < M.dim)
                k = row[k_col + h * M.dim + d0 + c] *
                    expf((float)(bT - w.b[(size_t)h * n + t0 + s]) + w.ig[(size_t)h * n + t0 + s] - mT);
            if (v0 + c < M.vdim) v = row[v_col + h * M.vdim + v0 + c];
        }
        Ks[s][c] = k;
        Vs[s][c] = v;
    }
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {}, nk[4] = {};
#pragma unroll 8
    for (int s = 0; s < kMemChunk; s++) {
        const float4 a = *reinterpret_cast<const float4*>(&Ks[s][ty * 4]), b = *reinterpret_cast<const float4*>(&Vs[s][tx * 4]);
        const float aa[4] = {a.x, a.y, a.z, a.w}, bb[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            nk[i] += aa[i];
#pragma unroll
            for (int j = 0; j < 4; j++) acc[i][j] = fmaf(aa[i], bb[j], acc[i][j]);
        }
    }
    float* U = w.U + ((size_t)ch * M.heads + h) * M.dim * M.vdim;
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int d = d0 + ty * 4 + i;
        if (d >= M.dim) continue;
        if (v0 == 0 && tx == 0) w.nU[((size_t)ch * M.heads + h) * M.dim + d] = nk[i];
#pragma unroll
        for (int j = 0; j < 4; j++)
            if (v0 + tx * 4 + j < M.vdim) U[(size_t)d * M.vdim + v0 + tx * 4 + j] = acc[i][j];
    }
}

// Pass over the chunks: U becomes the state BEFORE each chunk, and the state after the last is stored.
__global__ void __launch_bounds__(256) mem_scan_kernel(MatMem M, int pos0, int n, int chunks, MemRows w) {
    const size_t per = (size_t)M.dim * M.vdim, all = M.heads * per, nall = (size_t)M.heads * M.dim;
    const size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= all + nall) return;
    const bool is_n = e >= all;
    const size_t i = is_n ? e - all : e;
    const int h = (int)(i / (is_n ? (size_t)M.dim : per));
    float* U = is_n ? w.nU + i : w.U + i;
    const size_t stride = is_n ? nall : all;
    float s = 0.f;
    if (pos0 > 0) s = is_n ? M.nrm[(pos0 & 1) * nall + i] : M.S[i];
    const float* g = w.g + (size_t)h * chunks;
    for (int c0 = 0; c0 < chunks; c0 += 8) {        // eight chunks' loads in flight
        float u[8], gg[8];
#pragma unroll
        for (int i = 0; i < 8; i++) {
            u[i] = c0 + i < chunks ? U[(c0 + i) * stride] : 0.f;
            gg[i] = c0 + i < chunks ? g[c0 + i] : 1.f;
        }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            if (c0 + i < chunks) U[(c0 + i) * stride] = s;
            s = fmaf(gg[i], s, u[i]);
        }
    }
    if (is_n) M.nrm[((pos0 + n) & 1) * nall + i] = s;
    else M.S[i] = s;
}

// Outputs of one chunk and head, 64 value columns per CTA.
__global__ void __launch_bounds__(256) mem_out_kernel(MatMem M, int q_col, int k_col, int v_col, const float* proj, int ldp,
                                                      int n, MemRows w) {
    __shared__ __align__(16) float Qs[32][68], Ks[32][68], Ss[32][68];
    __shared__ __align__(16) float P[kMemChunk][68];            // [s][t]
    __shared__ float nq_s[kMemChunk], ns[32];
    __shared__ double bs[kMemChunk];
    __shared__ float is[kMemChunk], ms[kMemChunk];
    float (*Vs)[68] = reinterpret_cast<float (*)[68]>(&Qs[0][0]);   // 64 rows over Qs and Ks once they are consumed
    static_assert(sizeof(Qs) + sizeof(Ks) == 64 * 68 * 4, "the value tile reuses the query and key tiles");
    const int ch = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 64;
    const int t0 = ch * kMemChunk, T = min(kMemChunk, n - t0);
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    if (threadIdx.x < kMemChunk) {
        const int t = threadIdx.x;
        bs[t] = t < T ? w.b[(size_t)h * n + t0 + t] : 0.0;
        is[t] = t < T ? w.ig[(size_t)h * n + t0 + t] : -INFINITY;
        ms[t] = t < T ? w.mm[(size_t)h * n + t0 + t] : 0.f;
    }
    const float mprev = mem_before(w, h, n, t0);
    const float qscale = 1.0f / sqrtf((float)M.dim);
    const float* U = w.U + ((size_t)ch * M.heads + h) * M.dim * M.vdim;
    const float* nU = w.nU + ((size_t)ch * M.heads + h) * M.dim;
    float pa[4][4] = {}, oa[4][4] = {};         // rows t = ty*4.., columns s or v = tx*4..
    float nq = 0.f;                             // thread t < 64: n_prev . q_t
    for (int k0 = 0; k0 < M.dim; k0 += 32) {
        __syncthreads();
#pragma unroll
        for (int i = threadIdx.x; i < 32 * 64; i += 256) {
            const int t = i >> 5, d = i & 31;
            float q = 0.f, k = 0.f;
            if (t < T && k0 + d < M.dim) {
                const float* row = proj + (size_t)(t0 + t) * ldp + h * M.dim + k0 + d;
                q = row[q_col] * qscale;
                k = row[k_col];
            }
            Qs[d][t] = q;
            Ks[d][t] = k;
            const int sd = i >> 6, sv = i & 63;
            Ss[sd][sv] = k0 + sd < M.dim && v0 + sv < M.vdim ? U[(size_t)(k0 + sd) * M.vdim + v0 + sv] : 0.f;
        }
        if (threadIdx.x < 32) ns[threadIdx.x] = k0 + threadIdx.x < M.dim ? nU[k0 + threadIdx.x] : 0.f;
        __syncthreads();
        if (threadIdx.x < kMemChunk) {
#pragma unroll 8
            for (int d = 0; d < 32; d++) nq = fmaf(ns[d], Qs[d][threadIdx.x], nq);
        }
#pragma unroll 8
        for (int d = 0; d < 32; d++) {
            const float4 a = *reinterpret_cast<const float4*>(&Qs[d][ty * 4]), b = *reinterpret_cast<const float4*>(&Ks[d][tx * 4]),
                         c = *reinterpret_cast<const float4*>(&Ss[d][tx * 4]);
            const float aa[4] = {a.x, a.y, a.z, a.w}, bb[4] = {b.x, b.y, b.z, b.w}, cc[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    pa[i][j] = fmaf(aa[i], bb[j], pa[i][j]);
                    oa[i][j] = fmaf(aa[i], cc[j], oa[i][j]);
                }
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int t = ty * 4 + i;
        const float inter = t < T ? expf((float)bs[t] + mprev - ms[t]) : 0.f;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int s = tx * 4 + j;
            P[s][t] = s <= t && t < T ? pa[i][j] * expf((float)(bs[t] - bs[s]) + is[s] - ms[t]) : 0.f;
            oa[i][j] *= inter;
        }
    }
    for (int i = threadIdx.x; i < kMemChunk * 64; i += 256) {
        const int s = i >> 6, c = i & 63;
        Vs[s][c] = s < T && v0 + c < M.vdim ? proj[(size_t)(t0 + s) * ldp + v_col + h * M.vdim + v0 + c] : 0.f;
    }
    __syncthreads();
    if (threadIdx.x < kMemChunk) {
        const int t = threadIdx.x;
        float d = nq * (t < T ? expf((float)bs[t] + mprev - ms[t]) : 0.f);
        for (int s = 0; s < kMemChunk; s++) d += P[s][t];
        nq_s[t] = 1.0f / (fmaxf(fabsf(d), expf(-ms[t])) + 1e-6f);
    }
#pragma unroll 8
    for (int s = 0; s < kMemChunk; s++) {
        const float4 a = *reinterpret_cast<const float4*>(&P[s][ty * 4]), b = *reinterpret_cast<const float4*>(&Vs[s][tx * 4]);
        const float aa[4] = {a.x, a.y, a.z, a.w}, bb[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) oa[i][j] = fmaf(aa[i], bb[j], oa[i][j]);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int t = ty * 4 + i;
        if (t >= T) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int v = v0 + tx * 4 + j;
            if (v < M.vdim) w.o[(size_t)(t0 + t) * M.heads * M.vdim + h * M.vdim + v] = oa[i][j] * nq_s[t];
        }
    }
}

// One warp per (token, head): unit rms, norm weight, output gate.
template <typename AT>
__global__ void __launch_bounds__(256) head_norm_rows_kernel(int heads, int vdim, float eps, const float* norm, const float* gate, int ldg,
                                                             int gate_kind, int n, const float* o, AT* act, int ld_act) {
    const int wq = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    const int t = wq / heads, h = wq - t * heads;
    if (t >= n) return;
    const float* p = o + ((size_t)t * heads + h) * vdim;
    float ss = 0.f;
    for (int v = lane; v < vdim; v += 32) ss = fmaf(p[v], p[v], ss);
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int v = lane; v < vdim; v += 32) {
        const int c = h * vdim + v;
        const float g = gate[(size_t)t * ldg + c];
        from_f32(p[v] * r * norm[c] * (gate_kind == GATE_SILU ? silu(g) : sigmoid(g)), act + (size_t)t * ld_act + c);
    }
}

// The same with a quad of values per lane and `lanes` lanes (a power of two) per head: head sizes that are whole
// quads, up to 128.
template <typename AT>
__global__ void __launch_bounds__(256) head_norm_quads_kernel(int heads, int vdim, int lanes, float eps, const float* norm, const float* gate,
                                                              int ldg, int gate_kind, int n, const float* o, AT* act, int ld_act) {
    const int unit = (blockIdx.x * 256 + threadIdx.x) / lanes, sub = threadIdx.x & (lanes - 1);
    const int t = unit / heads, h = unit - t * heads, c = h * vdim + sub * 4;
    const bool in = t < n && sub * 4 < vdim;
    float v[4] = {}, g[4], w[4];
    if (in) {
        load_values<4>(o + (size_t)t * heads * vdim + c, v);
        load_values<4>(gate + (size_t)t * ldg + c, g);
        load_values<4>(norm + c, w);
    }
    float ss = v[0] * v[0] + v[1] * v[1] + v[2] * v[2] + v[3] * v[3];
    for (int m = lanes / 2; m > 0; m >>= 1) ss += __shfl_xor_sync(MG_FULL_MASK, ss, m);
    const float r = 1.0f / sqrtf(ss / (float)vdim + eps);
    if (!in) return;
#pragma unroll
    for (int q = 0; q < 4; q++) v[q] *= r * w[q] * (gate_kind == GATE_SILU ? silu(g[q]) : sigmoid(g[q]));
    store_values<4>(v, act + (size_t)t * ld_act + c);
}

template <typename KT, int NQ>
cudaError_t attn_rows_for(const GateAttn& at, const void* qh, int pos0, int n, void* out, int ld_out, cudaStream_t s) {
    int tile;
    const size_t smem = attn_smem(at, NQ, sizeof(KT), 32, &tile);
    if (!smem) return cudaErrorInvalidValue;
    auto run = [&](auto kern) {
        cudaError_t c = cudaFuncSetAttribute((const void*)kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (c != cudaSuccess) return c;
        kern<<<(n + NQ - 1) / NQ, kAttnThreads, smem, s>>>(at, (const KT*)qh, pos0, n, tile, (KT*)out, ld_out);
        return cudaGetLastError();
    };
    switch (attn_pairs(at)) {
        case 1: return run(gate_attn_rows_kernel<KT, NQ, 1>);
        case 2: return run(gate_attn_rows_kernel<KT, NQ, 2>);
        case 4: return run(gate_attn_rows_kernel<KT, NQ, 4>);
        case 8: return run(gate_attn_rows_kernel<KT, NQ, 8>);
        case 16: return run(gate_attn_rows_kernel<KT, NQ, 16>);
    }
    return cudaErrorInvalidValue;
}

}  // namespace

cudaError_t launch_embed_rows(const WeightView& embed, int ld_embed, const float* pos_tab, const int* tokens, int pos0, int n,
                              int width, float* x, void* act, int ld_act, bool f32, cudaStream_t s) {
    if (f32) embed_rows_kernel<float><<<n, 256, 0, s>>>(embed, ld_embed, pos_tab, tokens, pos0, width, x, (float*)act, ld_act);
    else embed_rows_kernel<__nv_bfloat16><<<n, 256, 0, s>>>(embed, ld_embed, pos_tab, tokens, pos0, width, x, (__nv_bfloat16*)act, ld_act);
    return cudaGetLastError();
}

cudaError_t launch_gemm_f32(const GemmF32& g, cudaStream_t s) {
    gemm_f32_kernel<<<dim3((g.rows + 63) / 64, (g.n + 63) / 64), 256, 0, s>>>(g);
    return cudaGetLastError();
}

cudaError_t launch_qk_rows(const GateAttn& at, const float* proj, int ldp, int q_col, int k_col, int pos0, int n, void* qh, bool f32,
                           cudaStream_t s) {
    const int grid = (n * (at.heads + at.kv_heads) + 7) / 8;
    if (f32) qk_rows_kernel<float><<<grid, 256, 0, s>>>(at, proj, ldp, q_col, k_col, pos0, n, (float*)qh);
    else qk_rows_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(at, proj, ldp, q_col, k_col, pos0, n, (__nv_bfloat16*)qh);
    return cudaGetLastError();
}

size_t gate_attn_rows_smem(const GateAttn& at, bool f32, int* tile) { return attn_smem(at, 1, f32 ? 4 : 2, 32, tile); }

cudaError_t launch_gate_attn_rows(const GateAttn& at, const void* qh, int pos0, int n, void* out, int ld_out, bool f32, cudaStream_t s) {
    int tile;
    const bool four = attn_pairs(at) <= 8 && attn_smem(at, 4, f32 ? 4 : 2, 32, &tile) > 0;
    if (f32) return four ? attn_rows_for<float, 4>(at, qh, pos0, n, out, ld_out, s) : attn_rows_for<float, 1>(at, qh, pos0, n, out, ld_out, s);
    return four ? attn_rows_for<__nv_bfloat16, 4>(at, qh, pos0, n, out, ld_out, s)
                : attn_rows_for<__nv_bfloat16, 1>(at, qh, pos0, n, out, ld_out, s);
}

cudaError_t launch_post_rows(float* x, const float* z0, const float* z1, const float* w0, const float* w1, const float* post_w, float eps,
                             int n, int width, void* act, int ld_act, bool f32, cudaStream_t s) {
    const size_t smem = (size_t)width * sizeof(float);
    if (f32) post_rows_kernel<float><<<n, 256, smem, s>>>(x, z0, z1, w0, w1, post_w, eps, width, (float*)act, ld_act);
    else post_rows_kernel<__nv_bfloat16><<<n, 256, smem, s>>>(x, z0, z1, w0, w1, post_w, eps, width, (__nv_bfloat16*)act, ld_act);
    return cudaGetLastError();
}

cudaError_t launch_last_norm_rows(const float* x, const int* rows, const float* w, int kind, float eps, int n, int width, void* act,
                                  int ld_act, bool f32, cudaStream_t s) {
    if (f32) last_norm_rows_kernel<float><<<n, 256, 0, s>>>(x, rows, w, kind, eps, width, (float*)act, ld_act);
    else last_norm_rows_kernel<__nv_bfloat16><<<n, 256, 0, s>>>(x, rows, w, kind, eps, width, (__nv_bfloat16*)act, ld_act);
    return cudaGetLastError();
}

cudaError_t launch_prenorm_rows(const PrenormRows& a, bool f32, cudaStream_t s) {
    const size_t smem = (size_t)a.width * sizeof(float);
    const bool quads = a.width % 4 == 0;
    if (f32 && quads) prenorm_rows_kernel<float, 4><<<a.n, 256, smem, s>>>(a);
    else if (f32) prenorm_rows_kernel<float, 1><<<a.n, 256, smem, s>>>(a);
    else if (quads) prenorm_rows_kernel<__nv_bfloat16, 4><<<a.n, 256, smem, s>>>(a);
    else prenorm_rows_kernel<__nv_bfloat16, 1><<<a.n, 256, smem, s>>>(a);
    return cudaGetLastError();
}

template <typename AT>
static cudaError_t head_norm_for(int heads, int vdim, float eps, const float* norm, const float* gate, int ldg, int gate_kind, int n, const float* o,
                                 AT* act, int ld_act, cudaStream_t s) {
    const bool quads = vdim % 4 == 0 && vdim <= 128 && ldg % 4 == 0 && (reinterpret_cast<uintptr_t>(gate) & 15) == 0;
    int lanes = 1;
    while (lanes * 4 < vdim) lanes *= 2;
    if (quads)
        head_norm_quads_kernel<AT><<<(int)(((long long)n * heads * lanes + 255) / 256), 256, 0, s>>>(heads, vdim, lanes, eps, norm, gate, ldg, gate_kind, n, o, act, ld_act);
    else
        head_norm_rows_kernel<AT><<<(n * heads + 7) / 8, 256, 0, s>>>(heads, vdim, eps, norm, gate, ldg, gate_kind, n, o, act, ld_act);
    return cudaGetLastError();
}

cudaError_t launch_head_norm_rows(int heads, int vdim, float eps, const float* norm, const float* gate, int ldg, int gate_kind, int n,
                                  const float* o, void* act, int ld_act, bool f32, cudaStream_t s) {
    return f32 ? head_norm_for(heads, vdim, eps, norm, gate, ldg, gate_kind, n, o, (float*)act, ld_act, s)
               : head_norm_for(heads, vdim, eps, norm, gate, ldg, gate_kind, n, o, (__nv_bfloat16*)act, ld_act, s);
}

cudaError_t launch_mem_rows(const MatMem& mem, const ProjCols& c, const float* proj, int ldp, int pos0, int n, const MemRows& w, void* act,
                            int ld_act, bool f32, cudaStream_t s) {
    const int chunks = (n + kMemChunk - 1) / kMemChunk, dt = (mem.dim + 63) / 64, vt = (mem.vdim + 63) / 64;
    mem_gates_kernel<<<mem.heads, kGateWarps * 32, 0, s>>>(mem, c.mi, c.mf, proj, ldp, pos0, n, w);
    mem_chunk_kernel<<<dim3(chunks, mem.heads, dt * vt), 256, 0, s>>>(mem, c.mk, c.mv, proj, ldp, n, vt, w);
    const size_t elems = (size_t)mem.heads * mem.dim * (mem.vdim + 1);
    mem_scan_kernel<<<(unsigned)((elems + 255) / 256), 256, 0, s>>>(mem, pos0, n, chunks, w);
    mem_out_kernel<<<dim3(chunks, mem.heads, vt), 256, 0, s>>>(mem, c.mq, c.mk, c.mv, proj, ldp, n, w);
    return launch_head_norm_rows(mem.heads, mem.vdim, mem.eps, mem.norm, proj + c.mg, ldp, GATE_SIGMOID, n, w.o, act, ld_act, f32, s);
}

}  // namespace mg
