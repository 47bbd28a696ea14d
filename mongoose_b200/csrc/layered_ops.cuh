// Device code shared by the one-token and the prompt kernels of layer-described models.
#pragma once

#include "layered.h"

namespace mg {

constexpr int kAttnThreads = 256;

__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f32(float v, float* p) { *p = v; }
__device__ __forceinline__ void from_f32(float v, __nv_bfloat16* p) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float2 pair_f32(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 pair_f32(const __nv_bfloat16* p) {
    const uint32_t w = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(__uint_as_float(w << 16), __uint_as_float(w & 0xffff0000u));
}
// V values at once (V = 4: the address is a multiple of 16 bytes, of 8 for bf16)
template <int V>
__device__ __forceinline__ void load_values(const float* p, float (&o)[V]) {
    if constexpr (V == 4) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
    } else {
        o[0] = *p;
    }
}
template <int V>
__device__ __forceinline__ void load_values(const __nv_bfloat16* p, float (&o)[V]) {
    if constexpr (V == 4) {
        const uint2 v = *reinterpret_cast<const uint2*>(p);
        o[0] = __uint_as_float(v.x << 16); o[1] = __uint_as_float(v.x & 0xffff0000u);
        o[2] = __uint_as_float(v.y << 16); o[3] = __uint_as_float(v.y & 0xffff0000u);
    } else {
        o[0] = __bfloat162float(*p);
    }
}
template <int V>
__device__ __forceinline__ void store_values(const float (&v)[V], float* p) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}
template <int V>
__device__ __forceinline__ void store_values(const float (&v)[V], __nv_bfloat16* p) {
    if constexpr (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    } else {
        *p = __float2bfloat16_rn(v[0]);
    }
}
// 16 bytes of keys as floats
template <typename KT>
struct Chunk16;
template <>
struct Chunk16<float> {
    static constexpr int n = 4;
    __device__ static __forceinline__ void load(const float* p, float* o) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
    }
};
template <>
struct Chunk16<__nv_bfloat16> {
    static constexpr int n = 8;
    __device__ static __forceinline__ void load(const __nv_bfloat16* p, float* o) {
        const uint4 v = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            o[2 * i] = __uint_as_float(w[i] << 16);
            o[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
};

__device__ __forceinline__ float query_temp(const GateAttn& A, int pos) {
    return 1.0f + A.temp_coef * logf((float)((pos + 1) / A.temp_every + 1));
}

// One warp: out[dim_s] = q * (1 / rms) * q_norm * k_norm * scale * temp.  The key's own 1 / rms is applied to
// the finished dot product, so that the raw key row serves the score and the value.
template <typename OT>
__device__ __forceinline__ void norm_query(const GateAttn& A, const float* q, float temp, OT* out, int lane) {
    float ss = 0.f;
    for (int d = lane; d < A.dim; d += 32) ss = fmaf(q[d], q[d], ss);
    const float r = temp * A.scale / sqrtf(warp_sum(ss) / (float)A.dim + A.eps);
    for (int d = lane; d < A.dim_s; d += 32) from_f32(d < A.dim ? q[d] * r * A.q_norm[d] * A.k_norm[d] : 0.f, out + d);
}

// The same for every head of one token by the whole CTA, eight lanes per head.
__device__ __forceinline__ void norm_queries(const GateAttn& A, const float* q, float temp, float* out, int qs) {
    const int sub = threadIdx.x & 7;
    const unsigned mask = 0xffu << (threadIdx.x & 24);
    for (int h = threadIdx.x >> 3; h < A.heads; h += kAttnThreads / 8) {
        const float* p = q + h * A.dim;
        float v[16], ss = 0.f;              // the first 128 values are loaded at once
#pragma unroll
        for (int i = 0; i < 16; i++) {
            const int d = sub + 8 * i;
            v[i] = d < A.dim ? p[d] : 0.f;
            ss = fmaf(v[i], v[i], ss);
        }
        for (int d = sub + 128; d < A.dim; d += 8) ss = fmaf(p[d], p[d], ss);
        ss += __shfl_xor_sync(mask, ss, 1);
        ss += __shfl_xor_sync(mask, ss, 2);
        ss += __shfl_xor_sync(mask, ss, 4);
        const float r = temp * A.scale / sqrtf(ss / (float)A.dim + A.eps);
#pragma unroll
        for (int i = 0; i < 16; i++) {
            const int d = sub + 8 * i;
            if (d < A.dim_s) out[h * qs + d] = d < A.dim ? v[i] * r * A.q_norm[d] * A.k_norm[d] : 0.f;
        }
        for (int d = sub + 128; d < A.dim_s; d += 8) out[h * qs + d] = d < A.dim ? p[d] * r * A.q_norm[d] * A.k_norm[d] : 0.f;
    }
}

// One warp: key head c of position pos into the cache, with the 1 / rms of the row as stored.
template <typename KT>
__device__ __forceinline__ void store_key(const GateAttn& A, const float* k, int pos, int c, int lane) {
    KT* dst = static_cast<KT*>(A.cache) + ((size_t)pos * A.kv_heads + c) * A.dim_s;
    float ss = 0.f;
    for (int d = lane; d < A.dim_s; d += 32) {
        KT t;
        from_f32(d < A.dim ? k[d] : 0.f, &t);
        dst[d] = t;
        const float v = to_f32(t);
        ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) A.cache_r[(size_t)pos * A.kv_heads + c] = 1.0f / sqrtf(ss / (float)A.dim + A.eps);
}

// Keys [j0, j1) of part `split` when `len` keys are cut into at most `splits` parts of whole tiles;
// returns the number of parts in use.
__host__ __device__ inline int key_split(int len, int splits, int tile, int split, int* j0, int* j1) {
    const int per = pad_to((len + splits - 1) / splits, tile);
    *j0 = split * per < len ? split * per : len;
    *j1 = *j0 + per < len ? *j0 + per : len;
    return (len + per - 1) / per;
}

// Accumulator pairs per thread (rounded up to an instance), 0 when the heads do not fit.
inline int attn_pairs(const GateAttn& at) {
    if (at.dim_s > 1024) return 0;          // KeyCopy: a key row is at most one piece per thread
    const int pairs = (at.heads * at.dim_s / 2 + kAttnThreads - 1) / kAttnThreads;
    for (int p = 1; p <= 16; p *= 2)
        if (pairs <= p) return p;
    return 0;
}

// Rows in shared memory are 16 bytes longer than their data (mixed-head rows one float), so that lanes that
// walk different rows meet different banks.
template <typename KT>
struct AttnSmem {
    KT* k;          // [2][tile][kv_heads][ks]
    float* r;       // [2][tile][kv_heads]
    float* q;       // [nq][heads][qs]
    float* w;       // [nq][heads][ws] sigmoid weights
    float* mix;     // [nq][heads][ws] mixed over heads
    float *talk, *bias, *slope;
    int ks, qs, ws, ts;
    __device__ __forceinline__ AttnSmem(const GateAttn& A, int nq, int tile, float* base) {
        ks = A.dim_s + 16 / (int)sizeof(KT);
        qs = A.dim_s + 4;
        ws = tile + 1;
        ts = A.heads + 1;
        k = reinterpret_cast<KT*>(base);
        r = reinterpret_cast<float*>(k + 2 * (size_t)tile * A.kv_heads * ks);
        q = r + pad_to(2 * tile * A.kv_heads, 4);
        w = q + nq * A.heads * qs;
        mix = w + nq * A.heads * ws;
        talk = mix + nq * A.heads * ws;
        bias = talk + A.heads * ts;
        slope = bias + A.heads;
    }
    __device__ __forceinline__ void load_tables(const GateAttn& A) const {
        for (int h = threadIdx.x / 32; h < A.heads; h += kAttnThreads / 32)
            for (int g = threadIdx.x % 32; g < A.heads; g += 32) talk[h * ts + g] = A.talk[h * A.heads + g];
        for (int i = threadIdx.x; i < A.heads; i += kAttnThreads) { bias[i] = A.head_bias[i]; slope[i] = A.slopes[i]; }
    }
};

// Bytes of AttnSmem with the largest tile of at most `most` keys (a power of two) that fits; 0 when none does.
inline size_t attn_smem(const GateAttn& at, int nq, int kt_bytes, int most, int* tile) {
    if (!attn_pairs(at)) return 0;
    for (int t = most; t >= 2; t /= 2) {
        const size_t b = 2 * (size_t)t * at.kv_heads * (at.dim_s * kt_bytes + 16) +
                         ((size_t)pad_to(2 * t * at.kv_heads, 4) + (size_t)nq * at.heads * (at.dim_s + 4 + 2 * (t + 1)) +
                          (size_t)at.heads * (at.heads + 1) + 2 * at.heads) * sizeof(float);
        if (b <= 200 * 1024) { *tile = t; return b; }
    }
    return 0;
}

// Maximum over a whole CTA; every thread gets it.  `red` as for block_sum.
__device__ __forceinline__ float block_max(float v, float* red) {
    v = warp_max(v);
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (lane == 0) red[wid] = v;
    __syncthreads();
    return warp_max(lane < nw ? red[lane] : -INFINITY);
}

// Two fp32 operations at once.
__device__ __forceinline__ unsigned long long pack2(float a, float b) {
    return (unsigned long long)__float_as_uint(a) | ((unsigned long long)__float_as_uint(b) << 32);
}
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
    unsigned long long d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b) {
    unsigned long long d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ float lo(unsigned long long v) { return __uint_as_float((unsigned)v); }
__device__ __forceinline__ float hi(unsigned long long v) { return __uint_as_float((unsigned)(v >> 32)); }

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void cp_async4(void* smem, const void* gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}

// Which 16-byte pieces of a tile this thread copies: piece `ch` of rows row0, row0 + step, ...
struct KeyCopy {
    int ch, row0, step;
    __device__ __forceinline__ KeyCopy(int pieces) {
        step = kAttnThreads / pieces;
        row0 = threadIdx.x / pieces;
        ch = threadIdx.x - row0 * pieces;
        if (row0 >= step) row0 = 1 << 30;       // no whole row left for these threads
    }
};

template <typename KT>
__device__ __forceinline__ void load_keys(const GateAttn& A, const AttnSmem<KT>& sm, const KeyCopy& cp, int buf, int j, int j1, int tile) {
    constexpr int CN = Chunk16<KT>::n;
    const int rows = tile * A.kv_heads, valid = min(rows, (j1 - j) * A.kv_heads);
    KT* dst = sm.k + (size_t)buf * rows * sm.ks + cp.ch * CN;
    const KT* src = static_cast<const KT*>(A.cache) + (size_t)j * A.kv_heads * A.dim_s + cp.ch * CN;
    for (int r = cp.row0; r < rows; r += cp.step) {
        if (r < valid) cp_async16(dst + r * sm.ks, src + (size_t)r * A.dim_s);
        else *reinterpret_cast<uint4*>(dst + r * sm.ks) = make_uint4(0u, 0u, 0u, 0u);
    }
    for (int i = threadIdx.x; i < valid; i += kAttnThreads) cp_async4(sm.r + buf * rows + i, A.cache_r + (size_t)j * A.kv_heads + i);
}

// acc[q][pair] += sum over keys [j0, j1) of the mixed weights times the raw keys, for the NQ queries in
// sm.q at positions pos0 .. pos0 + NQ - 1.  Thread t owns elements 2 * (t + p * kAttnThreads) and the next of the
// [heads][dim_s] output.  A score belongs to one thread, lanes over heads.
template <typename KT, int NQ, int EP>
__device__ __forceinline__ void attend(const GateAttn& A, const AttnSmem<KT>& sm, int pos0, int j0, int j1, int tile,
                                       float (&acc)[NQ][EP][2]) {
    constexpr int CN = Chunk16<KT>::n;
    const int H = A.heads, DS = A.dim_s, KV = A.kv_heads, group = H / KV, row = KV * sm.ks;
    const int chunks = DS / CN;
    const int tsh = 31 - __clz(tile);               // tiles are powers of two
    const KeyCopy cp(chunks);
    int head_of[EP], key_of[EP];                    // this thread's output elements
#pragma unroll
    for (int e = 0; e < EP; e++) {
        const int el = 2 * (threadIdx.x + e * kAttnThreads);
        const int h = el / DS;
        head_of[e] = el < H * DS ? h : -1;
        key_of[e] = h / group * sm.ks + el - h * DS;
    }
    load_keys<KT>(A, sm, cp, 0, j0, j1, tile);
    cp_async_commit();
    int buf = 0;
    for (int j = j0; j < j1; j += tile, buf ^= 1) {
        if (j + tile < j1) load_keys<KT>(A, sm, cp, buf ^ 1, j + tile, j1, tile);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const KT* K = sm.k + (size_t)buf * tile * row;
        const float* R = sm.r + buf * tile * KV;
        const int keys = min(tile, j1 - j);
        for (int u = threadIdx.x; u < H * tile; u += kAttnThreads) {
            const int p = u / H, h = u - p * H, c = h / group;
            const KT* kp = K + p * row + c * sm.ks;
            const float* qp = sm.q + h * sm.qs;
            float dot[NQ][2] = {};
#pragma unroll 2
            for (int ch = 0; ch < chunks; ch++) {
                float kk[CN];
                Chunk16<KT>::load(kp + ch * CN, kk);
#pragma unroll
                for (int q = 0; q < NQ; q++)
#pragma unroll
                    for (int i = 0; i < CN; i += 4) {
                        const float4 v = *reinterpret_cast<const float4*>(qp + q * H * sm.qs + ch * CN + i);
                        dot[q][0] = fmaf(kk[i], v.x, dot[q][0]);
                        dot[q][1] = fmaf(kk[i + 1], v.y, dot[q][1]);
                        dot[q][0] = fmaf(kk[i + 2], v.z, dot[q][0]);
                        dot[q][1] = fmaf(kk[i + 3], v.w, dot[q][1]);
                    }
            }
            const float r = p < keys ? R[p * KV + c] : 0.f;
#pragma unroll
            for (int q = 0; q < NQ; q++) {
                const int dist = pos0 + q - (j + p);
                const float s = (dot[q][0] + dot[q][1]) * r - sm.slope[h] * (float)dist + sm.bias[h];
                sm.w[(q * H + h) * sm.ws + p] = dist >= 0 && p < keys ? sigmoid(s) : 0.f;
            }
        }
        __syncthreads();
        for (int u = threadIdx.x; u < NQ * H * tile; u += kAttnThreads) {
            const int p = u & (tile - 1), qh = u >> tsh, h = NQ == 1 ? qh : qh % H;
            const float* wq = sm.w + (qh - h) * sm.ws + p;
            const float* t = sm.talk + h * sm.ts;
            float v0 = 0.f, v1 = 0.f;
            int g = 0;
#pragma unroll 8
            for (; g + 1 < H; g += 2) {
                v0 = fmaf(t[g], wq[g * sm.ws], v0);
                v1 = fmaf(t[g + 1], wq[(g + 1) * sm.ws], v1);
            }
            if (g < H) v0 = fmaf(t[g], wq[g * sm.ws], v0);
            sm.mix[qh * sm.ws + p] = v0 + v1;
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < EP; e++) {
            const int h = head_of[e], off = key_of[e];
            if (h >= 0) {
#pragma unroll 8
                for (int p = 0; p < tile; p++) {
                    const float2 kv = pair_f32(K + p * row + off);
#pragma unroll
                    for (int q = 0; q < NQ; q++) {
                        const float m = sm.mix[(q * H + h) * sm.ws + p];
                        acc[q][e][0] = fmaf(m, kv.x, acc[q][e][0]);
                        acc[q][e][1] = fmaf(m, kv.y, acc[q][e][1]);
                    }
                }
            }
        }
        __syncthreads();
    }
}

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

// Launch with the programmatic attribute, so that the kernel may start under its predecessor's tail.
template <typename F, typename... Args>
inline cudaError_t launch_pdl(F kern, dim3 grid, int threads, size_t smem, bool pdl, cudaStream_t s, Args... args) {
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid;
    cfg.blockDim = dim3((unsigned)threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kern, args...);
}

}  // namespace mg
