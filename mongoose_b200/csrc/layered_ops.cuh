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
__device__ __forceinline__ void norm_queries(const GateAttn& A, const float* q, float temp, float* out) {
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
            if (d < A.dim_s) out[h * A.dim_s + d] = d < A.dim ? v[i] * r * A.q_norm[d] * A.k_norm[d] : 0.f;
        }
        for (int d = sub + 128; d < A.dim_s; d += 8) out[h * A.dim_s + d] = d < A.dim ? p[d] * r * A.q_norm[d] * A.k_norm[d] : 0.f;
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
    const int pairs = (at.heads * at.dim_s / 2 + kAttnThreads - 1) / kAttnThreads;
    for (int p = 1; p <= 16; p *= 2)
        if (pairs <= p) return p;
    return 0;
}

template <typename KT>
struct AttnSmem {
    KT* k;          // [2][tile][kv_heads * dim_s]
    float* r;       // [2][tile][kv_heads]
    float* q;       // [nq][heads][dim_s]
    float* w;       // [nq][heads][tile] sigmoid weights
    float* mix;     // [nq][heads][tile] mixed over heads
    float *talk, *bias, *slope;
    __device__ __forceinline__ AttnSmem(const GateAttn& A, int nq, int tile, float* base) {
        k = reinterpret_cast<KT*>(base);
        r = reinterpret_cast<float*>(k + 2 * (size_t)tile * A.kv_heads * A.dim_s);
        q = r + pad_to(2 * tile * A.kv_heads, 4);
        w = q + nq * A.heads * A.dim_s;
        mix = w + nq * A.heads * tile;
        talk = mix + nq * A.heads * tile;
        bias = talk + A.heads * A.heads;
        slope = bias + A.heads;
    }
    __device__ __forceinline__ void load_tables(const GateAttn& A) const {
        for (int i = threadIdx.x; i < A.heads * A.heads; i += kAttnThreads) talk[i] = A.talk[i];
        for (int i = threadIdx.x; i < A.heads; i += kAttnThreads) { bias[i] = A.head_bias[i]; slope[i] = A.slopes[i]; }
    }
};

// Bytes of AttnSmem with the largest tile of at most `most` (32, 16 or 8) keys that fits; 0 when none does.
inline size_t attn_smem(const GateAttn& at, int nq, int kt_bytes, int most, int* tile) {
    if (!attn_pairs(at)) return 0;
    for (int t = most; t >= 8; t /= 2) {
        const size_t b = 2 * (size_t)t * at.kv_heads * at.dim_s * kt_bytes +
                         ((size_t)pad_to(2 * t * at.kv_heads, 4) + (size_t)nq * at.heads * (at.dim_s + 2 * t) +
                          (size_t)at.heads * at.heads + 2 * at.heads) * sizeof(float);
        if (b <= 200 * 1024) { *tile = t; return b; }
    }
    return 0;
}

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

template <typename KT>
__device__ __forceinline__ void load_keys(const GateAttn& A, const AttnSmem<KT>& sm, int buf, int j, int j1, int tile) {
    const int row = A.kv_heads * A.dim_s, per = row * (int)sizeof(KT) / 16;
    KT* dst = sm.k + (size_t)buf * tile * row;
    const KT* src = static_cast<const KT*>(A.cache) + (size_t)j * row;
    const int valid = (j1 - j < tile ? j1 - j : tile) * per;
    for (int i = threadIdx.x; i < tile * per; i += kAttnThreads) {
        void* d = reinterpret_cast<uint4*>(dst) + i;
        if (i < valid) cp_async16(d, reinterpret_cast<const uint4*>(src) + i);
        else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
    for (int i = threadIdx.x; i < tile * A.kv_heads; i += kAttnThreads)
        sm.r[buf * tile * A.kv_heads + i] = j + i / A.kv_heads < j1 ? A.cache_r[(size_t)j * A.kv_heads + i] : 0.f;
}

// acc[q][pair] += sum over keys [j0, j1) of the mixed weights times the raw keys, for the NQ queries in
// sm.q at positions pos0 .. pos0 + NQ - 1.  Thread t owns elements 2 * (t + p * kAttnThreads) and the next of the
// [heads][dim_s] output.
template <typename KT, int NQ, int EP>
__device__ __forceinline__ void attend(const GateAttn& A, const AttnSmem<KT>& sm, int pos0, int j0, int j1, int tile,
                                       float (&acc)[NQ][EP][2]) {
    constexpr int CN = Chunk16<KT>::n;
    const int H = A.heads, DS = A.dim_s, row = A.kv_heads * DS, group = H / A.kv_heads;
    const int sub = threadIdx.x & 7, gid = threadIdx.x >> 3;
    const int chunks = DS / CN;
    const int ts = 31 - __clz(tile);                // tiles are powers of two
    int head_of[EP], key_of[EP];                    // this thread's output elements
#pragma unroll
    for (int e = 0; e < EP; e++) {
        const int el = 2 * (threadIdx.x + e * kAttnThreads);
        const int h = el / DS;
        head_of[e] = el < H * DS ? h : -1;
        key_of[e] = h / group * DS + el - h * DS;
    }
    load_keys<KT>(A, sm, 0, j0, j1, tile);
    cp_async_commit();
    int buf = 0;
    for (int j = j0; j < j1; j += tile, buf ^= 1) {
        if (j + tile < j1) load_keys<KT>(A, sm, buf ^ 1, j + tile, j1, tile);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const KT* K = sm.k + (size_t)buf * tile * row;
        const float* R = sm.r + buf * tile * A.kv_heads;
        for (int u = gid; u < H * tile; u += kAttnThreads / 8) {
            const int h = u >> ts, p = u & (tile - 1), c = h / group;
            const KT* kp = K + (size_t)p * row + c * DS;
            float dot[NQ] = {};
            for (int ch = sub; ch < chunks; ch += 8) {
                float kk[CN];
                Chunk16<KT>::load(kp + ch * CN, kk);
#pragma unroll
                for (int q = 0; q < NQ; q++) {
                    const float* qp = sm.q + (q * H + h) * DS + ch * CN;
#pragma unroll
                    for (int i = 0; i < CN; i += 4) {
                        const float4 v = *reinterpret_cast<const float4*>(qp + i);
                        dot[q] = fmaf(kk[i], v.x, fmaf(kk[i + 1], v.y, fmaf(kk[i + 2], v.z, fmaf(kk[i + 3], v.w, dot[q]))));
                    }
                }
            }
            float mine = 0.f;
#pragma unroll
            for (int q = 0; q < NQ; q++) {
                float d = dot[q];
                d += __shfl_xor_sync(0xffu << (threadIdx.x & 24), d, 1);
                d += __shfl_xor_sync(0xffu << (threadIdx.x & 24), d, 2);
                d += __shfl_xor_sync(0xffu << (threadIdx.x & 24), d, 4);
                if (sub == q) mine = d;
            }
            if (sub < NQ) {
                const int dist = pos0 + sub - (j + p);
                const float s = mine * R[p * A.kv_heads + c] - sm.slope[h] * (float)dist + sm.bias[h];
                sm.w[(sub * H + h) * tile + p] = dist >= 0 && j + p < j1 ? sigmoid(s) : 0.f;
            }
        }
        __syncthreads();
        for (int u = threadIdx.x; u < NQ * H * tile; u += kAttnThreads) {
            const int p = u & (tile - 1), qh = u >> ts, h = NQ == 1 ? qh : qh % H;
            const float* wq = sm.w + (qh - h) * tile + p;
            const float* t = sm.talk + h * H;
            float v0 = 0.f, v1 = 0.f;
            int g = 0;
#pragma unroll 4
            for (; g + 1 < H; g += 2) {
                v0 = fmaf(t[g], wq[g * tile], v0);
                v1 = fmaf(t[g + 1], wq[(g + 1) * tile], v1);
            }
            if (g < H) v0 = fmaf(t[g], wq[g * tile], v0);
            sm.mix[u] = v0 + v1;
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < EP; e++) {
            const int h = head_of[e], off = key_of[e];
            if (h >= 0) {
#pragma unroll 8
                for (int p = 0; p < tile; p++) {
                    const float2 kv = pair_f32(K + (size_t)p * row + off);
#pragma unroll
                    for (int q = 0; q < NQ; q++) {
                        const float m = sm.mix[(q * H + h) * tile + p];
                        acc[q][e][0] = fmaf(m, kv.x, acc[q][e][0]);
                        acc[q][e][1] = fmaf(m, kv.y, acc[q][e][1]);
                    }
                }
            }
        }
        __syncthreads();
    }
}

}  // namespace mg
