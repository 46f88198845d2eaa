// What the attention kernels over pages with key and value sizes of their own share: the dot product
// of the generic forms, the fragments, copies and packing of the mma.sync forms, and the rule that
// shapes their launches.
#pragma once

#include "common.cuh"

#include <float.h>

constexpr int kMmaRows = 64, kMmaKeys = 64;
constexpr int kMaxParts = 8;           // blocks that may share a row tile's keys

template <typename T>
__device__ __forceinline__ float dv_dot(const float* __restrict__ q, const T* __restrict__ k, int n, bool vec) {
    float s = 0.f;
    if (vec) {
        if constexpr (sizeof(T) == 4) {
            for (int d = 0; d < n; d += 4) {
                const float4 kv = *reinterpret_cast<const float4*>(k + d);
                s += q[d] * kv.x + q[d + 1] * kv.y + q[d + 2] * kv.z + q[d + 3] * kv.w;
            }
        } else {
            for (int d = 0; d < n; d += 8) {
                const uint4 raw = *reinterpret_cast<const uint4*>(k + d);
                const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float2 f = __bfloat1622float2(p[j]);
                    s += q[d + 2 * j] * f.x + q[d + 2 * j + 1] * f.y;
                }
            }
        }
    } else {
        for (int d = 0; d < n; ++d) s += q[d] * lsb_to_float(k[d]);
    }
    return s;
}

__device__ __forceinline__ void dv_mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void dv_cp_async16(void* dst, const void* src, bool real) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    const int n = real ? 16 : 0;                       // 0: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ uint32_t dv_pack(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}

// How a step of this shape is launched: bit 0: 16-row blocks; bit 1: four tiles in flight; bits 8..:
// how many blocks share a row tile's keys.  A function of the shape alone (never of the sequences'
// lengths), so that a captured launch stays valid as sequences grow.  shape: 0 chooses; 1: 64-row
// blocks; 2: 16-row blocks, two tiles in flight; 3: 16-row blocks, four; 4: as 3, keys shared by 3 blocks.
static inline int dv_mma_plan(int n_requests, int max_q_len, int nh, int nkv, int chunk, int sms, int shape) {
    if (sms <= 0) sms = 148;
    const long long rows = (long long)max_q_len * (nh / nkv);
    const long long thin = (rows + 15) / 16 * nkv * n_requests;
    // (16-row blocks for prompt portions were measured too: with the grid small they gain nothing over
    // 64-row blocks, 56 against 49 us for one prompt of 2,048 tokens and four heads, and lose at any size
    // that fills the chip, since every block loads whole tiles for a quarter of the arithmetic)
    const int narrow = shape == 1 ? 0 : shape >= 2 ? 1 : rows <= 16 ? 1 : 0;
    const int deep = (shape >= 3 || (shape == 0 && narrow && thin <= 2 * sms)) ? 1 : 0;
    long long ksplit = 1;
    if (shape == 4) ksplit = 3;
    else if (shape == 0 && narrow) {
        ksplit = (2 * sms) / thin;
        if (ksplit > kMaxParts) ksplit = kMaxParts;
        if (chunk > 0 && ksplit > (chunk + kMmaKeys - 1) / kMmaKeys) ksplit = (chunk + kMmaKeys - 1) / kMmaKeys;
        if (ksplit < 1) ksplit = 1;
    }
    return narrow | (deep << 1) | ((int)ksplit << 8);
}
