// Device helpers shared by the ragged-batch kernel files: activation stores (f32 rows and / or bf16 planes), small async copies,
// KV page elements (f32, or bf16 with an optional low-order plane).
#pragma once

#include "ragged.cuh"

namespace cb {
namespace {

__device__ __forceinline__ void store_act(const ActOut& o, int r, int c, float v) {
    if (o.f) o.f[(size_t)r * o.ldf + c] = v;
    if (o.hi) {
        const bf16 h = __float2bfloat16_rn(v);
        bf16* p = o.hi + (size_t)r * o.ldb + c;
        *p = h;
        if (o.lo_off) p[o.lo_off] = __float2bfloat16_rn(v - __bfloat162float(h));
    }
}

// four neighbouring columns at once (c and the leading dimensions multiples of 4)
__device__ __forceinline__ void split4(const float* v, uint2& hi, uint2& lo) { split_bf16x2(v[0], v[1], hi.x, lo.x); split_bf16x2(v[2], v[3], hi.y, lo.y); }
__device__ __forceinline__ void store_act4(const ActOut& o, int r, int c, const float* v) {
    if (o.f) *reinterpret_cast<float4*>(o.f + (size_t)r * o.ldf + c) = make_float4(v[0], v[1], v[2], v[3]);
    if (o.hi) {
        uint2 hi, lo;
        split4(v, hi, lo);
        bf16* p = o.hi + (size_t)r * o.ldb + c;
        *reinterpret_cast<uint2*>(p) = hi;
        if (o.lo_off) *reinterpret_cast<uint2*>(p + o.lo_off) = lo;
    }
}

__device__ __forceinline__ void cp_async16s(void* smem_dst, const void* gsrc) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}
__device__ __forceinline__ void cp_async4(void* smem_dst, const void* gsrc) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}

// A short causal convolution over time that a warp walks row by row: NC * 32 channels starting at c0 (a lane owns c0 + lane + 32 i, i < NC,
// below c0 + width).  TAPS > 0: the tap window lives in registers; TAPS == 0: any number of taps, read back from memory.
struct ConvSrc {
    const float* in; int ld;          // [T, ld]
    const float* w;                   // [C, taps], last column on the current token
    float* state;                     // [slots, taps - 1, C] the inputs ahead of the step's rows
    int C, taps;
};
template <int NC, int TAPS>
struct ConvWalk {
    float w[NC][TAPS > 0 ? TAPS : 1], h[NC][TAPS > 1 ? TAPS - 1 : 1];
    int c0, width, lane, C;
    __device__ __forceinline__ void init(const ConvSrc& a, int c0_, int width_, int lane_) {
        c0 = c0_; width = width_; lane = lane_; C = a.C;
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int i = 0; i < NC; ++i) {
                const int c = lane + 32 * i;
#pragma unroll
                for (int k = 0; k < TAPS; ++k) w[i][k] = c < width ? a.w[(size_t)(c0 + c) * TAPS + k] : 0.f;
            }
        }
    }
    __device__ __forceinline__ float before(const ConvSrc& a, int slot, int in_entry, int r, int c, int k) const {      // what tap k of row r reads
        const int back = a.taps - 1 - k;
        return in_entry >= back ? a.in[(size_t)(r - back) * a.ld + c0 + c] : a.state[((size_t)slot * (a.taps - 1) + in_entry + k) * C + c0 + c];
    }
    __device__ __forceinline__ void refill(const ConvSrc& a, int slot, int in_entry, int r) {
        if constexpr (TAPS > 1) {
#pragma unroll
            for (int i = 0; i < NC; ++i) {
                const int c = lane + 32 * i;
#pragma unroll
                for (int k = 0; k < TAPS - 1; ++k) h[i][k] = c < width ? before(a, slot, in_entry, r, c, k) : 0.f;
            }
        }
    }
    // y[i] of row r from its own inputs x[i]; with `move` the carried window of the row's sequence moves on
    __device__ __forceinline__ void step(const ConvSrc& a, int slot, int in_entry, int r, const float* x, float* y, bool move) {
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const int c = lane + 32 * i;
            float acc = 0.f;
            if constexpr (TAPS > 0) {
#pragma unroll
                for (int k = 0; k < TAPS - 1; ++k) acc = fmaf(w[i][k], h[i][k], acc);
                acc = fmaf(w[i][TAPS - 1], x[i], acc);
                if (TAPS > 1) {
#pragma unroll
                    for (int k = 0; k < TAPS - 2; ++k) h[i][k] = h[i][k + 1];
                    h[i][TAPS - 2] = x[i];
                    if (move && c < width) {
#pragma unroll
                        for (int k = 0; k < TAPS - 1; ++k) a.state[((size_t)slot * (TAPS - 1) + k) * C + c0 + c] = h[i][k];
                    }
                }
            } else if (c < width) {
                for (int k = 0; k < a.taps - 1; ++k) acc = fmaf(a.w[(size_t)(c0 + c) * a.taps + k], before(a, slot, in_entry, r, c, k), acc);
                acc = fmaf(a.w[(size_t)(c0 + c) * a.taps + a.taps - 1], x[i], acc);
                if (move) {
                    float* win = a.state + (size_t)slot * (a.taps - 1) * C + c0 + c;
                    for (int k = 1; k < a.taps - 1; ++k) win[(size_t)(k - 1) * C] = win[(size_t)k * C];
                    win[(size_t)(a.taps - 2) * C] = x[i];
                }
            }
            y[i] = acc;
        }
    }
};

// KV page elements: f32, or bf16 with an optional low-order plane `lo` elements further on (x ~= hi + lo, ~16 mantissa bits)
template <typename KT> __device__ __forceinline__ float kv_load(const KT* p, long long lo);
template <> __device__ __forceinline__ float kv_load<float>(const float* p, long long) { return *p; }
template <> __device__ __forceinline__ float kv_load<bf16>(const bf16* p, long long lo) {
    const float h = __bfloat162float(*p);
    return lo ? h + __bfloat162float(p[lo]) : h;
}
template <typename KT> __device__ __forceinline__ void kv_store(KT* p, float v, long long lo);
template <> __device__ __forceinline__ void kv_store<float>(float* p, float v, long long) { *p = v; }
template <> __device__ __forceinline__ void kv_store<bf16>(bf16* p, float v, long long lo) {
    const bf16 h = __float2bfloat16_rn(v);
    *p = h;
    if (lo) p[lo] = __float2bfloat16_rn(v - __bfloat162float(h));
}

}  // namespace
}  // namespace cb
