// What the scan kernels share: a block owns one (sequence, head, slice of SCAN_VS value columns) and walks the
// sequence's tokens of the step in order; P lanes share one value column and hold R of its keys each in registers.
// Included by the files that have a scan; each walks a recurrence of its own (recurrent.cu says what P and R follow).
#pragma once
#include "common.cuh"
#include <math.h>

__device__ __forceinline__ float rc_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float rc_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float rc_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// Tokens staged in shared memory at a time: 32 (16 for the widest keys, to stay inside 48 KB).  A chunk costs one
// round trip to global memory that nothing hides when a block has its SM to itself (one long prompt), so the
// chunk is as long as shared memory allows; the results do not depend on it.
#define SCAN_TC(DP) ((DP) <= 128 ? 32 : 16)
#define SCAN_VS 32           // value columns per block; a block has 32 P threads

// Where a sequence's rows are: from `spans` [n_seq, 3] = {slot, first row, rows}, or, without spans, sequence
// i is row i alone (a decode step: the slot comes from tok_slot).
__device__ __forceinline__ void scan_span(const int* __restrict__ spans, const int* __restrict__ tok_slot, int seq,
                                          int& slot, int& start, int& len) {
    if (spans) { slot = spans[3 * seq]; start = spans[3 * seq + 1]; len = spans[3 * seq + 2]; }
    else { slot = tok_slot[seq]; start = seq; len = 1; }
}

// A thread's R state values: register e = 4 i + w holds key (P i + part) * 4 + w of its value column.
#define KEY_OF(i, part) (((i) * P + (part)) * 4)

template <int R, int P>
__device__ __forceinline__ void scan_load_state(float (&S)[R], const float* __restrict__ st, int part) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const float4 v = *reinterpret_cast<const float4*>(st + KEY_OF(i, part));
        S[4 * i] = v.x; S[4 * i + 1] = v.y; S[4 * i + 2] = v.z; S[4 * i + 3] = v.w;
    }
}
template <int R, int P>
__device__ __forceinline__ void scan_store_state(const float (&S)[R], float* __restrict__ st, int part) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i)
        *reinterpret_cast<float4*>(st + KEY_OF(i, part)) = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
}
template <int P>
__device__ __forceinline__ float part_sum(float v) {               // over the P lanes of one value column
#pragma unroll
    for (int o = 1; o < P; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// The padded key dimension for d: 16, 32, 64, 128 or 256 (0: too large).
static int scan_padded(int d) {
    for (int dp = 16; dp <= 256; dp *= 2)
        if (dp >= d) return dp;
    return 0;
}

// (registers, lanes per column) by padded key dimension: 16 -> (4, 4), 32 -> (8, 4), 64 -> (8, 8), 128 -> (16, 8),
// 256 -> (32, 8)
#define SCAN_DISPATCH_X(KERNEL, TT, X, ...)                                                              \
    switch (DP) {                                                                                        \
        case 16:  gi_launch(KERNEL<TT, 4, 4 X>, grid, dim3(SCAN_VS * 4), 0, s, __VA_ARGS__); break;      \
        case 32:  gi_launch(KERNEL<TT, 8, 4 X>, grid, dim3(SCAN_VS * 4), 0, s, __VA_ARGS__); break;      \
        case 64:  gi_launch(KERNEL<TT, 8, 8 X>, grid, dim3(SCAN_VS * 8), 0, s, __VA_ARGS__); break;      \
        case 128: gi_launch(KERNEL<TT, 16, 8 X>, grid, dim3(SCAN_VS * 8), 0, s, __VA_ARGS__); break;     \
        default:  gi_launch(KERNEL<TT, 32, 8 X>, grid, dim3(SCAN_VS * 8), 0, s, __VA_ARGS__); break;     \
    }
#define SCAN_NOTHING
#define SCAN_COMMA(v) , v
#define SCAN_DISPATCH(KERNEL, TT, ...) SCAN_DISPATCH_X(KERNEL, TT, SCAN_NOTHING, __VA_ARGS__)
// The same sizes for kernels that are launched by a macro LAUNCH(T, registers, lanes).
#define SCAN_SIZES(LAUNCH, TT)                         \
    switch (DP) {                                      \
        case 16:  LAUNCH(TT, 4, 4); break;             \
        case 32:  LAUNCH(TT, 8, 4); break;             \
        case 64:  LAUNCH(TT, 8, 8); break;             \
        case 128: LAUNCH(TT, 16, 8); break;            \
        default:  LAUNCH(TT, 32, 8); break;            \
    }

// Four neighbouring inputs as they lie in memory: kept raw in registers while a chunk is walked, so that nothing waits
// for the load before the next chunk is staged.
template <typename T> struct Raw4;
template <> struct Raw4<float> { typedef float4 type; };
template <> struct Raw4<bf16> { typedef uint2 type; };
__device__ __forceinline__ float4 raw4_f32(const float4& v) { return v; }
__device__ __forceinline__ float4 raw4_f32(const uint2& v) {
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
// The loads stay where they are written (ahead of a chunk's walk), and what is done with their values stays behind
// raw_arrived: a conversion that the compiler moves up to its load waits for it there.
__device__ __forceinline__ void raw4_load(float4& v, const float* p) {
    asm volatile("ld.global.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "l"(p));
}
__device__ __forceinline__ void raw4_load(uint2& v, const bf16* p) {
    asm volatile("ld.global.v2.u32 {%0, %1}, [%2];" : "=r"(v.x), "=r"(v.y) : "l"(p));
}
__device__ __forceinline__ void raw_arrived(float4& v) { asm volatile("" : "+f"(v.x), "+f"(v.y), "+f"(v.z), "+f"(v.w)); }
__device__ __forceinline__ void raw_arrived(uint2& v) { asm volatile("" : "+r"(v.x), "+r"(v.y)); }
__device__ __forceinline__ void raw_arrived(uint32_t& v) { asm volatile("" : "+r"(v)); }
__device__ __forceinline__ void raw4_zero(float4& v) { v = make_float4(0.f, 0.f, 0.f, 0.f); }
__device__ __forceinline__ void raw4_zero(uint2& v) { v = make_uint2(0u, 0u); }
// One input kept raw: a 16-bit value in a whole register of its own (two of them packed into one would wait for both loads).
__device__ __forceinline__ uint32_t raw1_load(const bf16* p) {
    uint32_t v;
    asm volatile("ld.global.u16 %0, [%1];" : "=r"(v) : "l"(p));
    return v;
}
__device__ __forceinline__ uint32_t raw1_load(const float* p) {
    uint32_t v;
    asm volatile("ld.global.u32 %0, [%1];" : "=r"(v) : "l"(p));
    return v;
}
template <typename T> __device__ __forceinline__ float raw1_f32(uint32_t v) { return __uint_as_float(sizeof(T) == 2 ? v << 16 : v); }

// P tokens' partial sums of a value column, one set per lane of its P lanes -> the whole sum of token `part` in lane
// `part`: P - 1 shuffles instead of P log2(P).  Every sum is the tree of part_sum (neighbours 1, 2, 4 apart), so a
// token has the same bits whichever of the two took it.
template <int P>
__device__ __forceinline__ float part_sum_tokens(float (&v)[P], int part) {
#pragma unroll
    for (int o = 1, n = P; o < P; o <<= 1, n >>= 1) {
        const bool up = part & o;
#pragma unroll
        for (int j = 0; j < n / 2; ++j) {
            const float keep = up ? v[2 * j + 1] : v[2 * j], send = up ? v[2 * j] : v[2 * j + 1];
            v[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
    return v[0];
}

// Pairs of floats as one 64-bit register pair: one instruction for both (each half rounded like fmaf and the product).
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 both2(float x) {
    f32x2 d;
    asm("mov.b64 %0, {%1, %1};" : "=l"(d) : "f"(x));
    return d;
}
__device__ __forceinline__ float sum2(f32x2 a, f32x2 b) {          // (a.x + a.y) + (b.x + b.y)
    float ax, ay, bx, by;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(ax), "=f"(ay) : "l"(a));
    asm("mov.b64 {%0, %1}, %2;" : "=f"(bx), "=f"(by) : "l"(b));
    return (ax + ay) + (bx + by);
}
// Two value columns to a thread (SCAN_HALF apart), the keys as above in pairs: what a lane reads of a
// token's keys from shared memory then serves two columns.
template <int R, int P>
__device__ __forceinline__ void scan_load_pairs(f32x2 (&S)[R / 2], const float* __restrict__ st, int part, bool live) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        ulonglong2 v = make_ulonglong2(0ull, 0ull);
        if (live) v = *reinterpret_cast<const ulonglong2*>(st + KEY_OF(i, part));
        S[2 * i] = v.x; S[2 * i + 1] = v.y;
    }
}
template <int R, int P>
__device__ __forceinline__ void scan_store_pairs(const f32x2 (&S)[R / 2], float* __restrict__ st, int part) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i)
        *reinterpret_cast<ulonglong2*>(st + KEY_OF(i, part)) = make_ulonglong2(S[2 * i], S[2 * i + 1]);
}
#define SCAN_HALF (SCAN_VS / 2)
#define SCAN_O_LD 36         // row length of the staged outputs: the lanes of part_sum_tokens write without bank conflicts
