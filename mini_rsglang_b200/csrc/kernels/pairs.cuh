// Two float32 in one 64-bit register pair: fma.rn.f32x2 and mul.rn.f32x2 are two independent float32 operations (each
// rounded like fmaf and *) in one instruction, so that work bound by instruction issue takes half the instructions.
#pragma once

typedef unsigned long long pair;         // two float32, the lower one in the lower half
__device__ __forceinline__ pair make_pair(float lo, float hi) {
    pair p;
    asm("mov.b64 %0, {%1, %2};" : "=l"(p) : "f"(lo), "f"(hi));
    return p;
}
__device__ __forceinline__ float2 split(pair p) {
    float2 f;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(p));
    return f;
}
__device__ __forceinline__ pair fma2(pair a, pair b, pair c) {
    pair d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ pair mul2(pair a, pair b) {
    pair d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ float both(pair p) {
    const float2 f = split(p);
    return f.x + f.y;
}
