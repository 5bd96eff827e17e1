// What the recurrences with a matrix of state a head share: a step's segments and where a segment's blocks of tokens lie, loads
// of 16 bytes as floats, products of two floats in one instruction, and the head norm with its gate behind a recurrence.
#pragma once

#include "common.cuh"

enum : int { KID_MATRIX_MEMORY = 100 };

struct MMSegment { int first, count, before, slot; };

__device__ __forceinline__ float mm_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float mm_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float mm_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float mm_logsigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
template <typename T> struct MMVec;
template <> struct MMVec<float> { static constexpr int N = 4; };
template <> struct MMVec<bf16> { static constexpr int N = 8; };

// 16 bytes at p (on a 16-byte boundary), times scale, as floats to shared memory (dst on a 16-byte boundary)
__device__ __forceinline__ void mm_fetch16(const float* p, float* dst, float scale) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    *reinterpret_cast<float4*>(dst) = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
}
__device__ __forceinline__ void mm_fetch16(const bf16* p, float* dst, float scale) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    *reinterpret_cast<float4*>(dst) = make_float4(__uint_as_float(r.x << 16) * scale, __uint_as_float(r.x & 0xffff0000u) * scale,
                                                  __uint_as_float(r.y << 16) * scale, __uint_as_float(r.y & 0xffff0000u) * scale);
    *reinterpret_cast<float4*>(dst + 4) = make_float4(__uint_as_float(r.z << 16) * scale, __uint_as_float(r.z & 0xffff0000u) * scale,
                                                      __uint_as_float(r.w << 16) * scale, __uint_as_float(r.w & 0xffff0000u) * scale);
}

// two float products, or multiply-adds, in one instruction
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 mm_pair(float x, float y) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};\n" : "=l"(r) : "f"(x), "f"(y));
    return r;
}
__device__ __forceinline__ float2 mm_unpair(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;\n" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 mm_mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ f32x2 mm_fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

// Block w of the step: the segments' blocks of L tokens one after the other.
struct MMBlock {
    int seg, tb, blocks;       // segment, which of its blocks, how many it has (seg -1: no such block)
    int rank;                  // its index among the blocks of segments of several blocks
};
__device__ __forceinline__ MMBlock mm_find_block(const MMSegment* __restrict__ segs, int n_segs, int w, int L) {
    const int lane = threadIdx.x & 31;
    int seen = 0, several = 0;
    for (int base = 0; base < n_segs; base += 32) {
        const int c = base + lane < n_segs ? segs[base + lane].count : 0;
        const int nb = c > 0 ? (c + L - 1) / L : 0, mb = nb > 1 ? nb : 0;
        int sum = nb, msum = mb;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int x = __shfl_up_sync(0xffffffffu, sum, o), y = __shfl_up_sync(0xffffffffu, msum, o);
            if (lane >= o) { sum += x; msum += y; }
        }
        const int first = seen + sum - nb;
        const unsigned hit = __ballot_sync(0xffffffffu, w >= first && w < first + nb);
        if (hit) {
            const int src = __ffs(hit) - 1;
            MMBlock b;
            b.seg = base + src;
            b.tb = w - __shfl_sync(0xffffffffu, first, src);
            b.blocks = __shfl_sync(0xffffffffu, nb, src);
            b.rank = several + __shfl_sync(0xffffffffu, msum - mb, src) + b.tb;
            return b;
        }
        seen += __shfl_sync(0xffffffffu, sum, 31);
        several += __shfl_sync(0xffffffffu, msum, 31);
    }
    MMBlock none;
    none.seg = -1; none.tb = none.blocks = none.rank = 0;
    return none;
}

// A warp a (token, head): o / rms(o) * gain * act(gate).  y float [tokens, H e]; gate: [tokens, g_stride] of the compute dtype;
// gain_per_head: the gain has H e entries, else e entries shared by the heads (null: no gain); kind 0 sigmoid, 1 silu.  With dn ([tokens, H, 2]:
// the normaliser's product with the query, exp(-m)) y holds numerators, and o = y / (max(|n . q|, exp(-m)) + 1e-6).
// N: entries a lane takes at a time (4 where rows are whole vectors of four, else 1).
__device__ __forceinline__ void head_quad_load(const float* p, float* v) {
    const float4 r = *reinterpret_cast<const float4*>(p);
    v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
}
__device__ __forceinline__ void head_quad_load(const bf16* p, float* v) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(r.x << 16); v[1] = __uint_as_float(r.x & 0xffff0000u);
    v[2] = __uint_as_float(r.y << 16); v[3] = __uint_as_float(r.y & 0xffff0000u);
}
__device__ __forceinline__ void head_quad_store(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void head_quad_store(bf16* p, const float* v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

template <typename T, int N>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* y, const float* __restrict__ dn, const T* gate, int g_stride,
                                                             const float* __restrict__ gain, T* __restrict__ out, long long n_rows,
                                                             int H, int E, int gain_per_head, int kind, float eps) {
    pdl_launch_dependents();
    pdl_wait(KID_MATRIX_MEMORY);
    const int lane = threadIdx.x & 31;
    const long long r = blockIdx.x * (long long)(blockDim.x >> 5) + (threadIdx.x >> 5);
    if (r >= n_rows) return;
    const long long t = r / H;
    const int h = (int)(r % H);
    const float* yr = y + r * E;
    const T* gr = gate + t * g_stride + (size_t)h * E;
    const float* gn = gain ? gain + (gain_per_head ? (size_t)h * E : 0) : nullptr;
    const float over = dn ? fmaxf(fabsf(dn[r * 2]), dn[r * 2 + 1]) + 1e-6f : 1.0f;
    constexpr int KEEP = N == 4 ? 4 : 8;          // rounds of a row that stay in registers
    float keep[KEEP][N];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < KEEP; j++) {
        const int i = (lane + 32 * j) * N;
        if (i >= E) break;
        if constexpr (N == 4) head_quad_load(yr + i, keep[j]); else keep[j][0] = yr[i];
#pragma unroll
        for (int k = 0; k < N; k++) { keep[j][k] /= over; ss += keep[j][k] * keep[j][k]; }
    }
    for (int i = (lane + 32 * KEEP) * N; i < E; i += 32 * N)
        for (int k = 0; k < N; k++) { const float v = yr[i + k] / over; ss += v * v; }
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)E + eps);
    auto finish = [&](int i, float* v) {
        float z[N], g[N];
        if constexpr (N == 4) {
            head_quad_load(gr + i, z);
            if (gn) head_quad_load(gn + i, g);
        } else {
            z[0] = to_f32(gr[i]);
            if (gn) g[0] = gn[i];
        }
#pragma unroll
        for (int k = 0; k < N; k++) {
            const float sg = mm_sigmoid(z[k]);
            v[k] = v[k] * inv * (gn ? g[k] : 1.0f) * (kind == 1 ? z[k] * sg : sg);
        }
        if constexpr (N == 4) head_quad_store(out + r * E + i, v); else out[r * E + i] = from_f32<T>(v[0]);
    };
#pragma unroll
    for (int j = 0; j < KEEP; j++) {
        const int i = (lane + 32 * j) * N;
        if (i >= E) break;
        finish(i, keep[j]);
    }
    for (int i = (lane + 32 * KEEP) * N; i < E; i += 32 * N) {
        float v[N];
        for (int k = 0; k < N; k++) v[k] = yr[i + k] / over;
        finish(i, v);
    }
}

template <typename T>
static void launch_head_norm_gate(const float* y, const float* dn, const void* gate, int g_stride, const float* gain, void* out, int n_tokens, int H, int E,
                                  int gain_per_head, int kind, float eps, cudaStream_t stream) {
    const long long rows = (long long)n_tokens * H;
    const bool quads = E % 4 == 0 && g_stride % 4 == 0 && (((uintptr_t)y | (uintptr_t)gain | (uintptr_t)out) & 15) == 0 &&
                       ((uintptr_t)gate & (4 * sizeof(T) - 1)) == 0;
    const dim3 grid((unsigned)((rows + 7) / 8));
    if (quads)
        launch_chained(head_norm_gate_kernel<T, 4>, grid, dim3(256), 0, stream, y, dn, (const T*)gate, g_stride, gain, (T*)out, rows, H, E,
                       gain_per_head, kind, eps);
    else
        launch_chained(head_norm_gate_kernel<T, 1>, grid, dim3(256), 0, stream, y, dn, (const T*)gate, g_stride, gain, (T*)out, rows, H, E,
                       gain_per_head, kind, eps);
}
