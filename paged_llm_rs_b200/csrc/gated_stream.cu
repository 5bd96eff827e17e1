// A float stream whose sublayers sit side by side: both read the same x, each through a norm of its own, each result is
// multiplied entry by entry by a sigmoid gate before it is added, and the mixer's input is shifted by a token.
//
//   gated_sum_norm32   everything between one layer's products and the next layer's, in one pass over the stream:
//                          x' = x + sigmoid(ga + ba) (s1 a1 + s2 a2) + sigmoid(gf + bf) f + embedded + vector
//                      (each term may be absent; x' is stored to a tensor of its own, x stays as it is), then
//                          h1 = norm(x') gain1         y1 = h1          (the gates' input, or the model's last norm)
//                          ys = h1 + (h1 of the token before - h1) shift     (the mixer's input)
//                          y2 = norm(x') gain2                          (the feed-forward's input)
//                      The token before a segment's first lies in the request's state slot (zeros at the start), which then
//                      takes the segment's last h1: both by the CTA of the segment's first token, so that nobody reads what
//                      another CTA has already replaced.  A CTA takes a run of rows and forms the row before its first again
//                      rather than wait for the CTA that has it.
//   poly_norm          y = a N(u) + b N(u^2) + c N(u^3) + e, N(z) = z / sqrt(mean(z^2) + eps) over a row, powers entry by entry
//   softcap32          x = cap tanh(x / cap)
//   add_terms_norm32   x += c1 d1 + c2 d2 + c3 d3 (in place; terms may be absent), y = norm(x): the root mean square's or, with
//                      the mean taken off first, a layer norm with a bias.  What a block does whose sublayers read ONE norm.
//
// Norms, gates, sums and the shift are float whatever the compute dtype; each output is rounded once.
#include "matrix_memory.cuh"

enum : int { KID_GATED_STREAM = 130 };

// what is added to the stream; values are rows of the compute dtype with strides in elements
struct GatedSum {
    const float* x;
    const void *a1, *a2, *ga, *f, *gf;
    const float *ba, *bf, *embedded, *vector;
    float s1, s2;
    int a1_stride, a2_stride, ga_stride, f_stride, gf_stride;
};

template <typename T, int N> __device__ __forceinline__ void gs_load(const T* p, float* v) {
    if constexpr (N == 1) {
        v[0] = to_f32(p[0]);
    } else {
        Vec16<T> r;
        r.load(p); r.unpack(v);
    }
}
template <typename T, int N> __device__ __forceinline__ void gs_store(T* p, const float* v) {
    if constexpr (N == 1) {
        p[0] = from_f32<T>(v[0]);
    } else {
        Vec16<T> r;
        r.pack(v); r.store(p);
    }
}
template <int N> __device__ __forceinline__ void gs_load32(const float* p, float* v) {
    if constexpr (N == 1) {
        v[0] = p[0];
    } else {
#pragma unroll
        for (int k = 0; k < N; k += 4) {
            const float4 r = *reinterpret_cast<const float4*>(p + k);
            v[k] = r.x; v[k + 1] = r.y; v[k + 2] = r.z; v[k + 3] = r.w;
        }
    }
}
template <int N> __device__ __forceinline__ void gs_store32(float* p, const float* v) {
    if constexpr (N == 1) {
        p[0] = v[0];
    } else {
#pragma unroll
        for (int k = 0; k < N; k += 4) *reinterpret_cast<float4*>(p + k) = make_float4(v[k], v[k + 1], v[k + 2], v[k + 3]);
    }
}

// N entries of row r from column c on, summed
template <typename T, int N>
__device__ __forceinline__ void gs_form(const GatedSum& g, size_t r, int width, int c, float* v) {
    float t[N], z[N];
    gs_load32<N>(g.x + r * width + c, v);
    if (g.a1) {
        float a[N];
        gs_load<T, N>((const T*)g.a1 + r * g.a1_stride + c, a);
        if (g.ga) gs_load<T, N>((const T*)g.ga + r * g.ga_stride + c, z);
        if (g.a2) {
            gs_load<T, N>((const T*)g.a2 + r * g.a2_stride + c, t);
#pragma unroll
            for (int k = 0; k < N; k++) a[k] = g.s1 * a[k] + g.s2 * t[k];
        } else {
#pragma unroll
            for (int k = 0; k < N; k++) a[k] *= g.s1;
        }
        if (g.ga) {
            gs_load32<N>(g.ba + c, t);
#pragma unroll
            for (int k = 0; k < N; k++) a[k] *= mm_sigmoid(z[k] + t[k]);
        }
#pragma unroll
        for (int k = 0; k < N; k++) v[k] += a[k];
    }
    if (g.f) {
        float f[N];
        gs_load<T, N>((const T*)g.f + r * g.f_stride + c, f);
        if (g.gf) {
            gs_load<T, N>((const T*)g.gf + r * g.gf_stride + c, z);
            gs_load32<N>(g.bf + c, t);
#pragma unroll
            for (int k = 0; k < N; k++) f[k] *= mm_sigmoid(z[k] + t[k]);
        }
#pragma unroll
        for (int k = 0; k < N; k++) v[k] += f[k];
    }
    if (g.embedded) {
        gs_load32<N>(g.embedded + r * width + c, t);
#pragma unroll
        for (int k = 0; k < N; k++) v[k] += t[k];
    }
    if (g.vector) {
        gs_load32<N>(g.vector + c, t);
#pragma unroll
        for (int k = 0; k < N; k++) v[k] += t[k];
    }
}

// the segment that row r is in, -1: none (a captured step's padding)
__device__ __forceinline__ int gs_segment(const MMSegment* __restrict__ segs, int n_segs, int r) {
    int hit = -1;
    for (int i = threadIdx.x & 31; i < n_segs; i += 32) {
        const MMSegment s = segs[i];
        if (r >= s.first && r < s.first + s.count) hit = i;
    }
    return __reduce_max_sync(0xffffffffu, hit);
}

// One CTA: `run` rows one after the other; a thread has the same entries of every row (N at a time), kept in shared memory:
// cur the row's h1 (first its sum), before the h1 of the token before.
template <typename T, int N>
__global__ void __launch_bounds__(512) gated_sum_norm32_kernel(GatedSum g, float* __restrict__ x_out, const float* __restrict__ gain1,
                                                               T* __restrict__ y1, const float* __restrict__ shift, T* __restrict__ ys,
                                                               const float* __restrict__ gain2, T* __restrict__ y2,
                                                               const MMSegment* __restrict__ segs, int n_segs, float* state,
                                                               long long state_stride, const int* __restrict__ rows, int n_rows, int width,
                                                               float eps, int run) {
    extern __shared__ __align__(16) float gs_smem[];
    __shared__ float scratch[32];
    float* cur = gs_smem;
    float* before = gs_smem + width;
    const int stride = blockDim.x * N, c0 = threadIdx.x * N;
    pdl_launch_dependents();
    pdl_wait(KID_GATED_STREAM);
    // h1 of row r into buf
    auto normed = [&](size_t r, float* buf) {
        float ss = 0.f;
        for (int c = c0; c < width; c += stride) {
            float v[N];
            gs_form<T, N>(g, r, width, c, v);
#pragma unroll
            for (int k = 0; k < N; k++) ss = fmaf(v[k], v[k], ss);
            gs_store32<N>(buf + c, v);
        }
        ss = block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / (float)width + eps);
        for (int c = c0; c < width; c += stride) {
            float v[N], w[N];
            gs_load32<N>(buf + c, v);
            gs_load32<N>(gain1 + c, w);
#pragma unroll
            for (int k = 0; k < N; k++) v[k] = v[k] * inv * w[k];
            gs_store32<N>(buf + c, v);
        }
    };
    const int i0 = blockIdx.x * run, i1 = min(n_rows, i0 + run);
    for (int i = i0; i < i1; i++) {
        const size_t r = rows ? (size_t)rows[i] : (size_t)i;
        int si = -1;
        MMSegment s = {0, 0, 0, 0};
        bool first = false;
        if (ys) {
            si = gs_segment(segs, n_segs, i);
            if (si >= 0) s = segs[si];
            first = si >= 0 && i == s.first;
            if (si < 0 || (first && s.before <= 0)) {
                for (int c = c0; c < width; c += stride)
#pragma unroll
                    for (int k = 0; k < N; k++) before[c + k] = 0.f;
            } else if (first) {
                const float* st = state + (size_t)s.slot * state_stride;
                for (int c = c0; c < width; c += stride) {
                    float v[N];
                    gs_load32<N>(st + c, v);
                    gs_store32<N>(before + c, v);
                }
            } else if (i == i0) {
                normed((size_t)i - 1, before);
            }
        }
        float ss = 0.f;
        for (int c = c0; c < width; c += stride) {
            float v[N];
            gs_form<T, N>(g, r, width, c, v);
#pragma unroll
            for (int k = 0; k < N; k++) ss = fmaf(v[k], v[k], ss);
            if (x_out) gs_store32<N>(x_out + r * width + c, v);
            gs_store32<N>(cur + c, v);
        }
        ss = block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / (float)width + eps);
        for (int c = c0; c < width; c += stride) {
            float v[N], w[N], h[N], o[N];
            gs_load32<N>(cur + c, v);
            gs_load32<N>(gain1 + c, w);
#pragma unroll
            for (int k = 0; k < N; k++) { v[k] *= inv; h[k] = v[k] * w[k]; }
            gs_store<T, N>(y1 + (size_t)i * width + c, h);
            if (y2) {
                gs_load32<N>(gain2 + c, w);
#pragma unroll
                for (int k = 0; k < N; k++) o[k] = v[k] * w[k];
                gs_store<T, N>(y2 + (size_t)i * width + c, o);
            }
            if (ys) {
                float b[N];
                gs_load32<N>(before + c, b);
                gs_load32<N>(shift + c, w);
#pragma unroll
                for (int k = 0; k < N; k++) o[k] = h[k] + (b[k] - h[k]) * w[k];
                gs_store<T, N>(ys + (size_t)i * width + c, o);
                gs_store32<N>(cur + c, h);
            }
        }
        if (ys) {
            if (first) {
                // (the slot was read above, by the same threads)
                if (s.count > 1) normed((size_t)s.first + s.count - 1, before);
                const float* last = s.count > 1 ? before : cur;
                float* st = state + (size_t)s.slot * state_stride;
                for (int c = c0; c < width; c += stride) {
                    float v[N];
                    gs_load32<N>(last + c, v);
                    gs_store32<N>(st + c, v);
                }
            }
            float* swap = cur; cur = before; before = swap;
        }
    }
}

// (gate, value) strides in elements.  With `rows` (n_rows of them) only those rows are formed and normed, into row i of y1;
// then neither x_out, ys nor y2 may be asked for.
PLLM_EXPORT int pllm_gated_sum_norm32(int dtype, const float* x, const void* a1, int a1_stride, float s1, const void* a2, int a2_stride, float s2,
                                      const void* ga, int ga_stride, const float* ba, const void* f, int f_stride, const void* gf,
                                      int gf_stride, const float* bf, const float* embedded, const float* vector, float* x_out,
                                      const float* gain1, void* y1, const float* shift, void* ys, const float* gain2, void* y2,
                                      const int* segs, int n_segs, float* state, long long state_stride, const int* rows, int n_rows,
                                      int width, float eps, cudaStream_t stream) {
    if (n_rows <= 0) return PLLM_OK;
    if (width <= 0 || !x || !gain1 || !y1 || (a2 && !a1) || (ga && (!ba || !a1)) || (gf && (!bf || !f)) || (y2 && !gain2)) return PLLM_ERR_SIZE;
    if (rows && (x_out || ys || y2)) return PLLM_ERR_SIZE;
    if (ys && (!shift || !segs || n_segs <= 0 || !state || state_stride < width)) return PLLM_ERR_SIZE;
    if (x_out == x) return PLLM_ERR_SIZE;          // (a row's neighbour is formed from the old stream)
    GatedSum g = {x, a1, a2, ga, f, gf, ba, bf, embedded, vector, s1, s2, a1_stride, a2_stride, ga_stride, f_stride, gf_stride};
    const size_t smem = (size_t)2 * width * sizeof(float);
    if (smem > 200 * 1024) return PLLM_ERR_LIMIT;
    PLLM_DISPATCH_DTYPE(dtype, {
        constexpr int V = Vec16<T>::N;
        uintptr_t p = 0;
        for (const void* q : {(const void*)x, a1, a2, ga, f, gf, (const void*)ba, (const void*)bf, (const void*)embedded, (const void*)vector,
                              (const void*)x_out, (const void*)gain1, (const void*)y1, (const void*)shift, (const void*)ys, (const void*)gain2,
                              (const void*)y2, (const void*)state}) p |= (uintptr_t)q;
        const bool vec = width % V == 0 && (p & 15) == 0 && a1_stride % V == 0 && a2_stride % V == 0 && ga_stride % V == 0 && f_stride % V == 0 &&
                         gf_stride % V == 0 && state_stride % 4 == 0;
        const int per = vec ? V : 1;
        int threads = ((width + per - 1) / per + 31) / 32 * 32;
        if (threads > 512) threads = 512;
        // a run of rows forms one row more than it has, so longer runs read less; shorter ones are more CTAs
        int run = 1;
        while (ys && run < 8 && (long long)n_rows * threads > (long long)run * sm_count() * 2048) run *= 2;
        const int grid = (n_rows + run - 1) / run;
#define GS_LAUNCH(N) do { \
            if (smem > 48 * 1024) cudaFuncSetAttribute(gated_sum_norm32_kernel<T, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            launch_chained(gated_sum_norm32_kernel<T, N>, dim3(grid), dim3(threads), smem, stream, g, x_out, gain1, (T*)y1, shift, (T*)ys, gain2, \
                           (T*)y2, (const MMSegment*)segs, n_segs, state, state_stride, rows, n_rows, width, eps, run); } while (0)
        if (vec) GS_LAUNCH(V); else GS_LAUNCH(1);
    });
    return launch_status();
}

// Up to three terms a stream still has to take: rows of the compute dtype with strides in elements, a constant each.
#define GS_TERMS 3
struct StreamTerms {
    const void* d[GS_TERMS];
    float c[GS_TERMS];
    int stride[GS_TERMS];
};

// A CTA a row; a thread has the same entries of it in every pass, N at a time: the first ones in registers, the others in
// shared memory.  The sum is stored only when every row is taken (rows null).  bias null and centered 0: the root mean square's
// norm; centered: (x - mean) / sqrt(mean of squared deviations + eps).
template <typename T, int N>
__global__ void __launch_bounds__(512) add_terms_norm32_kernel(float* x, StreamTerms terms, const float* __restrict__ gain, const float* __restrict__ bias,
                                                               int centered, T* __restrict__ y, const int* __restrict__ rows, int width, float eps) {
    extern __shared__ __align__(16) float gs_smem[];          // [width - blockDim.x N]: what the registers do not hold
    __shared__ float scratch[32];
    const int stride = blockDim.x * N, c0 = threadIdx.x * N;
    float w0[N], b0[N];
    const bool some = c0 < width;
    if (some) {                                               // the weights do not come from the kernel before
        gs_load32<N>(gain + c0, w0);
        if (bias) gs_load32<N>(bias + c0, b0);
    }
    pdl_launch_dependents();
    pdl_wait(KID_GATED_STREAM);
    const size_t r = rows ? (size_t)rows[blockIdx.x] : (size_t)blockIdx.x;
    float* xr = x + r * width;
    const bool store = terms.d[0] != nullptr && rows == nullptr;
    float keep[N];
    float sum = 0.f, ss = 0.f;
    for (int c = c0; c < width; c += stride) {
        float v[N];
        gs_load32<N>(xr + c, v);
#pragma unroll
        for (int i = 0; i < GS_TERMS; i++) {
            if (!terms.d[i]) break;
            float t[N];
            gs_load<T, N>((const T*)terms.d[i] + r * terms.stride[i] + c, t);
#pragma unroll
            for (int k = 0; k < N; k++) v[k] = fmaf(terms.c[i], t[k], v[k]);
        }
        if (store) gs_store32<N>(xr + c, v);
#pragma unroll
        for (int k = 0; k < N; k++) { sum += v[k]; ss = fmaf(v[k], v[k], ss); }
        if (c == c0) {
#pragma unroll
            for (int k = 0; k < N; k++) keep[k] = v[k];
        } else {
            gs_store32<N>(gs_smem + c - stride, v);
        }
    }
    float mean = 0.f;
    if (centered) {
        mean = block_sum(sum, scratch) / (float)width;
        ss = 0.f;
        for (int c = c0; c < width; c += stride) {
            float v[N];
            if (c == c0) {
#pragma unroll
                for (int k = 0; k < N; k++) v[k] = keep[k];
            } else {
                gs_load32<N>(gs_smem + c - stride, v);
            }
#pragma unroll
            for (int k = 0; k < N; k++) { const float o = v[k] - mean; ss = fmaf(o, o, ss); }
        }
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)width + eps);
    T* yr = y + (size_t)blockIdx.x * width;
    for (int c = c0; c < width; c += stride) {
        float v[N], w[N], b[N];
        if (c == c0) {
#pragma unroll
            for (int k = 0; k < N; k++) { v[k] = keep[k]; w[k] = w0[k]; b[k] = bias ? b0[k] : 0.f; }
        } else {
            gs_load32<N>(gs_smem + c - stride, v);
            gs_load32<N>(gain + c, w);
            if (bias) gs_load32<N>(bias + c, b);
            else {
#pragma unroll
                for (int k = 0; k < N; k++) b[k] = 0.f;
            }
        }
#pragma unroll
        for (int k = 0; k < N; k++) v[k] = fmaf((v[k] - mean) * inv, w[k], b[k]);
        gs_store<T, N>(yr + c, v);
    }
}

// Terms from the first on; an absent one ends them.  With `rows` (n_rows of them) only those rows are formed and normed, into
// row i of y, and x stays as it is.
PLLM_EXPORT int pllm_add_terms_norm32(int dtype, float* x, const void* d1, int s1, float c1, const void* d2, int s2, float c2, const void* d3, int s3,
                                      float c3, const float* gain, const float* bias, int centered, void* y, const int* rows, int n_rows, int width,
                                      float eps, cudaStream_t stream) {
    if (n_rows <= 0) return PLLM_OK;
    if (width <= 0 || !x || !gain || !y || (d2 && !d1) || (d3 && !d2)) return PLLM_ERR_SIZE;
    StreamTerms terms = {{d1, d2, d3}, {c1, c2, c3}, {s1, s2, s3}};
    PLLM_DISPATCH_DTYPE(dtype, {
        constexpr int V = Vec16<T>::N;
        const uintptr_t p = (uintptr_t)x | (uintptr_t)d1 | (uintptr_t)d2 | (uintptr_t)d3 | (uintptr_t)gain | (uintptr_t)bias | (uintptr_t)y;
        const bool vec = width % V == 0 && (p & 15) == 0 && (!d1 || s1 % V == 0) && (!d2 || s2 % V == 0) && (!d3 || s3 % V == 0);
        // four entries a thread at the least where the dtype's vectors are four, eight else; rows of few vectors in small CTAs
        const int per = vec ? V : 1;
        int threads = ((width + per - 1) / per + 31) / 32 * 32;
        if (threads > 512) threads = 512;
        const int held = threads * per;
        const size_t smem = width > held ? (size_t)(width - held) * sizeof(float) : 0;
        if (smem > 200 * 1024) return PLLM_ERR_LIMIT;
        auto kernel = vec ? add_terms_norm32_kernel<T, V> : add_terms_norm32_kernel<T, 1>;
        if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch_chained(kernel, dim3(n_rows), dim3(threads), smem, stream, x, terms, gain, bias, centered, (T*)y, rows, width, eps);
    });
    return launch_status();
}

// A CTA a row of u ([rows, u_stride], the first `width` columns); abce: four floats on the device.
template <typename T, int N>
__global__ void __launch_bounds__(512) poly_norm_kernel(const T* u, int u_stride, const float* __restrict__ abce, T* __restrict__ y, int width,
                                                        float eps) {
    __shared__ float part[3][16];
    pdl_launch_dependents();
    pdl_wait(KID_GATED_STREAM);
    const T* ur = u + (size_t)blockIdx.x * u_stride;
    T* yr = y + (size_t)blockIdx.x * width;
    const int stride = blockDim.x * N, c0 = threadIdx.x * N;
    float s1 = 0.f, s2 = 0.f, s3 = 0.f;
    float keep[N];
    for (int c = c0; c < width; c += stride) {
        float v[N];
        gs_load<T, N>(ur + c, v);
#pragma unroll
        for (int k = 0; k < N; k++) {
            const float q = v[k] * v[k];
            s1 += q; s2 = fmaf(q, q, s2); s3 = fmaf(q * q, q, s3);
            if (c == c0) keep[k] = v[k];
        }
    }
    s1 = warp_sum(s1); s2 = warp_sum(s2); s3 = warp_sum(s3);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    if (lane == 0) { part[0][warp] = s1; part[1][warp] = s2; part[2][warp] = s3; }
    __syncthreads();
    s1 = s2 = s3 = 0.f;
    for (int w = 0; w < warps; w++) { s1 += part[0][w]; s2 += part[1][w]; s3 += part[2][w]; }
    const float n = (float)width;
    const float fa = abce[0] / sqrtf(s1 / n + eps), fb = abce[1] / sqrtf(s2 / n + eps), fc = abce[2] / sqrtf(s3 / n + eps), fe = abce[3];
    for (int c = c0; c < width; c += stride) {
        float v[N];
        if (c == c0) {
#pragma unroll
            for (int k = 0; k < N; k++) v[k] = keep[k];
        } else {
            gs_load<T, N>(ur + c, v);
        }
#pragma unroll
        for (int k = 0; k < N; k++) v[k] = fmaf(v[k], fmaf(v[k], fmaf(v[k], fc, fb), fa), fe);
        gs_store<T, N>(yr + c, v);
    }
}

PLLM_EXPORT int pllm_poly_norm(int dtype, const void* u, int u_stride, const float* abce, void* y, int n_rows, int width, float eps,
                               cudaStream_t stream) {
    if (n_rows <= 0) return PLLM_OK;
    if (width <= 0 || u_stride < width || !abce) return PLLM_ERR_SIZE;
    PLLM_DISPATCH_DTYPE(dtype, {
        constexpr int V = Vec16<T>::N;
        const bool vec = width % V == 0 && u_stride % V == 0 && (((uintptr_t)u | (uintptr_t)y) & 15) == 0;
        const int per = vec ? V : 1;
        int threads = ((width + per - 1) / per + 31) / 32 * 32;
        if (threads > 512) threads = 512;
        if (vec) launch_chained(poly_norm_kernel<T, V>, dim3(n_rows), dim3(threads), 0, stream, (const T*)u, u_stride, abce, (T*)y, width, eps);
        else launch_chained(poly_norm_kernel<T, 1>, dim3(n_rows), dim3(threads), 0, stream, (const T*)u, u_stride, abce, (T*)y, width, eps);
    });
    return launch_status();
}

__global__ void __launch_bounds__(256) softcap32_kernel(float* x, float cap, long long total) {
    pdl_launch_dependents();
    pdl_wait(KID_GATED_STREAM);
    const float inv = 1.0f / cap;
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] * inv);
}

PLLM_EXPORT int pllm_softcap32(float* x, float cap, long long total, cudaStream_t stream) {
    if (total <= 0) return PLLM_OK;
    if (!(cap > 0.f)) return PLLM_ERR_SIZE;
    const int blocks = (int)min((long long)sm_count() * 8, (total + 255) / 256);
    launch_chained(softcap32_kernel, dim3(blocks), dim3(256), 0, stream, x, cap, total);
    return launch_status();
}

PLLM_TRACE_EXPORT(gated_stream)
