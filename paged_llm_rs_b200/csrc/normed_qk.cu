// What stands between an attention mixer's input projection and its attention kernel, for mixers that norm their
// queries and keys, and the gate on an attention's output.
//
//   normed_qk_kv_write   one pass over the stacked projection [q | k | (v) | ...] of the step's tokens, a CTA a token:
//                          biases on q, k and v (each may be absent)
//                          norm      0 none; 1 each head by its own root mean square, one gain of dk entries shared by the
//                                    heads; 2 the whole projection (all heads of q, and likewise of k) by one root mean
//                                    square, a gain of its full size; 3 each head by its own root mean square as it is behind
//                                    the rotation, no gain
//                          q *= 1 + coef * ln(floor((p + 1) / every) + 1)     (every = 0: no such factor)
//                          rotation of the first `rot` entries of every q and k head, entry i with entry i + rot / 2 or entry
//                                    2i with entry 2i + 1, by the angle p * inv_freq[i], a float product; cos and sin times a
//                                    factor
//                          q to its own tensor; k | v to the token's row of the joined pool; v is the projection's v
//                          part, or (values_are_keys) the raw key projection, neither normed nor rotated
//                        Everything is float from the projection's values to the one rounding on the way out.
//   gate_mul             y[t, c] *= sigmoid(g[t, c / per]) (kind 0) or silu(g[t, c / per]) (kind 1); g rows may be strided; per 1: a
//                        gate an entry, per = a head's size: a gate a head
#include "matrix_memory.cuh"

enum : int { KID_NORMED_QK = 90 };

__device__ __forceinline__ float nq_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// Sum over the CTA, for every thread (scratch: 32 floats).
__device__ __forceinline__ float nq_block_sum(float v, float* scratch) { return block_sum(v, scratch); }

// What the pass over a token's projection does.
struct NormedQK {
    int k_off, v_off;                // columns of the keys and the values (k_off negative: queries only)
    const float *q_bias, *k_bias, *v_bias;       // nh dk, nkv dk, nkv dv (null: none)
    const float *q_gain, *k_gain;
    int norm;                        // 0 none; 1 a head; 2 the whole projection; 3 a head, behind the rotation, no gain
    float eps;
    float temp_coef;
    int temp_every;
    const float* inv_freq;
    int rot;                         // leading entries of each head that turn
    int pairs;                       // 0: entry i turns with entry i + rot / 2; 1: entry 2i with entry 2i + 1
    float rot_factor;                // on cos and sin
    int nh, nkv, dk, dv, values_are_keys, page_size;
    long long pool_rows;
};

// entry e of a head that lies in shared memory, normed and turned
__device__ __forceinline__ float nq_entry(const float* head, const float* __restrict__ gain, int e, float inv, const NormedQK& a, const float2* turn) {
    float v = head[e] * inv;
    if (gain) v *= gain[e];
    if (e < a.rot) {
        const int half = a.rot >> 1;
        const bool first = a.pairs ? !(e & 1) : e < half;
        const int f = a.pairs ? e >> 1 : (first ? e : e - half);
        const int j = a.pairs ? e ^ 1 : (first ? e + half : e - half);
        float other = head[j] * inv;
        if (gain) other *= gain[j];
        const float2 t = turn[f];
        v = first ? v * t.x - other * t.y : v * t.x + other * t.y;
    }
    return v;
}

// A CTA a token.  Its queries and keys lie in shared memory as floats; the cos and sin of its angles are formed once for all heads.
// N: entries a thread takes at a time (4 where every part and head is whole groups of four, else 1).
template <typename T, int N>
__global__ void __launch_bounds__(256) normed_qk_kv_write_kernel(const T* proj, int row_stride, NormedQK a, T* __restrict__ q_out,
                                                                 const int* __restrict__ positions, const int* __restrict__ slots,
                                                                 T* kv_pool, int* status) {
    extern __shared__ __align__(16) float nq_smem[];
    const int nh = a.nh, nkv = a.k_off >= 0 ? a.nkv : 0, dk = a.dk, dv = a.dv;
    const int qw = nh * dk, kw = nkv * dk;
    float* q_s = nq_smem;                                     // [qw]
    float* k_s = q_s + (qw + 3) / 4 * 4;                      // [kw]
    float2* turn = reinterpret_cast<float2*>(k_s + (kw + 3) / 4 * 4);      // [rot / 2] cos and sin times the factor
    float* head_inv = reinterpret_cast<float*>(turn + a.rot / 2);          // [nh + nkv] 1 / rms of each head (norms 1 and 3)
    __shared__ float scratch[32];
    pdl_launch_dependents();
    // (the step's packed buffer is in place before the kernels of the step begin)
    const int t = blockIdx.x;
    const int pos = positions[t];
    const int slot = slots ? slots[t] : -1;
    for (int f = threadIdx.x; f < a.rot / 2; f += blockDim.x) {
        float s, c;
        sincosf((float)pos * a.inv_freq[f], &s, &c);
        turn[f] = make_float2(c * a.rot_factor, s * a.rot_factor);
    }
    pdl_wait(KID_NORMED_QK);
    const T* row = proj + (size_t)t * row_stride;
    const T* kr = row + a.k_off;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * N; i < qw; i += blockDim.x * N) {
        float v[N];
        if constexpr (N == 4) head_quad_load(row + i, v); else v[0] = to_f32(row[i]);
#pragma unroll
        for (int k = 0; k < N; k++) {
            if (a.q_bias) v[k] += a.q_bias[i + k];
            q_s[i + k] = v[k];
            sq = fmaf(v[k], v[k], sq);
        }
    }
    for (int i = threadIdx.x * N; i < kw; i += blockDim.x * N) {
        float v[N];
        if constexpr (N == 4) head_quad_load(kr + i, v); else v[0] = to_f32(kr[i]);
#pragma unroll
        for (int k = 0; k < N; k++) {
            if (a.k_bias) v[k] += a.k_bias[i + k];
            k_s[i + k] = v[k];
            sk = fmaf(v[k], v[k], sk);
        }
    }
    float q_inv = 1.f, k_inv = 1.f;
    if (a.norm == 2) {
        sq = nq_block_sum(sq, scratch);
        q_inv = 1.0f / sqrtf(sq / (float)qw + a.eps);
        if (kw) {
            sk = nq_block_sum(sk, scratch);
            k_inv = 1.0f / sqrtf(sk / (float)kw + a.eps);
        }
    } else {
        __syncthreads();
        if (a.norm) {
            // (a pair keeps its length when it turns, but for the factor: a head's mean square behind the rotation follows from
            // the entries ahead of it)
            const float turned = a.norm == 3 ? a.rot_factor * a.rot_factor : 1.f;
            const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
            for (int h = warp; h < nh + nkv; h += warps) {
                const float* hr = h < nh ? q_s + h * dk : k_s + (h - nh) * dk;
                float s = 0.f;
                for (int e = lane; e < dk; e += 32) { const float v = hr[e]; s = fmaf(e < a.rot ? v * turned : v, v, s); }
                s = warp_sum(s);
                if (lane == 0) head_inv[h] = 1.0f / sqrtf(s / (float)dk + a.eps);
            }
            __syncthreads();
        }
    }
    float temp = 1.f;
    if (a.temp_every > 0) temp = 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every + 1));
    const bool a_head = a.norm == 1 || a.norm == 3;
    const int gain_stride = a.norm == 2 ? dk : 0;             // a gain of the projection's size, or one a head shared by the heads
    T* qo = q_out + (size_t)t * qw;
    for (int i = threadIdx.x * N; i < qw; i += blockDim.x * N) {
        const int h = i / dk, e = i - h * dk;
        const float inv = a_head ? head_inv[h] : q_inv;
        const float* g = a.q_gain ? a.q_gain + h * gain_stride : nullptr;
        float v[N];
#pragma unroll
        for (int k = 0; k < N; k++) v[k] = nq_entry(q_s + h * dk, g, e + k, inv, a, turn) * temp;
        if constexpr (N == 4) head_quad_store(qo + i, v); else qo[i] = from_f32<T>(v[0]);
    }
    if (kv_pool == nullptr || slot < 0 || nkv == 0) return;
    if ((long long)slot >= a.pool_rows) { if (threadIdx.x == 0) atomicOr(status, 2); return; }
    const int page = slot / a.page_size, off = slot % a.page_size;
    const int w = dk + dv;
    const T* vr = row + a.v_off;
    for (int i = threadIdx.x * N; i < nkv * w; i += blockDim.x * N) {
        const int g = i / w, e = i - g * w;
        T* dst = kv_pool + (((size_t)page * nkv + g) * a.page_size + off) * w + e;
        float v[N];
        if (e < dk) {
            const float inv = a_head ? head_inv[nh + g] : k_inv;
            const float* gn = a.k_gain ? a.k_gain + g * gain_stride : nullptr;
#pragma unroll
            for (int k = 0; k < N; k++) v[k] = nq_entry(k_s + g * dk, gn, e + k, inv, a, turn);
        } else if (a.values_are_keys) {
            // the raw key projection, neither normed nor turned
#pragma unroll
            for (int k = 0; k < N; k++) v[k] = k_s[g * dk + e - dk + k];
        } else {
            const int c = g * dv + e - dk;
            if constexpr (N == 4) head_quad_load(vr + c, v); else v[0] = to_f32(vr[c]);
            if (a.v_bias) {
#pragma unroll
                for (int k = 0; k < N; k++) v[k] += a.v_bias[c + k];
            }
        }
        if constexpr (N == 4) head_quad_store(dst, v); else dst[0] = from_f32<T>(v[0]);
    }
}

// proj: [tokens, row_stride] with q at 0, k at k_off (negative: queries only), v at v_off (ignored when values_are_keys, which
// needs dv == dk).  Biases: float, one an entry, or null.  q_gain / k_gain: float, dk entries (norm 1) or nh * dk and nkv * dk
// (norm 2), null for the others; inv_freq: rot / 2 floats.
PLLM_EXPORT int pllm_normed_qk_kv_write(int dtype, const void* proj, int row_stride, int k_off, int v_off, const float* q_bias, const float* k_bias,
                                        const float* v_bias, void* q_out, const float* q_gain, const float* k_gain, int norm, float eps,
                                        float temp_coef, int temp_every, const float* inv_freq, int rot, int pairs, float rot_factor,
                                        const int* positions, const int* slots, void* kv_pool, int n_tokens, int nh, int nkv, int dk, int dv,
                                        int values_are_keys, int page_size, long long pool_rows, int* status, cudaStream_t stream) {
    if (n_tokens <= 0) return PLLM_OK;
    if (nh <= 0 || nkv <= 0 || dk <= 0 || dv <= 0 || page_size <= 0 || rot < 0 || rot > dk || rot % 2) return PLLM_ERR_SIZE;
    const bool gains = norm == 1 || norm == 2;
    if (norm < 0 || norm > 3 || (gains && !q_gain) || (gains && k_off >= 0 && !k_gain) || (rot && !inv_freq) || temp_every < 0) return PLLM_ERR_SIZE;
    if (values_are_keys && dv != dk) return PLLM_ERR_SIZE;
    NormedQK a = {k_off, v_off, q_bias, k_bias, v_bias, gains ? q_gain : nullptr, gains ? k_gain : nullptr, norm, eps, temp_coef, temp_every,
                  inv_freq, rot, pairs ? 1 : 0, rot_factor, nh, nkv, dk, dv, values_are_keys, page_size, pool_rows};
    const size_t smem = ((size_t)nh * dk + (k_off >= 0 ? (size_t)nkv * dk : 0) + 8 + rot + nh + nkv) * sizeof(float);
    if (smem > 200 * 1024) return PLLM_ERR_LIMIT;
    PLLM_DISPATCH_DTYPE(dtype, {
        const bool quads = dk % 4 == 0 && dv % 4 == 0 && row_stride % 4 == 0 && (k_off < 0 || k_off % 4 == 0) && (values_are_keys || v_off % 4 == 0) &&
                           (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)kv_pool) & (4 * sizeof(T) - 1)) == 0;
        auto kernel = quads ? normed_qk_kv_write_kernel<T, 4> : normed_qk_kv_write_kernel<T, 1>;
        if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch_chained(kernel, dim3(n_tokens), dim3(256), smem, stream, (const T*)proj, row_stride, a, (T*)q_out, positions, slots, (T*)kv_pool, status);
    });
    return launch_status();
}

template <typename T>
__global__ void gate_mul_kernel(T* y, const T* g, int g_stride, int width, long long total, int kind, int per) {
    pdl_launch_dependents();
    pdl_wait(KID_NORMED_QK);
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / width;
        const int c = (int)(i % width);
        const float z = to_f32(g[r * g_stride + c / per]);
        const float s = nq_sigmoid(z);
        y[i] = from_f32<T>(to_f32(y[i]) * (kind == 1 ? z * s : s));
    }
}

PLLM_EXPORT int pllm_gate_mul(int dtype, void* y, const void* g, int g_stride, int n_rows, int width, int kind, int per,
                              cudaStream_t stream) {
    if (n_rows <= 0) return PLLM_OK;
    if (width <= 0 || kind < 0 || kind > 1 || per < 1 || width % per) return PLLM_ERR_SIZE;
    PLLM_DISPATCH_DTYPE(dtype, {
        const long long total = (long long)n_rows * width;
        const int blocks = (int)min((long long)sm_count() * 8, (total + 255) / 256);
        launch_chained(gate_mul_kernel<T>, dim3(blocks), dim3(256), 0, stream, (T*)y, (const T*)g, g_stride, width, total, kind, per);
    });
    return launch_status();
}

PLLM_TRACE_EXPORT(normed_qk)
