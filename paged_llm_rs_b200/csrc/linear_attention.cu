// Linear attention with decay: recurrent mixers without softmax or denominator whose state is one matrix a head, S (d x e:
// key entries by value entries), carried from token to token in float for every request (a state slot):
//
//     S <- diag(alpha_t) S + k_t v_t^T        o_t = S^T q_t
//
//   alpha      one constant a head (retention), or one number a key entry and token (gated linear attention):
//              alpha = sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau), z = W_a2 a1 + b with a1 = W_a1 h a short float vector
//   q, k       times a constant each; the first `rot` entries of a head turned by position * inv_freq[i] (entry i with
//              entry i + rot / 2), an angle formed in float
//   behind it  each head's o over its root mean square, times a gain shared by the heads (or none), times silu of a gate
//
// A step is a list of segments {first token, tokens, tokens before, state slot} on the device, as for the other recurrences.
//
//   channel_decay_kernel    alpha for every token (a step with portions of prompts)
//   la_scan_kernel          portions of prompts.  A segment is cut into blocks of L tokens that run AT THE SAME TIME: the first
//                           starts from the request's slot, the others from zero.  Thread (columns, part) holds NPT rows of
//                           four columns of S in registers (so that a key or query entry read from shared memory serves four
//                           products) and goes through the block's tokens; a column's shares of a read-out are added once a
//                           chunk, in the order of the parts.
//   la_block_states_kernel  the state at every block's end from the block before it (S_b += A_b S_(b-1), A_b the product of
//                           a block's decays, at most one), the last one into the slot
//   la_block_outputs_kernel o_t += (A_t q_t)^T S_(b-1) for the blocks behind the first, A_t the product of the decays from the
//                           block's start to t: a small float product.  Nothing is divided by a decay, so strong decays only
//                           take these terms to zero.
//   la_step_kernel          decoded tokens: a CTA a (request, head, slice of columns) streams its part of S through registers
//                           once; a head's slices are one cluster and meet (shared memory of each other's SM) for the head's
//                           root mean square, so that the gated, normed output leaves this kernel.
//
// What a token's output is depends on where a prompt was cut, and on L, only by the order of the sums.
#include <cooperative_groups.h>

#include "matrix_memory.cuh"

namespace cg = cooperative_groups;

enum : int { KID_LINEAR_ATT = 120 };

#define LA_MAX_RANK 256        // entries of a1
#define LA_COLS 4              // columns of S a thread of the scan holds

struct LAShape {
    int H, d, E;               // heads, key entries, value entries
    int q_off, k_off, v_off, g_off, u_stride;      // columns of the stacked projection
    float q_scale, k_scale;
    int rot;
    const float* inv_freq;     // rot / 2
    const float* decay;        // [H] constants, or null: a decay a key entry
};

// entry i of a head of q or k, turned if it is among the first `rot` (by its angle's cos and sin, rope null: formed here)
template <typename T>
__device__ __forceinline__ float la_entry(const T* head, int i, const LAShape& s, float position, float scale, const float2* rope = nullptr) {
    float v = to_f32(head[i]);
    if (i < s.rot) {
        const int half = s.rot >> 1, f = i < half ? i : i - half;
        const float other = to_f32(head[i < half ? i + half : i - half]);
        float sn, c;
        if (rope) { c = rope[f].x; sn = rope[f].y; }
        else sincosf(position * s.inv_freq[f], &sn, &c);
        v = i < half ? v * c - other * sn : v * c + other * sn;
    }
    return v * scale;
}

// alpha of key entry n (of all heads'): a2 [H d, rank]
template <typename T>
__device__ __forceinline__ float la_channel_decay(const T* __restrict__ a2, const float* a1, float bias, int rank, float inv_tau) {
    float z = bias;
    for (int r = 0; r < rank; r++) z = fmaf(to_f32(a2[r]), a1[r], z);
    return expf(mm_logsigmoid(z) * inv_tau);
}

// grid (runs of LA_DECAY_TOKENS tokens, blocks of 128 key entries): a thread has one key entry, its row of a2 in registers 16
// entries at a time.
#define LA_DECAY_TOKENS 16
template <typename T>
__global__ void __launch_bounds__(128) channel_decay_kernel(const float* a1, const T* __restrict__ a2, const float* __restrict__ bias,
                                                            float* __restrict__ alpha, int n_tokens, int n, int rank, float inv_tau) {
    extern __shared__ __align__(16) float mm_smem[];      // [LA_DECAY_TOKENS][rank up to a multiple of 16, zeros behind it]
    pdl_launch_dependents();
    pdl_wait(KID_LINEAR_ATT);
    const int t0 = blockIdx.x * LA_DECAY_TOKENS, nt = min(LA_DECAY_TOKENS, n_tokens - t0), padded = (rank + 15) / 16 * 16;
    for (int i = threadIdx.x; i < LA_DECAY_TOKENS * padded; i += blockDim.x) {
        const int t = i / padded, r = i - t * padded;
        mm_smem[i] = (t < nt && r < rank) ? a1[(size_t)(t0 + t) * rank + r] : 0.f;
    }
    __syncthreads();
    const int i = blockIdx.y * 128 + threadIdx.x;
    if (i >= n) return;
    const float b = bias[i];
    float z[LA_DECAY_TOKENS];
#pragma unroll
    for (int t = 0; t < LA_DECAY_TOKENS; t++) z[t] = b;
    for (int r0 = 0; r0 < rank; r0 += 16) {
        float w[16];
#pragma unroll
        for (int r = 0; r < 16; r++) w[r] = r0 + r < rank ? to_f32(a2[(size_t)i * rank + r0 + r]) : 0.f;
#pragma unroll
        for (int t = 0; t < LA_DECAY_TOKENS; t++) {
            const float4* a4 = reinterpret_cast<const float4*>(mm_smem + t * padded + r0);
#pragma unroll
            for (int r = 0; r < 4; r++) {
                const float4 v = a4[r];
                z[t] = fmaf(w[4 * r], v.x, z[t]); z[t] = fmaf(w[4 * r + 1], v.y, z[t]);
                z[t] = fmaf(w[4 * r + 2], v.z, z[t]); z[t] = fmaf(w[4 * r + 3], v.w, z[t]);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < LA_DECAY_TOKENS; t++)
        if (t < nt) alpha[(size_t)(t0 + t) * n + i] = expf(mm_logsigmoid(z[t]) * inv_tau);
}

// cos and sin of every token's angles: rope [tokens, half] of (cos, sin), for the layers of a step that turn alike.
__global__ void __launch_bounds__(128) rope_table_kernel(const int* __restrict__ positions, const float* __restrict__ inv_freq,
                                                         float2* __restrict__ rope, long long total, int half) {
    pdl_launch_dependents();
    pdl_wait(KID_LINEAR_ATT);
    const long long i = blockIdx.x * 128LL + threadIdx.x;
    if (i >= total) return;
    float sn, c;
    sincosf((float)positions[i / half] * inv_freq[i % half], &sn, &c);
    rope[i] = make_float2(c, sn);
}

PLLM_EXPORT int pllm_rope_table(const int* positions, const float* inv_freq, float* rope, int n_tokens, int half, cudaStream_t stream) {
    if (n_tokens <= 0) return PLLM_OK;
    if (half <= 0) return PLLM_ERR_SIZE;
    const long long total = (long long)n_tokens * half;
    launch_chained(rope_table_kernel, dim3((unsigned)((total + 127) / 128)), dim3(128), 0, stream, positions, inv_freq, (float2*)rope, total, half);
    return launch_status();
}

// grid (blocks, heads, slices of e).  u: [tokens, u_stride] of the compute dtype; alpha: [tokens, H d] float (per entry).
template <typename T, int NPT, bool CHANNEL>
__global__ void __launch_bounds__(256, 2) la_scan_kernel(const T* u, LAShape sh, const float2* rope, const float* alpha, const MMSegment* __restrict__ segs, int n_segs,
                                                      float* state, long long state_stride, float* __restrict__ y,
                                                      float* __restrict__ block_state, float* __restrict__ block_decay,
                                                      float* __restrict__ qa, int Ps, int parts, int ck, int L) {
    extern __shared__ __align__(16) float mm_smem[];
    constexpr int VEC = MMVec<T>::N;
    const int NP = NPT * parts, H = sh.H, d = sh.d, E = sh.E;
    float* q_s = mm_smem;                                   // [ck][NP]
    float* k_s = q_s + ck * NP;                             // [ck][NP]
    float* a_s = k_s + ck * NP;                             // CHANNEL: [ck][NP]
    float* run_s = a_s + (CHANNEL ? ck * NP : 0);           // [NP] product of the decays since the block's start
    float* pow_s = run_s + NP;                              // constant decays: [32] decay^(t + 1), [32] decay^-(t + 1)
    float* v_s = pow_s + (CHANNEL ? 0 : 64);                // [ck][Ps]
    float* y_s = v_s + ck * Ps;                             // [ck][parts][Ps]
    pdl_launch_dependents();
    pdl_wait(KID_LINEAR_ATT);
    const MMBlock b = mm_find_block(segs, n_segs, blockIdx.x, L);
    if (b.seg < 0) return;
    const MMSegment s = segs[b.seg];
    const int h = blockIdx.y, p0 = blockIdx.z * Ps, tid = threadIdx.x;
    const int begin = b.tb * L, count = min(L, s.count - begin);
    const int groups = Ps / LA_COLS, col = tid % groups * LA_COLS, part = tid / groups, e = p0 + col;
    const bool live = part < parts && e < E;
    const float decay = CHANNEL ? 0.f : sh.decay[h];
    float* S = state + (size_t)s.slot * state_stride + (size_t)h * d * E;
    f32x2 st[LA_COLS][NPT / 2];
#pragma unroll
    for (int k = 0; k < NPT; k += 2) {
        const int n = part * NPT + k;
        const bool from = live && b.tb == 0 && s.before > 0;
#pragma unroll
        for (int c = 0; c < LA_COLS; c++) {
            const float* p = S + (size_t)n * E + e + c;
            const bool in = from && e + c < E;
            st[c][k / 2] = mm_pair((in && n < d) ? p[0] : 0.f, (in && n + 1 < d) ? p[E] : 0.f);
        }
    }
    // A constant decay that is not too strong leaves the token loop: a chunk's state is kept over decay^(t + 1), so that values
    // come in times decay^-(t + 1), read-outs leave times decay^(t + 1), and the state is multiplied once a chunk.
    bool scaled = false;
    if (!CHANNEL) {
        if (tid < ck) {
            const double l = (double)(tid + 1) * log((double)fmaxf(decay, 1e-30f));
            pow_s[tid] = (float)exp(l);
            pow_s[32 + tid] = (float)exp(fmin(-l, 80.0));
        }
        __syncthreads();
        scaled = pow_s[ck - 1] > 1e-8f;
    }
    // this slice's share of the head's key entries, for the running products and the decayed queries
    const int share = (d + gridDim.z - 1) / gridDim.z, n_lo = min(d, (int)blockIdx.z * share), n_hi = min(d, n_lo + share);
    const bool several = b.blocks > 1;
    for (int i = tid; i < NP; i += blockDim.x) run_s[i] = 1.f;
    if (NP > d) for (int i = tid; i < 2 * ck * NP; i += blockDim.x) q_s[i] = 0.f;      // (the padding rows stay zero)
    if (NP > d && CHANNEL) for (int i = tid; i < ck * NP; i += blockDim.x) a_s[i] = 0.f;
    const int half = sh.rot >> 1;
    const bool vec = d % VEC == 0 && half % VEC == 0 && sh.u_stride % VEC == 0 && sh.q_off % VEC == 0 && sh.k_off % VEC == 0 &&
                     (reinterpret_cast<uintptr_t>(u) & 15) == 0;
    const bool vec_v = Ps % VEC == 0 && E % VEC == 0 && sh.u_stride % VEC == 0 && sh.v_off % VEC == 0 && (reinterpret_cast<uintptr_t>(u) & 15) == 0;
    for (int t0 = 0; t0 < count; t0 += ck) {
        const int nt = min(ck, count - t0);
        const size_t tok0 = (size_t)s.first + begin + t0;
        __syncthreads();
        if (vec) {
            const int pairs = half / VEC, units = pairs + (d - sh.rot) / VEC;
            for (int i = tid; i < nt * units; i += blockDim.x) {
                const int t = i / units, j = i - t * units;
                const T* qr = u + (tok0 + t) * sh.u_stride + sh.q_off + (size_t)h * d;
                const T* kr = u + (tok0 + t) * sh.u_stride + sh.k_off + (size_t)h * d;
                const float2* turn = rope + (tok0 + t) * half;
                if (j >= pairs) {
                    const int n = sh.rot + (j - pairs) * VEC;
                    mm_fetch16(qr + n, q_s + t * NP + n, sh.q_scale);
                    mm_fetch16(kr + n, k_s + t * NP + n, sh.k_scale);
                    continue;
                }
                const int n = j * VEC;
                Vec16<T> q0, q1, k0, k1;
                q0.load(qr + n); q1.load(qr + half + n); k0.load(kr + n); k1.load(kr + half + n);
                float qa0[VEC], qb0[VEC], ka0[VEC], kb0[VEC];
                q0.unpack(qa0); q1.unpack(qb0); k0.unpack(ka0); k1.unpack(kb0);
#pragma unroll
                for (int x = 0; x < VEC; x++) {
                    const float c = turn[n + x].x, sn = turn[n + x].y;
                    q_s[t * NP + n + x] = (qa0[x] * c - qb0[x] * sn) * sh.q_scale;
                    q_s[t * NP + half + n + x] = (qb0[x] * c + qa0[x] * sn) * sh.q_scale;
                    k_s[t * NP + n + x] = (ka0[x] * c - kb0[x] * sn) * sh.k_scale;
                    k_s[t * NP + half + n + x] = (kb0[x] * c + ka0[x] * sn) * sh.k_scale;
                }
            }
        } else {
            for (int i = tid; i < nt * d; i += blockDim.x) {
                const int t = i / d, n = i - t * d;
                const T* row = u + (tok0 + t) * sh.u_stride + (size_t)h * d;
                q_s[t * NP + n] = la_entry(row + sh.q_off, n, sh, 0.f, sh.q_scale, rope + (tok0 + t) * half);
                k_s[t * NP + n] = la_entry(row + sh.k_off, n, sh, 0.f, sh.k_scale, rope + (tok0 + t) * half);
            }
        }
        if (vec_v) {
            const int units = Ps / VEC;
            for (int i = tid; i < nt * units; i += blockDim.x) {
                const int t = i / units, c = (i - t * units) * VEC;
                if (p0 + c < E) mm_fetch16(u + (tok0 + t) * sh.u_stride + sh.v_off + (size_t)h * E + p0 + c, v_s + t * Ps + c, scaled ? pow_s[32 + t] : 1.f);
            }
        } else {
            for (int i = tid; i < nt * Ps; i += blockDim.x) {
                const int t = i / Ps, ee = p0 + i - t * Ps;
                float v = ee < E ? to_f32(u[(tok0 + t) * sh.u_stride + sh.v_off + (size_t)h * E + ee]) : 0.f;
                if (scaled) v *= pow_s[32 + t];
                v_s[i] = v;
            }
        }
        if (CHANNEL) {
            if (d % 4 == 0) {
                const int d4 = d >> 2;
                for (int i = tid; i < nt * d4; i += blockDim.x) {
                    const int t = i / d4, n = (i - t * d4) * 4;
                    *reinterpret_cast<float4*>(a_s + t * NP + n) = *reinterpret_cast<const float4*>(alpha + (tok0 + t) * H * d + (size_t)h * d + n);
                }
            } else {
                for (int i = tid; i < nt * d; i += blockDim.x) {
                    const int t = i / d, n = i - t * d;
                    a_s[t * NP + n] = alpha[(tok0 + t) * H * d + (size_t)h * d + n];
                }
            }
        }
        __syncthreads();
        if (several) {
            for (int n = n_lo + tid; n < n_hi; n += blockDim.x) {
                float run = run_s[n];
                for (int t = 0; t < nt; t++) {
                    run *= CHANNEL ? a_s[t * NP + n] : decay;
                    if (b.tb > 0) qa[(tok0 + t) * H * d + (size_t)h * d + n] = q_s[t * NP + n] * run;
                }
                run_s[n] = run;
            }
        }
        if (part < parts) {
            const f32x2 dd = mm_pair(decay, decay);
            const f32x2 zero = mm_pair(0.f, 0.f);
#define LA_TOKENS(UPDATE) do { \
            for (int t = 0; t < nt; t++) { \
                const float4 v4 = *reinterpret_cast<const float4*>(v_s + t * Ps + col); \
                const f32x2 v[LA_COLS] = {mm_pair(v4.x, v4.x), mm_pair(v4.y, v4.y), mm_pair(v4.z, v4.z), mm_pair(v4.w, v4.w)}; \
                const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(k_s + t * NP + part * NPT); \
                const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(q_s + t * NP + part * NPT); \
                const ulonglong2* a4 = reinterpret_cast<const ulonglong2*>(a_s + t * NP + part * NPT); \
                (void)a4; \
                f32x2 acc[LA_COLS] = {zero, zero, zero, zero}; \
                _Pragma("unroll") \
                for (int k = 0; k < NPT / 4; k++) { \
                    const ulonglong2 kv = k4[k], qv = q4[k]; \
                    const ulonglong2 av = CHANNEL ? a4[k] : make_ulonglong2(dd, dd); \
                    (void)av; \
                    _Pragma("unroll") \
                    for (int c = 0; c < LA_COLS; c++) { \
                        UPDATE; \
                        acc[c] = mm_fma2(st[c][2 * k], qv.x, acc[c]); acc[c] = mm_fma2(st[c][2 * k + 1], qv.y, acc[c]); \
                    } \
                } \
                const float2 r0 = mm_unpair(acc[0]), r1 = mm_unpair(acc[1]), r2 = mm_unpair(acc[2]), r3 = mm_unpair(acc[3]); \
                *reinterpret_cast<float4*>(y_s + (t * parts + part) * Ps + col) = make_float4(r0.x + r0.y, r1.x + r1.y, r2.x + r2.y, r3.x + r3.y); \
            } } while (0)
            if (scaled)
                LA_TOKENS(st[c][2 * k] = mm_fma2(kv.x, v[c], st[c][2 * k]); st[c][2 * k + 1] = mm_fma2(kv.y, v[c], st[c][2 * k + 1]));
            else
                LA_TOKENS(st[c][2 * k] = mm_fma2(av.x, st[c][2 * k], mm_mul2(kv.x, v[c]));
                          st[c][2 * k + 1] = mm_fma2(av.y, st[c][2 * k + 1], mm_mul2(kv.y, v[c])));
            if (scaled) {
                const f32x2 f = mm_pair(pow_s[nt - 1], pow_s[nt - 1]);
#pragma unroll
                for (int c = 0; c < LA_COLS; c++)
#pragma unroll
                    for (int k = 0; k < NPT / 2; k++) st[c][k] = mm_mul2(st[c][k], f);
            }
        }
        __syncthreads();
        for (int i = tid; i < nt * groups; i += blockDim.x) {
            const int t = i / groups, c = (i - t * groups) * LA_COLS;
            if (p0 + c >= E) continue;
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int q = 0; q < parts; q++) {                                               // always in the order of the parts
                const float4 x = *reinterpret_cast<const float4*>(y_s + (t * parts + q) * Ps + c);
                acc.x += x.x; acc.y += x.y; acc.z += x.z; acc.w += x.w;
            }
            const float f = scaled ? pow_s[t] : 1.f;
            acc.x *= f; acc.y *= f; acc.z *= f; acc.w *= f;
            float* yr = y + (tok0 + t) * H * E + (size_t)h * E + p0 + c;
            if (E % LA_COLS == 0) {
                *reinterpret_cast<float4*>(yr) = acc;
            } else {
                yr[0] = acc.x;
                if (p0 + c + 1 < E) yr[1] = acc.y;
                if (p0 + c + 2 < E) yr[2] = acc.z;
                if (p0 + c + 3 < E) yr[3] = acc.w;
            }
        }
    }
    float* dst = several ? block_state + ((size_t)b.rank * H + h) * d * E : S;
    if (live) {
#pragma unroll
        for (int k = 0; k < NPT; k += 2) {
            const int n = part * NPT + k;
#pragma unroll
            for (int c = 0; c < LA_COLS; c++) {
                if (e + c >= E) break;
                const float2 x = mm_unpair(st[c][k / 2]);
                if (n < d) dst[(size_t)n * E + e + c] = x.x;
                if (n + 1 < d) dst[(size_t)(n + 1) * E + e + c] = x.y;
            }
        }
    }
    if (several) for (int n = n_lo + tid; n < n_hi; n += blockDim.x) block_decay[((size_t)b.rank * H + h) * d + n] = run_s[n];
}

// grid (segments, heads, blocks of 256 state entries): for a segment of several blocks, block_state[b] becomes the state at
// block b's end, the last one also the slot's.
__global__ void __launch_bounds__(256) la_block_states_kernel(const MMSegment* __restrict__ segs, int n_segs, float* state, long long state_stride,
                                                              float* block_state, const float* block_decay, int H, int d, int E, int L) {
    pdl_launch_dependents();
    pdl_wait(KID_LINEAR_ATT);
    const MMSegment s = segs[blockIdx.x];
    if (s.count <= L) return;
    const int blocks = (s.count + L - 1) / L, h = blockIdx.y;
    int rank = 0;
    for (int i = 0; i < (int)blockIdx.x; i++) rank += segs[i].count > L ? (segs[i].count + L - 1) / L : 0;
    const long long i = blockIdx.z * 256LL + threadIdx.x;
    if (i >= (long long)d * E) return;
    const int n = (int)(i / E);
    const size_t step = (size_t)H * d * E;
    float* bs = block_state + ((size_t)rank * H + h) * d * E + i;
    const float* bd = block_decay + ((size_t)rank * H + h) * d + n;
    float cur = bs[0];
    for (int b0 = 1; b0 < blocks; b0 += 8) {           // (eight blocks' loads leave before the first is used)
        float x[8], a[8];
#pragma unroll
        for (int j = 0; j < 8; j++) {
            x[j] = b0 + j < blocks ? bs[(b0 + j) * step] : 0.f;
            a[j] = b0 + j < blocks ? bd[(size_t)(b0 + j) * H * d] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < 8; j++) {
            if (b0 + j >= blocks) break;
            cur = fmaf(a[j], cur, x[j]);
            bs[(b0 + j) * step] = cur;
        }
    }
    state[(size_t)s.slot * state_stride + (size_t)h * d * E + i] = cur;
}

// grid (blocks, heads x column tiles of 64, token tiles of 64): y += qa S for the tokens of blocks behind a segment's first.
// A thread has four tokens and four columns.
#define LA_TT 64
#define LA_TC 64
#define LA_TK 32
__global__ void __launch_bounds__(256) la_block_outputs_kernel(const MMSegment* __restrict__ segs, int n_segs, const float* qa, const float* block_state,
                                                               float* y, int H, int d, int E, int L, int col_tiles) {
    __shared__ __align__(16) float q_s[LA_TK][LA_TT + 4];
    __shared__ __align__(16) float S_s[LA_TK][LA_TC];
    pdl_launch_dependents();
    pdl_wait(KID_LINEAR_ATT);
    const MMBlock b = mm_find_block(segs, n_segs, blockIdx.x, L);
    if (b.seg < 0 || b.tb == 0) return;
    const MMSegment s = segs[b.seg];
    const int h = blockIdx.y / col_tiles, c0 = (blockIdx.y % col_tiles) * LA_TC, t0 = blockIdx.z * LA_TT;
    const int begin = b.tb * L, nt = min(L, s.count - begin) - t0;
    if (nt <= 0) return;
    const size_t tok0 = (size_t)s.first + begin + t0;
    const float* S = block_state + ((size_t)(b.rank - 1) * H + h) * d * E;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const bool vec = E % 4 == 0;
    f32x2 acc[4][2];
#pragma unroll
    for (int r = 0; r < 4; r++) acc[r][0] = acc[r][1] = mm_pair(0.f, 0.f);
    for (int k0 = 0; k0 < d; k0 += LA_TK) {
        __syncthreads();
#pragma unroll
        for (int j = 0; j < LA_TT * LA_TK / 256; j++) {
            const int i = threadIdx.x + j * 256, t = i / LA_TK, k = i % LA_TK;
            q_s[k][t] = (t < nt && k0 + k < d) ? qa[(tok0 + t) * H * d + (size_t)h * d + k0 + k] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < LA_TK * LA_TC / 1024; j++) {
            const int i = threadIdx.x + j * 256, k = i / (LA_TC / 4), c = i % (LA_TC / 4) * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            const float* row = S + (size_t)(k0 + k) * E + c0 + c;
            if (k0 + k < d) {
                if (vec && c0 + c < E) v = *reinterpret_cast<const float4*>(row);
                else {
                    if (c0 + c < E) v.x = row[0];
                    if (c0 + c + 1 < E) v.y = row[1];
                    if (c0 + c + 2 < E) v.z = row[2];
                    if (c0 + c + 3 < E) v.w = row[3];
                }
            }
            *reinterpret_cast<float4*>(&S_s[k][c]) = v;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < LA_TK; k++) {
            const ulonglong2 sv = *reinterpret_cast<const ulonglong2*>(&S_s[k][tx * 4]);
            const float4 qv = *reinterpret_cast<const float4*>(&q_s[k][ty * 4]);
            const float qq[4] = {qv.x, qv.y, qv.z, qv.w};
#pragma unroll
            for (int r = 0; r < 4; r++) {
                const f32x2 q2 = mm_pair(qq[r], qq[r]);
                acc[r][0] = mm_fma2(q2, sv.x, acc[r][0]); acc[r][1] = mm_fma2(q2, sv.y, acc[r][1]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const int t = ty * 4 + r, c = c0 + tx * 4;
        if (t >= nt) continue;
        float* yr = y + (tok0 + t) * H * E + (size_t)h * E + c;
        const float2 x0 = mm_unpair(acc[r][0]), x1 = mm_unpair(acc[r][1]);
        if (c < E) yr[0] += x0.x;
        if (c + 1 < E) yr[1] += x0.y;
        if (c + 2 < E) yr[2] += x1.x;
        if (c + 3 < E) yr[3] += x1.y;
    }
}

// grid (segments, slices of e, heads), a head's slices one cluster; 256 threads: thread (cv, row group) has VEC columns and
// every groups-th row.  Ps: columns a slice (a multiple of VEC, 256 / (Ps / VEC) row groups).
#define LA_STEP_THREADS 256
template <typename T, int VEC, bool CHANNEL>
__global__ void __launch_bounds__(LA_STEP_THREADS) la_step_kernel(const T* u, LAShape sh, const float* a1, const T* __restrict__ a2,
                                                                  const float* __restrict__ a_bias, int rank, float inv_tau,
                                                                  const MMSegment* __restrict__ segs, float* state, long long state_stride,
                                                                  const float* __restrict__ gain, T* __restrict__ out, float eps, int Ps) {
    extern __shared__ __align__(16) float mm_smem[];
    __shared__ float scratch[32];
    __shared__ float slice_ss;                 // this slice's sum of squares, read by the head's other slices
    const int H = sh.H, d = sh.d, E = sh.E, tid = threadIdx.x;
    const int cols = Ps / VEC, groups = LA_STEP_THREADS / cols;
    float* q_s = mm_smem;                      // [d]
    float* k_s = q_s + d;                      // [d]
    float* a_s = k_s + d;                      // [d]
    float* o_s = a_s + d;                      // [groups][Ps]
    float* a1_s = o_s + groups * Ps;           // [rank]
    pdl_launch_dependents();
    pdl_wait(KID_LINEAR_ATT);
    const MMSegment s = segs[blockIdx.x];
    if (s.count <= 0) return;                  // (a head's slices share the segment: the whole cluster leaves)
    const int h = blockIdx.z, p0 = blockIdx.y * Ps;
    const int cv = tid % cols, grp = tid / cols, e = p0 + cv * VEC;
    const bool live = grp < groups && e < E;
    float* S = state + (size_t)s.slot * state_stride + (size_t)h * d * E;
    cg::cluster_group cluster = cg::this_cluster();
    for (int tt = 0; tt < s.count; tt++) {
        const size_t tok = (size_t)s.first + tt;
        const T* row = u + tok * sh.u_stride;
        const float position = (float)(s.before + tt);
        const bool fresh = s.before + tt == 0;
        if (CHANNEL) {
            for (int r = tid; r < rank; r += LA_STEP_THREADS) a1_s[r] = a1[tok * rank + r];
            __syncthreads();
        }
        for (int n = tid; n < d; n += LA_STEP_THREADS) {
            q_s[n] = la_entry(row + sh.q_off + (size_t)h * d, n, sh, position, sh.q_scale);
            k_s[n] = la_entry(row + sh.k_off + (size_t)h * d, n, sh, position, sh.k_scale);
            a_s[n] = CHANNEL ? la_channel_decay(a2 + ((size_t)h * d + n) * rank, a1_s, a_bias[h * d + n], rank, inv_tau) : sh.decay[h];
        }
        float v[VEC], o[VEC];
#pragma unroll
        for (int x = 0; x < VEC; x++) {
            v[x] = live ? to_f32(row[sh.v_off + (size_t)h * E + e + x]) : 0.f;
            o[x] = 0.f;
        }
        __syncthreads();
        if (live) {
#pragma unroll 8
            for (int n = grp; n < d; n += groups) {
                float x[VEC];
                float* p = S + (size_t)n * E + e;
                if (fresh) {
#pragma unroll
                    for (int j = 0; j < VEC; j++) x[j] = 0.f;
                } else if constexpr (VEC == 4) {
                    const float4 f = *reinterpret_cast<const float4*>(p);
                    x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
                } else {
                    x[0] = p[0];
                }
                const float a = a_s[n], k = k_s[n], q = q_s[n];
#pragma unroll
                for (int j = 0; j < VEC; j++) { x[j] = fmaf(a, x[j], k * v[j]); o[j] = fmaf(x[j], q, o[j]); }
                if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
                else p[0] = x[0];
            }
        }
        if (grp < groups) {
#pragma unroll
            for (int x = 0; x < VEC; x++) o_s[grp * Ps + cv * VEC + x] = o[x];
        }
        __syncthreads();
        // the row groups' shares, in their order; then the head's sum of squares over its slices
        float ss = 0.f;
        for (int c = tid; c < Ps; c += LA_STEP_THREADS) {
            float acc = 0.f;
            if (p0 + c < E) for (int g = 0; g < groups; g++) acc += o_s[g * Ps + c];
            o_s[c] = acc;                      // (column c's shares are read by this thread alone)
            ss = fmaf(acc, acc, ss);
        }
        ss = block_sum(ss, scratch);
        if (gridDim.y > 1) {
            if (tid == 0) slice_ss = ss;
            cluster.sync();
            ss = 0.f;
            for (int r = 0; r < (int)gridDim.y; r++) ss += *cluster.map_shared_rank(&slice_ss, r);       // in the order of the slices
            cluster.sync();                    // (nobody leaves, or overwrites its sum, while it may still be read)
        }
        const float inv = 1.0f / sqrtf(ss / (float)E + eps);
        for (int c = tid; c < Ps; c += LA_STEP_THREADS) {
            if (p0 + c >= E) continue;
            const size_t he = (size_t)h * E + p0 + c;
            const float z = to_f32(row[sh.g_off + he]);
            out[tok * H * E + he] = from_f32<T>(o_s[c] * inv * (gain ? gain[p0 + c] : 1.0f) * mm_silu(z));
        }
        __syncthreads();
    }
}

struct LAScan { int npt, parts, Ps, slices, threads, ck, L; size_t smem; };

// Rows a thread: 16, fewer where the state is so small that a CTA would have few threads; columns a CTA: up to 64.
static int la_scan_shape(int H, int d, int E, int n_tokens, int max_segment_tokens, bool channel, LAScan* o) {
    int npt = 16, Ps = LA_COLS;
    while (Ps < E && Ps < 64) Ps *= 2;
    int parts = (d + npt - 1) / npt;
    while (npt > 4 && Ps / LA_COLS * parts < 128) { npt /= 2; parts = (d + npt - 1) / npt; }
    while (Ps > LA_COLS && Ps / LA_COLS * parts > 256) Ps /= 2;
    if (Ps / LA_COLS * parts > 256) return PLLM_ERR_LIMIT;
    o->npt = npt; o->parts = parts; o->Ps = Ps; o->slices = (E + Ps - 1) / Ps;
    o->threads = (Ps / LA_COLS * parts + 31) / 32 * 32;
    int ck = 16;
    auto smem_of = [&](int c) { return ((size_t)c * ((channel ? 3 : 2) * npt * parts + Ps + parts * Ps) + npt * parts + 64) * sizeof(float); };
    while (ck > 1 && smem_of(ck) > 72 * 1024) ck /= 2;
    o->ck = ck; o->smem = smem_of(ck);
    if (o->smem > 200 * 1024) return PLLM_ERR_LIMIT;
    // blocks of tokens for four CTAs an SM, but none shorter than 64 tokens (a 2048-token prompt, retention of 4 x 128 x 256 /
    // gated linear attention of 8 x 128 x 128, all kernels of the mixer, us: two CTAs an SM 110 / 160, three 124 / 150, four 102 / 139)
    int want = 4 * sm_count() / (H * o->slices);
    if (want < 1) want = 1;
    int L = ((n_tokens + want - 1) / want + 31) / 32 * 32;
    if (L < 64) L = 64;
    if (max_segment_tokens > 0 && L > max_segment_tokens) L = max_segment_tokens;
    o->L = L;
    return PLLM_OK;
}

static inline bool la_several(const LAScan& s, int n_tokens, int max_segment_tokens) {
    return (max_segment_tokens > 0 ? max_segment_tokens : n_tokens) > s.L;
}

PLLM_EXPORT long long pllm_linear_attention_state_floats(int H, int d, int E) { return (long long)H * d * E; }

// Float scratch of a step's recurrence (no decoded-tokens form): alpha (per entry only), decayed queries, block states and
// block decays.  0: none needed.
PLLM_EXPORT long long pllm_linear_attention_scratch_floats(int n_tokens, int max_segment_tokens, int H, int d, int E, int channel) {
    LAScan sc;
    if (la_scan_shape(H, d, E, n_tokens, max_segment_tokens, channel != 0, &sc) != PLLM_OK) return 0;
    long long n = channel ? ((long long)n_tokens * H * d + 3) / 4 * 4 : 0;
    if (la_several(sc, n_tokens, max_segment_tokens)) {
        const long long blocks = 2LL * n_tokens / sc.L + 2;
        n += ((long long)n_tokens * H * d + 3) / 4 * 4 + blocks * H * d * (E + 1);
    }
    return n;
}

// u: [tokens, u_stride] of the compute dtype with q (H d) at q_off, k (H d) at k_off, v (H e) at v_off and the gate (H e) at
// g_off; decay: H floats, or null: a1 [tokens, rank] float, a2 [H d, rank] of the compute dtype, a_bias [H d] float, inv_tau.
// gain: e floats or null.  scratch: as asked for above; y_buf: [tokens, H e] float (both unused when every segment has one
// token: max_segment_tokens 1); rope: the step's cos and sin (pllm_rope_table; the other steps form theirs from inv_freq); out: [tokens, H e] of the compute dtype.
PLLM_EXPORT int pllm_linear_attention_mix(int dtype, const void* u, int u_stride, int q_off, int k_off, int v_off, int g_off, float q_scale,
                                          float k_scale, int rot, const float* inv_freq, const float* rope, const float* decay, const float* a1,
                                          const void* a2, const float* a_bias, int rank, float inv_tau, const float* gain, const int* segs,
                                          int n_segs, int max_segment_tokens, float* state, long long state_stride, float* scratch,
                                          float* y_buf, void* out, int n_tokens, int H, int d, int E, float eps, cudaStream_t stream) {
    if (n_tokens <= 0 || n_segs <= 0) return PLLM_OK;
    if (H <= 0 || d <= 0 || E <= 0 || rot < 0 || rot > d || rot % 2 || (rot && !inv_freq)) return PLLM_ERR_SIZE;
    if (state_stride < (long long)H * d * E || q_off + H * d > u_stride || k_off + H * d > u_stride || v_off + H * E > u_stride ||
        g_off + H * E > u_stride) return PLLM_ERR_SIZE;
    const bool channel = decay == nullptr;
    if (channel && (!a1 || !a2 || !a_bias || rank < 1)) return PLLM_ERR_SIZE;
    if (channel && rank > LA_MAX_RANK) return PLLM_ERR_LIMIT;
    LAShape sh = {H, d, E, q_off, k_off, v_off, g_off, u_stride, q_scale, k_scale, rot, inv_freq, decay};
    const MMSegment* sg = (const MMSegment*)segs;
    if (max_segment_tokens == 1) {
        // columns a slice: all of them, fewer (at most eight slices, one cluster) while SMs are left without a CTA
        const int VEC = (E % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0) ? 4 : 1;
        int slices = 1;
        while (slices < 8 && (long long)n_segs * H * slices * 2 <= sm_count() && E / (slices * 2) >= 8 * VEC) slices *= 2;
        int Ps = 1;
        while (Ps * slices < E) Ps *= 2;
        if (Ps < VEC) Ps = VEC;
        while (slices < 8 && Ps / VEC > LA_STEP_THREADS) { slices *= 2; Ps /= 2; }
        if (Ps / VEC > LA_STEP_THREADS) return PLLM_ERR_LIMIT;
        const int groups = LA_STEP_THREADS / (Ps / VEC);
        const size_t smem = ((size_t)3 * d + (size_t)groups * Ps + (channel ? rank : 0)) * sizeof(float);
        if (smem > 200 * 1024) return PLLM_ERR_LIMIT;
        PLLM_DISPATCH_DTYPE(dtype, {
#define LA_STEP(V, C) do { \
            if (smem > 48 * 1024) cudaFuncSetAttribute(la_step_kernel<T, V, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            launch_chained_cluster_y(la_step_kernel<T, V, C>, dim3(n_segs, slices, H), dim3(LA_STEP_THREADS), smem, stream, slices, \
                                     (const T*)u, sh, a1, (const T*)a2, a_bias, rank, inv_tau, sg, state, state_stride, gain, (T*)out, \
                                     eps, Ps); } while (0)
            if (VEC == 4) { if (channel) LA_STEP(4, true); else LA_STEP(4, false); }
            else { if (channel) LA_STEP(1, true); else LA_STEP(1, false); }
        });
        return launch_status();
    }
    LAScan sc;
    const int rc = la_scan_shape(H, d, E, n_tokens, max_segment_tokens, channel, &sc);
    if (rc != PLLM_OK) return rc;
    if (!y_buf || (rot && !rope)) return PLLM_ERR_SIZE;
    const bool several = la_several(sc, n_tokens, max_segment_tokens);
    if ((several || channel) && !scratch) return PLLM_ERR_SIZE;
    const size_t per = ((size_t)n_tokens * H * d + 3) / 4 * 4;
    float* alpha = channel ? scratch : nullptr;
    float* qa = several ? scratch + (channel ? per : 0) : nullptr;
    const long long blocks = 2LL * n_tokens / sc.L + 2;
    float* bs = several ? qa + per : nullptr;
    float* bd = several ? bs + blocks * H * d * E : nullptr;
    const int grid_blocks = n_segs + n_tokens / sc.L;
    PLLM_DISPATCH_DTYPE(dtype, {
        if (channel)
            launch_chained(channel_decay_kernel<T>, dim3((n_tokens + LA_DECAY_TOKENS - 1) / LA_DECAY_TOKENS, (H * d + 127) / 128), dim3(128),
                           LA_DECAY_TOKENS * ((rank + 15) / 16 * 16) * sizeof(float), stream, a1, (const T*)a2, a_bias, alpha, n_tokens, H * d,
                           rank, inv_tau);
#define LA_SCAN(N, C) do { \
            if (sc.smem > 48 * 1024) cudaFuncSetAttribute(la_scan_kernel<T, N, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sc.smem); \
            launch_chained(la_scan_kernel<T, N, C>, dim3(grid_blocks, H, sc.slices), dim3(sc.threads), sc.smem, stream, (const T*)u, sh, \
                           (const float2*)rope, (const float*)alpha, sg, n_segs, state, state_stride, y_buf, bs, bd, qa, sc.Ps, sc.parts, sc.ck, sc.L); } while (0)
#define LA_SCAN_N(N) do { if (channel) LA_SCAN(N, true); else LA_SCAN(N, false); } while (0)
        if (sc.npt == 4) LA_SCAN_N(4); else if (sc.npt == 8) LA_SCAN_N(8); else LA_SCAN_N(16);
        if (several) {
            launch_chained(la_block_states_kernel, dim3(n_segs, H, (unsigned)(((long long)d * E + 255) / 256)), dim3(256), 0, stream, sg, n_segs,
                           state, state_stride, bs, (const float*)bd, H, d, E, sc.L);
            const int col_tiles = (E + LA_TC - 1) / LA_TC;
            launch_chained(la_block_outputs_kernel, dim3(grid_blocks, H * col_tiles, (sc.L + LA_TT - 1) / LA_TT), dim3(256), 0, stream, sg,
                           n_segs, (const float*)qa, (const float*)bs, y_buf, H, d, E, sc.L, col_tiles);
        }
        launch_head_norm_gate<T>(y_buf, nullptr, (const T*)u + g_off, u_stride, gain, out, n_tokens, H, E, 0, 1, eps, stream);
    });
    return launch_status();
}

PLLM_TRACE_EXPORT(linear_attention)
