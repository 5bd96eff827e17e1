// The gated delta rule with a decay a key entry: a recurrent mixer whose state is one matrix a head, S (d x e: key entries by
// value entries), carried from token to token in float for every request (a state slot), between its projections.
//
//   q, k, v   pass a short causal convolution a channel (no bias) and silu; q and k become unit vectors a head
//             (x / sqrt(sum x^2 + 1e-6)), q times d^(-1/2); head h uses q/k head h / (H / G)
//   decay     g = exp(-exp(A_log_h) softplus(W_a2 a1 + dt_bias)), one number a key entry of every head; a1 a short float vector
//   step      S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q           beta = sigmoid(b_raw), one a head
//   behind    each head's o over its root mean square, times a gain shared by the heads, times sigmoid of a gate
//   slot      [H * d * e | taps * channels: the convolution's inputs, that of position p in row p mod taps].  One row more than
//             the convolution reaches back to, so that a token's own input overwrites none that the same token still reads.
//
// A step is a list of segments {first token, tokens, tokens before, state slot} on the device; grids are sized by the list's
// capacity and a segment of no tokens does nothing, so a captured step replays for any step that fits.
//
// Portions of prompts: FOUR tokens are taken in one go.  With P_i the product of a block's first i decays (entry by entry) and
// S the state at its start,
//     u_i = beta_i (v_i - S^T (P_i k_i) - sum over j < i of u_j (k_j . (P_i / P_j) k_i))
//     o_i =               S^T (P_i q_i) + sum over j <= i of u_j (k_j . (P_i / P_j) q_i)
//     S  <- diag(P_4) S + sum over j of ((P_4 / P_j) k_j) u_j^T
// where P_i / P_j is formed as the product of the decays between, so nothing is ever divided by a decay.
//   delta_prepare_kernel   for every run of sixteen tokens and head: convolution, unit vectors, decays, then the vectors and
//                          scalars above, as one record that the scan copies as it lies
//   delta_blocks_kernel    the recurrence: a thread holds 4 NQ rows of two columns of S in registers; the threads of a column are
//                          neighbours in a warp, take their shares of the eight products with S and meet once for four tokens
//   head_norm_gate         the norm and the gate
// Decoded tokens: delta_step_kernel does everything between the projections.  A CTA a (request, head, slice of columns) has its
// part of S in registers before it waits for the products; a head's slices are one cluster and meet for the head's root mean
// square.  Columns never meet otherwise, so outputs do not depend on how they are shared out; where a prompt was cut decides
// only the order of a few float sums.
#include <cooperative_groups.h>

#include "matrix_memory.cuh"

namespace cg = cooperative_groups;

enum : int { KID_DELTA_RULE = 140 };

#define DR_RUN 16              // tokens of a record
#define DR_BLOCK 4             // tokens taken in one go
#define DR_MAX_TAPS 16
#define DR_MAX_RANK 256        // entries of a1, and of the gate's short vector
#define DR_COLS 2              // columns a thread holds

struct DRShape {
    int H, G, d, E, taps;
    int channels;              // q (G d) | k (G d) | v (H e): the first columns of the projection
    int u_stride;
    int dp;                    // d rounded up to what the scan's threads hold
    long long state_stride;
};

// the convolution's input of channel ch, r tokens behind the segment's first (negative: from the slot; before the start: zero)
template <typename T>
__device__ __forceinline__ float dr_input(const T* u, const DRShape& sh, const MMSegment& s, const float* ring, int r, int ch) {
    if (r >= 0) return to_f32(u[(size_t)(s.first + r) * sh.u_stride + ch]);
    const int pos = s.before + r;
    return pos >= 0 ? ring[(size_t)(pos % sh.taps) * sh.channels + ch] : 0.f;
}

// row . vec for a row of the compute dtype (rank entries) and a float vector in shared memory
template <typename T>
__device__ __forceinline__ float dr_dot(const T* __restrict__ row, const float* vec, int rank, bool vectors) {
    float z = 0.f;
    if (vectors) {
        constexpr int N = Vec16<T>::N;
        for (int r = 0; r < rank; r += N) {
            Vec16<T> w;
            w.load(row + r);
            float f[N];
            w.unpack(f);
#pragma unroll
            for (int k = 0; k < N; k++) z = fmaf(f[k], vec[r + k], z);
        }
    } else {
        for (int r = 0; r < rank; r++) z = fmaf(to_f32(row[r]), vec[r], z);
    }
    return z;
}

// A block's part of a record: P k [4][dp] | P q [4][dp] | (P_4 / P) k [4][dp] | P_4 [dp] | k . k scalars [4][4] (below the
// diagonal, zeros elsewhere) | k . q scalars [4][4] (on and below it) | beta [4]
__host__ __device__ __forceinline__ int dr_block_floats(int dp) { return 13 * dp + 36; }
__host__ __device__ __forceinline__ int dr_record_floats(int dp) { return DR_RUN / DR_BLOCK * dr_block_floats(dp); }

// grid (runs of the step's segments, heads), 128 threads.  The scan behind it is not let in early: its CTAs would crowd onto the SMs
// that this kernel leaves first.  small: [tokens, small_stride] float, b_raw at 0 (H), a1 at a1_off.
template <typename T>
__global__ void __launch_bounds__(128, 5) delta_prepare_kernel(const T* u, DRShape sh, const T* __restrict__ conv_w, const float* small, int small_stride,
                                                            int a1_off, const T* __restrict__ a2, int rank, const float* __restrict__ a_log,
                                                            const float* __restrict__ dt_bias, const MMSegment* __restrict__ segs, int n_segs,
                                                            const float* state, float* __restrict__ records, float* __restrict__ v_buf) {
    extern __shared__ __align__(16) float dr_smem[];
    const int d = sh.d, dp = sh.dp, E = sh.E, padded = (rank + 15) / 16 * 16;
    float* q_s = dr_smem;                    // [DR_RUN][dp]
    float* k_s = q_s + DR_RUN * dp;
    float* g_s = k_s + DR_RUN * dp;
    float* a1_s = g_s + DR_RUN * dp;         // [DR_RUN][padded]
    float* x_s = a1_s + DR_RUN * padded;     // [DR_RUN + taps - 1][128] the convolution's inputs, a channel a thread
    const MMBlock b = mm_find_block(segs, n_segs, blockIdx.x, DR_RUN);
    if (b.seg < 0) return;
    const MMSegment s = segs[b.seg];
    const int h = blockIdx.y, kh = h / (sh.H / sh.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int t0 = b.tb * DR_RUN, nt = min(DR_RUN, s.count - t0);
    const float* ring = state + (size_t)s.slot * sh.state_stride + (size_t)sh.H * d * E;
    // rows and entries beyond the run's: keys and queries of zeros, decays of one
    if (nt < DR_RUN || dp > d)
        for (int i = tid; i < DR_RUN * dp; i += blockDim.x) { q_s[i] = 0.f; k_s[i] = 0.f; g_s[i] = 1.f; }
    pdl_wait(KID_DELTA_RULE);
    for (int i = tid; i < DR_RUN * padded; i += blockDim.x) {
        const int t = i / padded, r = i - t * padded;
        a1_s[i] = (t < nt && r < rank) ? small[(size_t)(s.first + t0 + t) * small_stride + a1_off + r] : 0.f;
    }
    // the convolutions, 128 channels at a time: q's and k's of the kv head, then v's of the head
    const int rows = DR_RUN + sh.taps - 1, chans = 2 * d + E;
    auto channel = [&](int it) { return it < d ? kh * d + it : it < 2 * d ? sh.G * d + kh * d + (it - d) : 2 * sh.G * d + h * E + (it - 2 * d); };
    constexpr int V = Vec16<T>::N;
    const bool vec = d % V == 0 && E % V == 0 && sh.u_stride % V == 0 && (reinterpret_cast<uintptr_t>(u) & 15) == 0;
    for (int c0 = 0; c0 < chans; c0 += 128) {
        __syncthreads();
        if (vec) {
#pragma unroll 4
            for (int i = tid; i < rows * (128 / V); i += 128) {
                const int j = i / (128 / V), it = c0 + i % (128 / V) * V, r = t0 + j - (sh.taps - 1);
                float f[V];
                if (it >= chans || r >= t0 + nt) {
#pragma unroll
                    for (int k = 0; k < V; k++) f[k] = 0.f;
                } else if (r >= 0) {
                    Vec16<T> v;
                    v.load(u + (size_t)(s.first + r) * sh.u_stride + channel(it));
                    v.unpack(f);
                } else {
#pragma unroll
                    for (int k = 0; k < V; k++) f[k] = dr_input(u, sh, s, ring, r, channel(it) + k);
                }
#pragma unroll
                for (int k = 0; k < V; k += 4) *reinterpret_cast<float4*>(x_s + j * 128 + it - c0 + k) = make_float4(f[k], f[k + 1], f[k + 2], f[k + 3]);
            }
        } else {
#pragma unroll 4
            for (int j = 0; j < rows; j++) {
                const int it = c0 + tid, r = t0 + j - (sh.taps - 1);
                x_s[j * 128 + tid] = (it < chans && r < t0 + nt) ? dr_input(u, sh, s, ring, r, channel(it)) : 0.f;
            }
        }
        __syncthreads();
        const int it = c0 + tid;
        if (it >= chans) continue;
        const T* wr = conv_w + (size_t)channel(it) * sh.taps;
        float acc[DR_RUN];
#pragma unroll
        for (int t = 0; t < DR_RUN; t++) acc[t] = 0.f;
        for (int j = 0; j < sh.taps; j++) {
            const float w = to_f32(wr[j]);
#pragma unroll
            for (int t = 0; t < DR_RUN; t++) acc[t] = fmaf(w, x_s[(t + j) * 128 + tid], acc[t]);
        }
        float* dst = it < d ? q_s + it : k_s + (it - d);
#pragma unroll
        for (int t = 0; t < DR_RUN; t++) {
            if (t >= nt) break;
            const float c = mm_silu(acc[t]);
            if (it < 2 * d) dst[t * dp] = c;
            else v_buf[((size_t)(s.first + t0 + t) * sh.H + h) * E + (it - 2 * d)] = c;
        }
    }
    // the decays: a thread has one key entry, its row of a2 in registers 16 entries at a time
    const float rate = -expf(a_log[h]);
    const bool vec_a = rank % V == 0 && (reinterpret_cast<uintptr_t>(a2) & 15) == 0;
    for (int n = tid; n < d; n += blockDim.x) {
        const float bias = dt_bias[h * d + n];
        float z[DR_RUN];
#pragma unroll
        for (int t = 0; t < DR_RUN; t++) z[t] = bias;
        const T* row = a2 + (size_t)(h * d + n) * rank;
        for (int r0 = 0; r0 < rank; r0 += 16) {
            float w[16];
#pragma unroll
            for (int r = 0; r < 16; r++) w[r] = !vec_a && r0 + r < rank ? to_f32(row[r0 + r]) : 0.f;
            if (vec_a) {
#pragma unroll
                for (int r = 0; r < 16; r += V) {
                    if (r0 + r >= rank) break;
                    Vec16<T> v;
                    v.load(row + r0 + r);
                    v.unpack(w + r);
                }
            }
#pragma unroll
            for (int t = 0; t < DR_RUN; t++) {
                const float4* a4 = reinterpret_cast<const float4*>(a1_s + t * padded + r0);
#pragma unroll
                for (int r = 0; r < 4; r++) {
                    const float4 v = a4[r];
                    z[t] = fmaf(w[4 * r], v.x, z[t]); z[t] = fmaf(w[4 * r + 1], v.y, z[t]);
                    z[t] = fmaf(w[4 * r + 2], v.z, z[t]); z[t] = fmaf(w[4 * r + 3], v.w, z[t]);
                }
            }
        }
#pragma unroll
        for (int t = 0; t < DR_RUN; t++)
            if (t < nt) g_s[t * dp + n] = expf(rate * mm_softplus(z[t]));
    }
    __syncthreads();
    // unit vectors: a warp a token
    const float q_scale = rsqrtf((float)d);
    for (int t = warp; t < nt; t += 4) {
        float sq = 0.f, sk = 0.f;
        for (int n = lane; n < d; n += 32) { const float a = q_s[t * dp + n], c = k_s[t * dp + n]; sq = fmaf(a, a, sq); sk = fmaf(c, c, sk); }
        sq = warp_sum(sq); sk = warp_sum(sk);
        const float iq = q_scale / sqrtf(sq + 1e-6f), ik = 1.0f / sqrtf(sk + 1e-6f);
        for (int n = lane; n < d; n += 32) { q_s[t * dp + n] *= iq; k_s[t * dp + n] *= ik; }
    }
    __syncthreads();
    float* rec = records + ((size_t)blockIdx.x * sh.H + h) * dr_record_floats(dp);
    // the scalars: warp w has block w
    {
        const int i0 = warp * DR_BLOCK;
        float kk[6], kq[10];             // (i, j): kk 10 20 21 30 31 32; kq 00 10 11 20 21 22 30 31 32 33
#pragma unroll
        for (int i = 0; i < 6; i++) kk[i] = 0.f;
#pragma unroll
        for (int i = 0; i < 10; i++) kq[i] = 0.f;
        for (int n = lane; n < d; n += 32) {
            float g[4], k[4], q[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { g[i] = g_s[(i0 + i) * dp + n]; k[i] = k_s[(i0 + i) * dp + n]; q[i] = q_s[(i0 + i) * dp + n]; }
#pragma unroll
            for (int j = 0; j < 4; j++) {
                float run = k[j];         // k_j times the decays of the tokens behind it
                kq[j * (j + 1) / 2 + j] = fmaf(run, q[j], kq[j * (j + 1) / 2 + j]);
#pragma unroll
                for (int i = j + 1; i < 4; i++) {
                    run *= g[i];
                    kk[i * (i - 1) / 2 + j] = fmaf(run, k[i], kk[i * (i - 1) / 2 + j]);
                    kq[i * (i + 1) / 2 + j] = fmaf(run, q[i], kq[i * (i + 1) / 2 + j]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 6; i++) kk[i] = warp_sum(kk[i]);
#pragma unroll
        for (int i = 0; i < 10; i++) kq[i] = warp_sum(kq[i]);
        float* sc = rec + (size_t)warp * dr_block_floats(dp) + 13 * dp;
        float mine = 0.f;
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) {
                if (lane == i * 4 + j) mine = j < i ? kk[i * (i - 1) / 2 + (j < i ? j : 0)] : 0.f;
                if (lane == 16 + i * 4 + j) mine = j <= i ? kq[i * (i + 1) / 2 + (j <= i ? j : 0)] : 0.f;
            }
        sc[lane] = mine;
        if (lane < 4) sc[32 + lane] = i0 + lane < nt ? mm_sigmoid(small[(size_t)(s.first + t0 + i0 + lane) * small_stride + h]) : 0.f;
    }
    // the vectors
    for (int i = tid; i < DR_RUN / DR_BLOCK * dp; i += blockDim.x) {
        const int blk = i / dp, n = i - blk * dp;
        float* r = rec + (size_t)blk * dr_block_floats(dp) + n;
        float g[4], k[4], run = 1.f;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int o = (blk * DR_BLOCK + j) * dp + n;
            g[j] = g_s[o]; k[j] = k_s[o];
            run *= g[j];
            r[j * dp] = run * k[j];
            r[(4 + j) * dp] = run * q_s[o];
        }
        r[12 * dp] = run;
        run = 1.f;
#pragma unroll
        for (int j = 3; j >= 0; j--) { r[(8 + j) * dp] = run * k[j]; run *= g[j]; }
    }
}

__device__ __forceinline__ void dr_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void dr_copy4(float* dst, const float* src, bool valid) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(valid ? 4 : 0));
}

// PARTS neighbouring lanes hold shares of the same sixteen sums: afterwards each holds R = max(16 / PARTS, 1) whole ones, in
// val[0 .. R - 1]: sums part * R + r (PARTS 32: sum part / 2, twice).
template <int PARTS>
__device__ __forceinline__ void dr_meet(float (&val)[16], int part) {
#pragma unroll
    for (int m = PARTS / 2, n = 16; m > 0; m /= 2) {
        if (n > 1) {
            n /= 2;
            const bool up = (part & m) != 0;
#pragma unroll
            for (int k = 0; k < 8; k++) {
                if (k >= n) break;
                const float keep = up ? val[k + n] : val[k], send = up ? val[k] : val[k + n];
                val[k] = keep + __shfl_xor_sync(0xffffffffu, send, m);
            }
        } else {
            val[0] += __shfl_xor_sync(0xffffffffu, val[0], m);
        }
    }
}

// grid (segments, heads, slices of e).  u is read for the convolution's last inputs only (bf16: its dtype).  Thread (columns p0 + 2 cg, p0 + 2 cg + 1; part): rows (j PARTS + part) 4 ... + 3, j < NQ.
template <int PARTS, int NQ>
__global__ void __launch_bounds__(256, 1) delta_blocks_kernel(const void* u, int is_bf16, DRShape sh, const float* records, const float* v_buf,
                                                           const MMSegment* __restrict__ segs, int n_segs, float* state,
                                                           float* __restrict__ y, int Ps) {
    extern __shared__ __align__(16) float dr_smem[];
    constexpr int R = PARTS >= 16 ? 1 : 16 / PARTS;
    constexpr int dp = PARTS * NQ * 4, RB = 13 * dp + 36, RR = DR_RUN / DR_BLOCK * RB;        // (dr_padded, dr_block_floats, dr_record_floats)
    const int H = sh.H, d = sh.d, E = sh.E;
    const int STAGE = RR + DR_RUN * Ps;              // a record, then the run's values [16][Ps]
    pdl_launch_dependents();
    const MMSegment s = segs[blockIdx.x];
    if (s.count <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31, part = tid % PARTS;
    const int h = blockIdx.y, p0 = blockIdx.z * Ps, cl = tid / PARTS * DR_COLS, e = p0 + cl;
    int first_run = 0;
    for (int base = 0; base < (int)blockIdx.x; base += 32) {
        const int i = base + lane;
        const int c = i < (int)blockIdx.x ? segs[i].count : 0;
        first_run += __reduce_add_sync(0xffffffffu, c > 0 ? (c + DR_RUN - 1) / DR_RUN : 0);
    }
    float* S = state + (size_t)s.slot * sh.state_stride + (size_t)h * d * E;
    f32x2 st[DR_COLS][NQ * 2];
    pdl_wait(KID_DELTA_RULE);
#pragma unroll
    for (int j = 0; j < NQ; j++)
#pragma unroll
        for (int c = 0; c < DR_COLS; c++) {
            float x[4];
#pragma unroll
            for (int r = 0; r < 4; r++) {
                const int n = (j * PARTS + part) * 4 + r;
                x[r] = (s.before > 0 && n < d && cl + c < Ps && e + c < E) ? S[(size_t)n * E + e + c] : 0.f;
            }
            st[c][2 * j] = mm_pair(x[0], x[1]);
            st[c][2 * j + 1] = mm_pair(x[2], x[3]);
        }
    const int runs = (s.count + DR_RUN - 1) / DR_RUN;
    // where this lane's read-outs go: sums x = PARTS == 32 ? part / 2 : part * R + r, of which those from eight on are of queries
    float* yo = y + ((size_t)s.first * H + h) * E + e;
    auto fetch = [&](int run) {
        float* dst = dr_smem + (run & 1) * STAGE;
        const float* src = records + ((size_t)(first_run + run) * H + h) * RR;
        for (int i = tid * 4; i < RR; i += blockDim.x * 4) dr_copy16(dst + i, src + i);
        for (int i = tid; i < DR_RUN * Ps; i += blockDim.x) {
            const int t = i / Ps, c = i - t * Ps, tt = run * DR_RUN + t;
            const bool valid = tt < s.count && p0 + c < E;
            dr_copy4(dst + RR + i, v_buf + (valid ? ((size_t)(s.first + tt) * H + h) * E + p0 + c : 0), valid);
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    fetch(0);
    for (int run = 0; run < runs; run++) {
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();                             // the run has landed for every thread, and the one before it is no longer read
        if (run + 1 < runs) fetch(run + 1);
        const float* stage = dr_smem + (run & 1) * STAGE;
        const int nt = min(DR_RUN, s.count - run * DR_RUN);
        for (int t0 = 0; t0 < nt; t0 += DR_BLOCK) {
            const float* rec = stage + t0 / DR_BLOCK * RB;
            const float* mine = rec + part * 4;
            f32x2 acc[8][DR_COLS];
#pragma unroll
            for (int i = 0; i < 8; i++)
#pragma unroll
                for (int c = 0; c < DR_COLS; c++) acc[i][c] = mm_pair(0.f, 0.f);
#pragma unroll
            for (int j = 0; j < NQ; j++)
#pragma unroll
                for (int i = 0; i < 8; i++) {
                    const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(mine + i * dp + j * PARTS * 4);
#pragma unroll
                    for (int c = 0; c < DR_COLS; c++) {
                        acc[i][c] = mm_fma2(st[c][2 * j], a.x, acc[i][c]);
                        acc[i][c] = mm_fma2(st[c][2 * j + 1], a.y, acc[i][c]);
                    }
                }
            float val[16];                           // sum (kind, token, column): kind 0 with keys, 1 with queries
#pragma unroll
            for (int i = 0; i < 8; i++)
#pragma unroll
                for (int c = 0; c < DR_COLS; c++) {
                    const float2 x = mm_unpair(acc[i][c]);
                    val[i * 2 + c] = x.x + x.y;
                }
            dr_meet<PARTS>(val, part);
            const float* sc = rec + 13 * dp;
            const float4 m1 = *reinterpret_cast<const float4*>(sc + 4), m2 = *reinterpret_cast<const float4*>(sc + 8),
                         m3 = *reinterpret_cast<const float4*>(sc + 12), beta = *reinterpret_cast<const float4*>(sc + 32);
            float uu[4][DR_COLS];
#pragma unroll
            for (int c = 0; c < DR_COLS; c++) {
                float a[4], v[4];
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const int x = i * 2 + c;
                    a[i] = __shfl_sync(0xffffffffu, val[x % R], PARTS == 32 ? 2 * x : x / R, PARTS);
                    v[i] = cl + c < Ps ? stage[RR + (t0 + i) * Ps + cl + c] : 0.f;
                }
                uu[0][c] = beta.x * (v[0] - a[0]);
                uu[1][c] = beta.y * (v[1] - fmaf(uu[0][c], m1.x, a[1]));
                uu[2][c] = beta.z * (v[2] - fmaf(uu[1][c], m2.y, fmaf(uu[0][c], m2.x, a[2])));
                uu[3][c] = beta.w * (v[3] - fmaf(uu[2][c], m3.z, fmaf(uu[1][c], m3.y, fmaf(uu[0][c], m3.x, a[3]))));
            }
            // the next block's state
#pragma unroll
            for (int j = 0; j < NQ; j++) {
                const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(mine + 12 * dp + j * PARTS * 4);
#pragma unroll
                for (int c = 0; c < DR_COLS; c++) { st[c][2 * j] = mm_mul2(g.x, st[c][2 * j]); st[c][2 * j + 1] = mm_mul2(g.y, st[c][2 * j + 1]); }
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(mine + (8 + i) * dp + j * PARTS * 4);
#pragma unroll
                    for (int c = 0; c < DR_COLS; c++) {
                        const f32x2 u2 = mm_pair(uu[i][c], uu[i][c]);
                        st[c][2 * j] = mm_fma2(k.x, u2, st[c][2 * j]);
                        st[c][2 * j + 1] = mm_fma2(k.y, u2, st[c][2 * j + 1]);
                    }
                }
            }
            // the read-outs, by the lanes that hold their sums
#pragma unroll
            for (int r = 0; r < R; r++) {
                const int x = (PARTS == 32 ? part / 2 : part * R + r) - 8;
                if (x < 0 || (PARTS == 32 && (part & 1))) continue;
                const int i = x >> 1, c = x & 1;
                const float4 m = *reinterpret_cast<const float4*>(sc + 16 + i * 4);
                float o = val[r];
                o = fmaf(c ? uu[0][1] : uu[0][0], m.x, o); o = fmaf(c ? uu[1][1] : uu[1][0], m.y, o);
                o = fmaf(c ? uu[2][1] : uu[2][0], m.z, o); o = fmaf(c ? uu[3][1] : uu[3][0], m.w, o);
                if (t0 + i < nt && cl + c < Ps && e + c < E) yo[i * H * E + c] = o;
            }
            yo += (size_t)DR_BLOCK * H * E;
        }
    }
#pragma unroll
    for (int j = 0; j < NQ; j++)
#pragma unroll
        for (int c = 0; c < DR_COLS; c++) {
            const float2 lo = mm_unpair(st[c][2 * j]), hi = mm_unpair(st[c][2 * j + 1]);
            const float x[4] = {lo.x, lo.y, hi.x, hi.y};
#pragma unroll
            for (int r = 0; r < 4; r++) {
                const int n = (j * PARTS + part) * 4 + r;
                if (n < d && cl + c < Ps && e + c < E) S[(size_t)n * E + e + c] = x[r];
            }
        }
    // The convolution's last inputs: this CTA's value channels, and its kv head's q and k channels by the kv head's first head
    // and first slice.  The kernel that reads them has finished.
    float* ring = state + (size_t)s.slot * sh.state_stride + (size_t)H * d * E;
    const int hpg = H / sh.G, extra = (h % hpg == 0 && blockIdx.z == 0) ? 2 * d : 0, nv = min(Ps, E - p0), kh = h / hpg;
    for (int i = tid; i < nv + extra; i += blockDim.x) {
        const int ch = i < nv ? 2 * sh.G * d + h * E + p0 + i : i < nv + d ? kh * d + (i - nv) : sh.G * d + kh * d + (i - nv - d);
        for (int r = max(0, s.count - (sh.taps - 1)); r < s.count; r++)
            ring[(size_t)((s.before + r) % sh.taps) * sh.channels + ch] =
                is_bf16 ? to_f32(((const bf16*)u)[(size_t)(s.first + r) * sh.u_stride + ch]) : ((const float*)u)[(size_t)(s.first + r) * sh.u_stride + ch];
    }
}

// grid (segments, slices of e, heads), a head's slices one cluster; 256 threads: thread (cv, group) has VEC columns and NR of the
// rows, group, group + groups, ...  Ps: columns a slice (256 / (Ps / VEC) groups).  Every segment has one token at most.
// g1: [tokens, u_stride] at g1_off of the projection, the gate's short vector; g2 [H e, g_rank].
#define DR_STEP_THREADS 256
#define DR_STEP_ROWS 16          // rows a thread, where eight slices allow it (eight rows in twice the CTAs: 46 us against 31 at 64 requests of 8 x 128 x 128)
template <typename T, int VEC, int NR>
__global__ void __launch_bounds__(DR_STEP_THREADS, NR * VEC <= 64 ? 2 : 1) delta_step_kernel(
    const T* u, DRShape sh, const T* __restrict__ conv_w, const float* small, int small_stride, int a1_off, const T* __restrict__ a2, int rank,
    const float* __restrict__ a_log, const float* __restrict__ dt_bias, int g1_off, const T* __restrict__ g2, int g_rank,
    const float* __restrict__ gain, const MMSegment* __restrict__ segs, float* state, T* __restrict__ out, float eps, int Ps) {
    extern __shared__ __align__(16) float dr_smem[];
    __shared__ float scratch[3][8];
    __shared__ float slice_ss;                 // this slice's sum of squares, read by the head's other slices
    const int H = sh.H, d = sh.d, E = sh.E, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int cols = Ps / VEC, groups = DR_STEP_THREADS / cols;
    float* a1_s = dr_smem;                     // [rank up to a multiple of 4]
    float* g1_s = a1_s + (rank + 3) / 4 * 4;   // [g_rank up to a multiple of 4]
    float* q_s = g1_s + (g_rank + 3) / 4 * 4;  // [d]
    float* k_s = q_s + d;                      // [d]
    float* d_s = k_s + d;                      // [d] decays
    float* v_s = d_s + d;                      // [Ps] values, then what is written
    float* z_s = v_s + Ps;                     // [Ps] gates
    float* p_s = z_s + Ps;                     // [2][groups][Ps] shares of the products with key and query
    pdl_launch_dependents();
    const MMSegment s = segs[blockIdx.x];
    if (s.count <= 0) return;                  // (a head's slices share the segment: the whole cluster leaves)
    const int h = blockIdx.z, p0 = blockIdx.y * Ps, hpg = H / sh.G, kh = h / hpg;
    const int cv = tid % cols, grp = tid / cols, e = p0 + cv * VEC;
    const bool live = grp < groups && e < E;
    float* S = state + (size_t)s.slot * sh.state_stride + (size_t)h * d * E;
    float* ring = state + (size_t)s.slot * sh.state_stride + (size_t)H * d * E;
    // the state was left by an earlier step: it is fetched beside the end of the kernels before this one
    float st[NR][VEC];
#pragma unroll
    for (int r = 0; r < NR; r++) {
        const int n = grp + r * groups;
        const bool in = live && n < d && s.before > 0;
        if constexpr (VEC == 4) {
            const float4 f = in ? *reinterpret_cast<const float4*>(S + (size_t)n * E + e) : make_float4(0.f, 0.f, 0.f, 0.f);
            st[r][0] = f.x; st[r][1] = f.y; st[r][2] = f.z; st[r][3] = f.w;
        } else {
            st[r][0] = in ? S[(size_t)n * E + e] : 0.f;
        }
    }
    // the weights' rows do not come from the kernels before either
    for (int i = tid; i < d + Ps; i += DR_STEP_THREADS) {
        const char* row = i < d ? (const char*)(a2 + (size_t)(h * d + i) * rank) : (const char*)(g2 + (size_t)(h * E + min(p0 + i - d, E - 1)) * g_rank);
        for (int o = 0; o < (i < d ? rank : g_rank) * (int)sizeof(T); o += 128) asm volatile("prefetch.global.L2 [%0];\n" ::"l"(row + o));
    }
    pdl_wait(KID_DELTA_RULE);
    const size_t tok = s.first;
    for (int r = tid; r < rank; r += DR_STEP_THREADS) a1_s[r] = small[tok * small_stride + a1_off + r];
    for (int r = tid; r < g_rank; r += DR_STEP_THREADS) g1_s[r] = to_f32(u[tok * sh.u_stride + g1_off + r]);
    const bool keeps = h % hpg == 0 && blockIdx.y == 0;       // whose inputs go to the slot: its kv head's q and k (values: everybody's own)
    for (int i = tid; i < 2 * d + Ps; i += DR_STEP_THREADS) {
        const int c = i - 2 * d;
        if (c >= 0 && p0 + c >= E) { v_s[c] = 0.f; continue; }
        const int ch = i < d ? kh * d + i : i < 2 * d ? sh.G * d + kh * d + (i - d) : 2 * sh.G * d + h * E + p0 + c;
        float acc = 0.f;
#pragma unroll 4
        for (int j = 0; j < sh.taps; j++)
            acc = fmaf(to_f32(conv_w[(size_t)ch * sh.taps + j]), dr_input(u, sh, s, ring, j - (sh.taps - 1), ch), acc);
        acc = mm_silu(acc);
        if (i < d) q_s[i] = acc; else if (i < 2 * d) k_s[i - d] = acc; else v_s[c] = acc;
        // (nobody reads this row of the ring for this token)
        if (sh.taps > 1 && (c >= 0 || keeps)) ring[(size_t)(s.before % sh.taps) * sh.channels + ch] = to_f32(u[tok * sh.u_stride + ch]);
    }
    __syncthreads();
    const float rate = -expf(a_log[h]);
    const bool vec_a = rank % Vec16<T>::N == 0 && (reinterpret_cast<uintptr_t>(a2) & 15) == 0;
    const bool vec_g = g_rank % Vec16<T>::N == 0 && (reinterpret_cast<uintptr_t>(g2) & 15) == 0;
    float sq = 0.f, sk = 0.f, kq = 0.f;
    for (int i = tid; i < d + Ps; i += DR_STEP_THREADS) {
        if (i >= d) {
            if (p0 + i - d < E) z_s[i - d] = mm_sigmoid(dr_dot(g2 + (size_t)(h * E + p0 + i - d) * g_rank, g1_s, g_rank, vec_g));
            continue;
        }
        d_s[i] = expf(rate * mm_softplus(dr_dot(a2 + (size_t)(h * d + i) * rank, a1_s, rank, vec_a) + dt_bias[h * d + i]));
        const float a = q_s[i], b = k_s[i];
        sq = fmaf(a, a, sq); sk = fmaf(b, b, sk); kq = fmaf(a, b, kq);
    }
    sq = warp_sum(sq); sk = warp_sum(sk); kq = warp_sum(kq);
    if (lane == 0) { scratch[0][warp] = sq; scratch[1][warp] = sk; scratch[2][warp] = kq; }
    __syncthreads();
    sq = sk = kq = 0.f;
#pragma unroll
    for (int w = 0; w < DR_STEP_THREADS / 32; w++) { sq += scratch[0][w]; sk += scratch[1][w]; kq += scratch[2][w]; }
    const float iq = rsqrtf((float)d) / sqrtf(sq + 1e-6f), ik = 1.0f / sqrtf(sk + 1e-6f);
    kq *= iq * ik;
    float pa[VEC], pb[VEC];
#pragma unroll
    for (int x = 0; x < VEC; x++) pa[x] = pb[x] = 0.f;
#pragma unroll
    for (int r = 0; r < NR; r++) {
        const int n = grp + r * groups;
        if (n >= d || grp >= groups) break;
        const float g = d_s[n], k = k_s[n] * ik, q = q_s[n] * iq;
#pragma unroll
        for (int x = 0; x < VEC; x++) {
            st[r][x] *= g;
            pa[x] = fmaf(st[r][x], k, pa[x]); pb[x] = fmaf(st[r][x], q, pb[x]);
        }
    }
    if (grp < groups) {
#pragma unroll
        for (int x = 0; x < VEC; x++) { p_s[grp * Ps + cv * VEC + x] = pa[x]; p_s[(groups + grp) * Ps + cv * VEC + x] = pb[x]; }
    }
    __syncthreads();
    // a thread a column: the groups' shares in their order, what is written, what is read
    const float beta = mm_sigmoid(small[tok * small_stride + h]);
    float o = 0.f, ss = 0.f;
    if (tid < Ps) {
        float a = 0.f, b = 0.f;
        for (int g = 0; g < groups; g++) { a += p_s[g * Ps + tid]; b += p_s[(groups + g) * Ps + tid]; }
        const float uu = beta * (v_s[tid] - a);
        v_s[tid] = uu;
        o = p0 + tid < E ? fmaf(uu, kq, b) : 0.f;
        ss = o * o;
    }
    ss = warp_sum(ss);
    if (lane == 0) scratch[0][warp] = ss;
    __syncthreads();
    if (live) {
        float uu[VEC];
#pragma unroll
        for (int x = 0; x < VEC; x++) uu[x] = v_s[cv * VEC + x];
#pragma unroll
        for (int r = 0; r < NR; r++) {
            const int n = grp + r * groups;
            if (n >= d) break;
            const float k = k_s[n] * ik;
#pragma unroll
            for (int x = 0; x < VEC; x++) st[r][x] = fmaf(k, uu[x], st[r][x]);
            if constexpr (VEC == 4) *reinterpret_cast<float4*>(S + (size_t)n * E + e) = make_float4(st[r][0], st[r][1], st[r][2], st[r][3]);
            else S[(size_t)n * E + e] = st[r][0];
        }
    }
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < DR_STEP_THREADS / 32; w++) ss += scratch[0][w];
    if (gridDim.y > 1) {
        cg::cluster_group cluster = cg::this_cluster();
        if (tid == 0) slice_ss = ss;
        cluster.sync();
        ss = 0.f;
        for (int r = 0; r < (int)gridDim.y; r++) ss += *cluster.map_shared_rank(&slice_ss, r);       // in the order of the slices
        cluster.sync();                        // (nobody leaves while its sum may still be read)
    }
    if (tid < Ps && p0 + tid < E) out[tok * H * E + (size_t)h * E + p0 + tid] = from_f32<T>(o / sqrtf(ss / (float)E + eps) * gain[p0 + tid] * z_s[tid]);
}

// PARTS lanes a column and NQ quads of rows a lane: as many lanes as there are quads, up to a warp.
static int dr_scan_rows(int d, int* parts, int* nq) {
    int p = 1;
    while (p < 32 && p * 4 < d) p *= 2;
    int q = 1;
    while (q * p * 4 < d) q *= 2;
    *parts = p; *nq = q;
    return q > 4 ? PLLM_ERR_LIMIT : PLLM_OK;
}
static int dr_padded(int d) {
    int p, q;
    return dr_scan_rows(d, &p, &q) == PLLM_OK ? p * q * 4 : 0;
}

PLLM_EXPORT long long pllm_channel_delta_state_floats(int H, int G, int d, int E, int taps) {
    return (long long)H * d * E + (taps > 1 ? (long long)taps * (2 * G * d + H * E) : 0);
}

// Float scratch of a step with portions of prompts: the records of every run and head.
PLLM_EXPORT long long pllm_channel_delta_record_floats(int n_tokens, int n_segs, int H, int d) {
    const int dp = dr_padded(d);
    return dp ? (long long)(n_segs + n_tokens / DR_RUN) * H * dr_record_floats(dp) : 0;
}

// u: [tokens, u_stride] of the compute dtype, q (G d) | k (G d) | v (H e) in its first columns and (decoded tokens) the gate's
// short vector at g1_off; conv_w: [2 G d + H e, taps] of the same; small: [tokens, small_stride] float, b_raw (H) at 0 and a1
// (rank) at a1_off; a2: [H d, rank], g2: [H e, g_rank] of the compute dtype; a_log: H floats; dt_bias: H d; gain: e.
// gate: [tokens, H e] of the compute dtype, the gate's logits (portions of prompts; decoded tokens form them from g1 and g2).
// records, v_buf ([tokens, H e]) and y_buf ([tokens, H e]): float scratch, unused when every segment has one token
// (max_segment_tokens 1).  out: [tokens, H e] of the compute dtype.
PLLM_EXPORT int pllm_channel_delta_mix(int dtype, const void* u, int u_stride, const void* conv_w, const float* small, int small_stride, int a1_off,
                                       const void* a2, int rank, const float* a_log, const float* dt_bias, int g1_off, const void* g2, int g_rank,
                                       const void* gate, const float* gain, const int* segs, int n_segs, int max_segment_tokens, float* state,
                                       long long state_stride, float* records, float* v_buf, float* y_buf, void* out, int n_tokens, int H, int G,
                                       int d, int E, int taps, float eps, cudaStream_t stream) {
    if (n_tokens <= 0 || n_segs <= 0) return PLLM_OK;
    if (H <= 0 || G <= 0 || H % G || d <= 0 || E <= 0 || taps < 1 || rank < 1 || g_rank < 1) return PLLM_ERR_SIZE;
    if (taps > DR_MAX_TAPS || rank > DR_MAX_RANK || g_rank > DR_MAX_RANK) return PLLM_ERR_LIMIT;
    const int channels = 2 * G * d + H * E;
    if (u_stride < channels || small_stride < a1_off + rank || a1_off < H || state_stride < pllm_channel_delta_state_floats(H, G, d, E, taps))
        return PLLM_ERR_SIZE;
    DRShape sh = {H, G, d, E, taps, channels, u_stride, dr_padded(d), state_stride};
    const MMSegment* sg = (const MMSegment*)segs;
    if (max_segment_tokens == 1) {
        if (g1_off < channels || g1_off + g_rank > u_stride || !g2) return PLLM_ERR_SIZE;
        // columns a slice: all of them, fewer (at most eight slices, one cluster) while SMs are left without a CTA or a thread
        // would hold many rows
        const int VEC = (E % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0) ? 4 : 1;
        int slices = 1;
        while (slices < 8 && (long long)n_segs * H * slices * 2 <= sm_count() && E / (slices * 2) >= 8 * VEC) slices *= 2;
        int Ps = 1;
        while (Ps * slices < E) Ps *= 2;
        if (Ps < VEC) Ps = VEC;
        auto rows = [&]() { const int groups = DR_STEP_THREADS / (Ps / VEC); return groups > 0 ? (d + groups - 1) / groups : d; };
        while (slices < 8 && Ps > VEC && (Ps > DR_STEP_THREADS || rows() > DR_STEP_ROWS)) { slices *= 2; Ps /= 2; }
        if (Ps > DR_STEP_THREADS || rows() > 32) return PLLM_ERR_LIMIT;
        const int groups = DR_STEP_THREADS / (Ps / VEC), nr = rows();
        const size_t smem = ((size_t)(rank + 3) / 4 * 4 + (g_rank + 3) / 4 * 4 + 3 * d + 2 * Ps + 2 * (size_t)groups * Ps) * sizeof(float);
        if (smem > 200 * 1024) return PLLM_ERR_LIMIT;
        PLLM_DISPATCH_DTYPE(dtype, {
#define DR_STEP(V, N) do { \
            if (smem > 48 * 1024) cudaFuncSetAttribute(delta_step_kernel<T, V, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            launch_chained_cluster_y(delta_step_kernel<T, V, N>, dim3(n_segs, slices, H), dim3(DR_STEP_THREADS), smem, stream, slices, \
                                     (const T*)u, sh, (const T*)conv_w, small, small_stride, a1_off, (const T*)a2, rank, a_log, dt_bias, g1_off, \
                                     (const T*)g2, g_rank, gain, sg, state, (T*)out, eps, Ps); } while (0)
            if (VEC == 4) { if (nr <= 4) DR_STEP(4, 4); else if (nr <= 8) DR_STEP(4, 8); else if (nr <= 16) DR_STEP(4, 16); else DR_STEP(4, 32); }
            else { if (nr <= 8) DR_STEP(1, 8); else DR_STEP(1, 32); }
        });
        return launch_status();
    }
    int parts, nq;
    const int rc = dr_scan_rows(d, &parts, &nq);
    if (rc != PLLM_OK) return rc;
    if (!records || !v_buf || !y_buf || !gate || ((uintptr_t)records & 15)) return PLLM_ERR_SIZE;
    // columns a CTA: eight warps' worth, fewer while the step's CTAs leave SMs empty
    const int per_warp = 32 / parts * DR_COLS;
    int warps = 8;
    while (warps > 1 && ((warps / 2) * per_warp >= E || (long long)n_segs * H * ((E + warps * per_warp - 1) / (warps * per_warp)) * 2 <= sm_count() + sm_count() / 8))
        warps /= 2;
    const int Ps = warps * per_warp, slices = (E + Ps - 1) / Ps;
    const size_t smem = 2 * (size_t)(dr_record_floats(sh.dp) + DR_RUN * Ps) * sizeof(float);
    const size_t psmem = ((size_t)3 * DR_RUN * sh.dp + (size_t)DR_RUN * ((rank + 15) / 16 * 16) + (size_t)(DR_RUN + taps - 1) * 128) * sizeof(float);
    if (smem > 225 * 1024 || psmem > 225 * 1024) return PLLM_ERR_LIMIT;
    PLLM_DISPATCH_DTYPE(dtype, {
        if (psmem > 48 * 1024) cudaFuncSetAttribute(delta_prepare_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)psmem);
        launch_chained(delta_prepare_kernel<T>, dim3(n_segs + n_tokens / DR_RUN, H), dim3(128), psmem, stream, (const T*)u, sh, (const T*)conv_w, small,
                       small_stride, a1_off, (const T*)a2, rank, a_log, dt_bias, sg, n_segs, (const float*)state, records, v_buf);
    });
#define DR_SCAN(P, Q) do { \
        if (smem > 48 * 1024) cudaFuncSetAttribute(delta_blocks_kernel<P, Q>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        launch_chained(delta_blocks_kernel<P, Q>, dim3(n_segs, H, slices), dim3(warps * 32), smem, stream, u, dtype == PLLM_BF16 ? 1 : 0, sh, \
                       (const float*)records, (const float*)v_buf, sg, n_segs, state, y_buf, Ps); } while (0)
    if (parts == 1) DR_SCAN(1, 1); else if (parts == 2) DR_SCAN(2, 1); else if (parts == 4) DR_SCAN(4, 1);
    else if (parts == 8) DR_SCAN(8, 1); else if (parts == 16) DR_SCAN(16, 1);
    else if (nq == 1) DR_SCAN(32, 1); else if (nq == 2) DR_SCAN(32, 2); else DR_SCAN(32, 4);
    PLLM_DISPATCH_DTYPE(dtype, {
        launch_head_norm_gate<T>(y_buf, nullptr, gate, H * E, gain, out, n_tokens, H, E, 0, 0, eps, stream);
    });
    return launch_status();
}

PLLM_TRACE_EXPORT(delta_rule)
