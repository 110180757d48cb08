// Linear recurrences with a matrix state per request and head, carried from
// token to token in float32:
//
//   retention        S_t = decay_h S_{t-1} + k_t v_t^T                      o_t = S_t^T q_t
//   delta rule       S_t = diag(w_t) S_{t-1} - (a_t * u_t)(u_t^T S_{t-1}) + k_t v_t^T
//                                                                           o_t = S_t^T r_t
//   gated memory     m_t = max(f_t + m_{t-1}, i_t)   (m_0 = 0)
//                    S_t = e^(f_t + m_{t-1} - m_t) S_{t-1} + e^(i_t - m_t) k_t v_t^T,  n_t likewise with k_t alone
//                                        o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)
//   wkv              o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_{t-1} + k_t v_t^T
//                    (the output reads the OLD state; the bonus u counts the current token only;
//                    w = exp(-exp(w_raw + w_bias)) per head, key channel and token)
//   state space     S_t = exp(-exp(A_h) dt_t) S_{t-1} + dt_t B_t x_t^T,   y_t = S_t^T C_t + D_h x_t
//                    (the selective state space recurrence in its dual, matrix-state form: x, B and C
//                    pass a short causal convolution and silu first; dt = softplus(dt_raw + bias); the
//                    heads of a group share B and C; then the gate silu(z), a root-mean-square division
//                    in equal parts of the row, a weight)
//   gated delta     S <- diag(g_t) S_{t-1}, u_t = beta_t (v_t - S^T k_t), S_t = S + k_t u_t^T, o_t = S_t^T q_t
//                    (the delta rule with a decay per head, key channel and token, g = exp(-exp(A_h)
//                    softplus(a_raw + bias)), and a write rate per head and token; q, k and v pass a short
//                    causal convolution and silu first, q and k are unit vectors; the heads of a group share
//                    q and k; the weight after the root-mean-square division is shared by all heads)
//
// S is [key dim, value dim].  Retention rotates q and k by the step's (cos, sin)
// table (pair (i, i + rot/2), the first `rot` dims) and scales k afterwards; its
// decay is one number per head.  The delta rule's decay and removal rate are per
// key channel and token: w = exp(-exp(-1/2) sigmoid(w_raw + w_bias)), a =
// sigmoid(a_raw + a_bias), u = k / sqrt(sum k^2 + 1e-6); both of its terms read the
// old state.  After the recurrence each head's o is divided by its root mean
// square (eps inside the root), optionally multiplied by a weight, gated by
// silu or sigmoid of a projection, scaled by out_scale and stored in the compute
// type for the output projection.
//
// The gated memory (the matrix memory of the xLSTM) has a log input gate i = cap tanh((x_i + b_i) / cap)
// and a log forget gate f = logsigmoid(cap tanh((x_f + b_f) / cap)) per head and token, q scaled by
// q_scale.  Its n is carried as one more value column of S whose value is 1 in every token, so that
// n_t . q_t is that column's output; the running maximum m is kept per head beside S (one copy per
// slice of value columns, so that the blocks of a head do not share a word).  The state of a slot is
// [heads][dim][v_dim + 4] (columns v_dim + 1 .. v_dim + 3 stay zero) followed by [heads][slices] of m.
//
// Everything that enters the recurrence is formed in float32 from the
// projections (which arrive in the compute type); the state never leaves float32.
//
// Convolutions are a kernel of their own before the scan (conv_run_kernel: a thread walks a run of tokens
// of one channel with its weights in registers), and the inputs a slot keeps are written after it.
//
// The general form is three kernels per step.  (1) prepare: a warp per (token, head) forms the token's vectors in
// float32 (q/r, k, and for the delta rule w, a * u, u) in a workspace; fully parallel over the
// step's tokens.  (2) scan: a block per (entry, head, slice of 32 value columns) -- the columns
// of S evolve independently -- walks the entry's tokens in order; a thread owns one column and
// at most 32 key rows of it (every P-th row) in registers (P = 1, 2, 4, 8 or 16 threads per column, neighbours in a
// warp, their partial sums met by shuffles); the token vectors come through shared memory in
// batches.  The state is read from and written back to its slot once per launch; a decoded token
// is a batch of one.  (3) finish: a warp per (token, head) divides by the root mean square,
// applies weight, gate and scale and stores in the compute type.  The order of every sum depends
// on the sizes only.
//
// Two kinds have scans of their own for the sizes that divide by four: ssd_scan_kernel (straight from the
// convolved rows, no records) and gated_delta_scan_kernel.  There a thread works on pairs of float32 and the
// shuffles of one token's sums travel while the next token is worked on.  For steps of one token per request
// ssd_token_kernel and gated_delta_token_kernel do the convolution, the state and the output in one launch.
// A scan of many tokens starts when the kernel before it has left the GPU (kipp_launch_spread): blocks that
// were placed early share few multiprocessors, and a scan lasts as long as its most crowded one.
#include "common.cuh"
#include <math.h>
#include <algorithm>

#ifndef KIPP_SSD_WIDE
#define KIPP_SSD_WIDE 1
#endif
namespace {
constexpr int MAX_CHUNK = 32;

struct ScanArgs {
    void* out; long long ld_out;           // [T, heads * v_dim] compute type
    const void* proj; long long ld_proj;   // [T, ...] compute type: the fused projections
    int q_off, k_off, v_off, g_off, a_off; // column offsets of r/q, k, v, gate, removal rate in proj
    const void* w_raw; long long ld_w;     // delta: [T, heads * dim] compute type
    const float* a_bias;                   // delta: [heads * dim]
    const float* w_bias;                   // delta: [heads * dim]
    const float* norm_w;                   // [heads * v_dim] or null
    const float* decay;                    // retention: [heads]
    const float* cos_sin; int rot;         // retention: [T, rot / 2, 2] or null
    float* state;                          // [slots, heads, dim, v_dim]
    const int* q_start; const int* slots;
    int heads, dim, v_dim, batch, entries;
    float k_scale, eps, out_scale;
    int gate;                              // 0 none, 1 silu, 2 sigmoid
    // gated memory: columns of the two gates in proj, their biases [heads], the cap, the scale of q
    int i_off, f_off;
    const float* i_bias; const float* f_bias;
    float gate_cap, q_scale;
    long long slot_stride;                 // floats per slot of `state` (0: heads * dim * v_dim)
    const float* bonus;                    // wkv: u [heads * dim]
    // state space: columns of z, of the convolved channels [x: heads * v_dim | B: groups * dim | C: groups * dim]
    // and of dt in proj; the convolution [channels, taps] with its bias; per head dt's bias, A (as its
    // logarithm) and D; the slot keeps the last taps - 1 inputs of every channel behind S
    int z_off, xbc_off, dt_off, taps, groups, norm_groups;
    const float* conv_w; const float* conv_b;
    const float* dt_bias; const float* a_log; const float* d_skip;
    const int* entry_of_token;
    // the convolved channels and where a slot keeps their last inputs (floats behind its start)
    int channels; long long kept_off;
    // gated delta rule: a_raw and g_raw float32, [T, heads * dim] and [T, heads * v_dim]
    const float* a_raw; long long ld_a; const float* g_raw; long long ld_g; int b_off;
};
enum { RETENTION = 0, DELTA_RULE = 1, GATED_MEMORY = 2, WKV = 3, SSD = 4, GATED_DELTA = 5 };
// vectors per token besides v, extra floats after them, extra value columns
template <int KIND> struct Rec {
    static constexpr int NV = KIND == DELTA_RULE ? 5 : KIND == WKV || KIND == GATED_DELTA ? 3 : 2;     // wkv: r, k, w; gated delta: q, k, g
    // after the vectors: (i, f, 0, 0), wkv's (sum u k r, 0, 0, 0), the state space's (decay, dt, 0, 0) or the gated delta rule's (beta, q . k, 0, 0)
    static constexpr int XG = KIND == GATED_MEMORY || KIND == WKV || KIND == SSD || KIND == GATED_DELTA ? 4 : 0;
    static constexpr int XV = KIND == GATED_MEMORY ? 4 : 0;     // value columns (1, 0, 0, 0) after v
};
__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }

// (1) the token vectors: one record of NV * D + V floats per (head, token), heads outermost so that
// a head's consecutive tokens are neighbours: NV = 5 (delta: r, k, w, a*u, u) or 2 (q, k), then v
template <typename T, int KIND>
__global__ void __launch_bounds__(128)
recurrent_prepare_kernel(const ScanArgs a, float* __restrict__ vec, int tokens) {
    pdl_launch_dependents();
    pdl_wait();
    constexpr bool DELTA = KIND == DELTA_RULE;
    constexpr int NV = Rec<KIND>::NV, XG = Rec<KIND>::XG, XV = Rec<KIND>::XV;
    const int lane = threadIdx.x & 31;
    const long long wg = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    if (wg >= (long long)tokens * a.heads) return;
    const size_t row = (size_t)(wg / a.heads);
    const int h = (int)(wg % a.heads), D = a.dim;
    const T* pr = static_cast<const T*>(a.proj) + row * a.ld_proj;
    const int rec = NV * D + XG + a.v_dim + XV;
    float* dst = vec + ((size_t)h * tokens + row) * rec;
    for (int c = lane; c < a.v_dim; c += 32) dst[NV * D + XG + c] = to_f32(pr[a.v_off + h * a.v_dim + c]);
    if (KIND == GATED_MEMORY) {
        if (lane < XV) dst[NV * D + XG + a.v_dim + lane] = lane == 0 ? 1.f : 0.f;
        if (lane == 0) {
            const float cap = a.gate_cap;
            dst[NV * D] = cap * tanhf((to_f32(pr[a.i_off + h]) + a.i_bias[h]) / cap);
            dst[NV * D + 1] = log_sigmoid(cap * tanhf((to_f32(pr[a.f_off + h]) + a.f_bias[h]) / cap));
            dst[NV * D + 2] = 0.f;
            dst[NV * D + 3] = 0.f;
        }
        for (int d = lane; d < D; d += 32) {
            dst[d] = to_f32(pr[a.q_off + h * D + d]) * a.q_scale;
            dst[D + d] = to_f32(pr[a.k_off + h * D + d]);
        }
    } else if (KIND == WKV) {
        const T* w_raw = static_cast<const T*>(a.w_raw);
        float bonus = 0.f;
        for (int d = lane; d < D; d += 32) {
            const int c = h * D + d;
            const float r = to_f32(pr[a.q_off + c]), k = to_f32(pr[a.k_off + c]);
            const float wr = to_f32(w_raw[row * a.ld_w + c]) + a.w_bias[c];
            dst[d] = r;
            dst[D + d] = k;
            dst[2 * D + d] = expf(-expf(wr));
            bonus = fmaf(a.bonus[c] * k, r, bonus);
        }
        bonus = warp_sum(bonus);
        if (lane < XG) dst[NV * D + lane] = lane == 0 ? bonus : 0.f;
    } else if (DELTA) {
        const T* w_raw = static_cast<const T*>(a.w_raw);
        float ss = 0.f;
        for (int d = lane; d < D; d += 32) {
            const float k = to_f32(pr[a.k_off + h * D + d]);
            ss = fmaf(k, k, ss);
        }
        ss = warp_sum(ss);
        const float inv = 1.0f / sqrtf(ss + 1e-6f);
        for (int d = lane; d < D; d += 32) {
            const int c = h * D + d;
            const float k = to_f32(pr[a.k_off + c]);
            const float u = k * inv;
            const float rate = sigmoidf_(to_f32(pr[a.a_off + c]) + a.a_bias[c]);
            const float wr = to_f32(w_raw[row * a.ld_w + c]) + a.w_bias[c];
            dst[d] = to_f32(pr[a.q_off + c]);
            dst[D + d] = k;
            dst[2 * D + d] = expf(-0.6065306597126334f * sigmoidf_(wr));
            dst[3 * D + d] = rate * u;
            dst[4 * D + d] = u;
        }
    } else {
        const int half = a.rot / 2;
        const float2* cs = a.cos_sin ? reinterpret_cast<const float2*>(a.cos_sin) + row * half : nullptr;
        for (int d = lane; d < D; d += 32) {
            const int c = h * D + d;
            float q = to_f32(pr[a.q_off + c]), k = to_f32(pr[a.k_off + c]);
            if (cs != nullptr && d < a.rot) {
                const bool low = d < half;
                const float2 t = cs[low ? d : d - half];
                const float q2 = to_f32(pr[a.q_off + h * D + (low ? d + half : d - half)]);
                const float k2 = to_f32(pr[a.k_off + h * D + (low ? d + half : d - half)]);
                // low: u cos - v sin; high: v cos + u sin (u the low half, v the high one)
                q = low ? q * t.x - q2 * t.y : q * t.x + q2 * t.y;
                k = low ? k * t.x - k2 * t.y : k * t.x + k2 * t.y;
            }
            dst[d] = q;
            dst[D + d] = k * a.k_scale;
        }
    }
}

// (2) the recurrence; raw o goes to o_raw [T, heads * v_dim] float32.  The records of a batch of
// tokens come into shared memory by asynchronous copies, the next batch while this one is walked.
constexpr int VS = 32;                     // value columns per block
__device__ __forceinline__ void load_batch(float* __restrict__ tv, float* __restrict__ vv, const float* __restrict__ rec0,
                                           int rec, int nvd, int nb, int slice, int V, bool async, int threads) {
    // rec0: the record of the batch's first token; the vectors' part [nvd] and this slice's values
    if (async) {
        const int c4 = nvd / 4;
        for (int i = threadIdx.x; i < nb * c4; i += threads) {
            const int tt = i / c4, c = i % c4;
            cp_async16(smem_address(tv + (size_t)tt * nvd + c * 4), rec0 + (size_t)tt * rec + c * 4, 16);
        }
        for (int i = threadIdx.x; i < nb * (VS / 4); i += threads) {
            const int tt = i / (VS / 4), c = i % (VS / 4), col = slice * VS + c * 4;
            const bool ok = col < V;                    // V is a multiple of 4 here: a chunk is whole or absent
            cp_async16(smem_address(vv + (size_t)tt * VS + c * 4), ok ? rec0 + (size_t)tt * rec + nvd + col : rec0, ok ? 16 : 0);
        }
    } else {
        for (int i = threadIdx.x; i < nb * nvd; i += threads) tv[i] = rec0[(size_t)(i / nvd) * rec + i % nvd];
        for (int i = threadIdx.x; i < nb * VS; i += threads) {
            const int col = slice * VS + i % VS;
            vv[i] = col < V ? rec0[(size_t)(i / VS) * rec + nvd + col] : 0.f;
        }
    }
    cp_async_commit();
}

// VEC: the head's key size is a multiple of 4: a thread's rows come in groups of four neighbours
// (rows 4 (p + P g) .. + 3), read with one 16-byte load per vector.
template <typename T, int KIND, int P, int CHUNK, bool VEC>
__global__ void __launch_bounds__(VS * P)
recurrent_scan_kernel(const ScanArgs a, const float* __restrict__ vec, float* __restrict__ o_raw, int v_slices,
                      int tokens) {
    extern __shared__ __align__(16) float smem[];
    constexpr bool DELTA = KIND == DELTA_RULE;
    constexpr int NV = Rec<KIND>::NV;
    // V counts the value columns of the state: those of v and, for the gated memory, n's and its padding
    const int D = a.dim, V = a.v_dim + Rec<KIND>::XV, TB = a.batch;
    const int nvd = NV * D + Rec<KIND>::XG, rec = nvd + V;
    // two buffers of [TB][NV][D] vectors followed by [TB][VS] values; their addresses are formed
    // from the shared base each time (a table of pointers would turn the loads into generic ones)
    const int buf_floats = TB * (nvd + VS);
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x;
    const int slice = blockIdx.x % v_slices, eh = blockIdx.x / v_slices;
    const int e = eh / a.heads, h = eh % a.heads;
    const int row0 = a.q_start[e], n_tok = a.q_start[e + 1] - row0;
    const int p = tid % P, cl = tid / P, col = slice * VS + cl;
    // the key rows of a column are dealt out to its P threads in turn (thread p has rows p, p + P, ..., or
    // groups of four rows in turn): the threads of a column then read neighbouring words of a token's
    // vectors, which no bank serves twice
    auto row_of = [p](int i) { return VEC ? 4 * (p + P * (i >> 2)) + (i & 3) : p + P * i; };
    const bool live = col < V;
    float* slot_base = a.state + (size_t)a.slots[e] * (size_t)(a.slot_stride > 0 ? a.slot_stride : (long long)a.heads * D * V);
    float* S_slot = slot_base + (size_t)h * D * V;
    // the gated memory's running maximum: this block's own copy
    float* m_slot = slot_base + (size_t)a.heads * D * V + (size_t)h * v_slices + slice;
    float m_run = KIND == GATED_MEMORY ? *m_slot : 0.f;
    const float* recs = vec + ((size_t)h * tokens + row0) * rec;
    // 16-byte copies need every record and every part of it on a 16-byte boundary
    const bool async = nvd % 4 == 0 && V % 4 == 0;

    float S[CHUNK];
#pragma unroll
    for (int i = 0; i < CHUNK; ++i) S[i] = (live && row_of(i) < D) ? S_slot[(size_t)row_of(i) * V + col] : 0.f;
    const float decay = KIND == RETENTION ? a.decay[h] : 0.f;

    load_batch(smem, smem + TB * nvd, recs, rec, nvd, min(TB, n_tok), slice, V, async, VS * P);
    int buf = 0;
    for (int t0 = 0; t0 < n_tok; t0 += TB, buf ^= 1) {
        const int nb = min(TB, n_tok - t0);
        if (t0 + TB < n_tok)
            load_batch(smem + (buf ^ 1) * buf_floats, smem + (buf ^ 1) * buf_floats + TB * nvd,
                              recs + (size_t)(t0 + TB) * rec, rec, nvd, min(TB, n_tok - t0 - TB), slice, V, async, VS * P);
        else
            cp_async_commit();
        cp_async_wait<1>();                 // this batch has landed; the next one may still be on its way
        __syncthreads();
        const float* tvb = smem + buf * buf_floats;
        const float* vvb = tvb + TB * nvd;
        for (int tt = 0; tt < nb; ++tt) {
            const float v = vvb[tt * VS + cl];
            const float* base = tvb + tt * nvd + p;
            float us = 0.f, keep = 0.f, take = 0.f;
            if (KIND == GATED_MEMORY) {
                const float gi = tvb[tt * nvd + NV * D], gf = tvb[tt * nvd + NV * D + 1];
                const float m_new = fmaxf(gf + m_run, gi);
                keep = expf(gf + m_run - m_new);
                take = expf(gi - m_new);
                m_run = m_new;
            }
            if (KIND == SSD) {
                keep = tvb[tt * nvd + NV * D];          // exp(-exp(A) dt)
                take = tvb[tt * nvd + NV * D + 1];      // dt
            }
            const float* tok = tvb + tt * nvd;
            if (DELTA) {
                if (VEC) {
#pragma unroll
                    for (int g = 0; g < CHUNK / 4; ++g) {
                        const int r = 4 * (p + P * g);
                        if (r < D) {
                            const float4 u4 = *reinterpret_cast<const float4*>(tok + 4 * D + r);
                            us = fmaf(u4.x, S[4 * g], us); us = fmaf(u4.y, S[4 * g + 1], us);
                            us = fmaf(u4.z, S[4 * g + 2], us); us = fmaf(u4.w, S[4 * g + 3], us);
                        }
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < CHUNK; ++i)
                        if (p + P * i < D) us = fmaf(base[4 * D + P * i], S[i], us);
                }
#pragma unroll
                for (int x = P / 2; x > 0; x >>= 1) us += __shfl_xor_sync(0xffffffffu, us, x);
            }
            float o = 0.f;
            if (KIND == GATED_DELTA) {
                // the decayed state meets k and q in one pass and both sums travel together; the token's own
                // write then joins the output as (q . k) u
                float kr[CHUNK], us4[4] = {0.f, 0.f, 0.f, 0.f}, os4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int i = 0; i < CHUNK; ++i)
                    if (row_of(i) < D) {
                        const float s = S[i] * tok[2 * D + row_of(i)];
                        S[i] = s;
                        kr[i] = tok[D + row_of(i)];
                        us4[i & 3] = fmaf(kr[i], s, us4[i & 3]);
                        os4[i & 3] = fmaf(tok[row_of(i)], s, os4[i & 3]);
                    }
                us = (us4[0] + us4[1]) + (us4[2] + us4[3]);
                o = (os4[0] + os4[1]) + (os4[2] + os4[3]);
#pragma unroll
                for (int x = P / 2; x > 0; x >>= 1) {
                    us += __shfl_xor_sync(0xffffffffu, us, x);
                    o += __shfl_xor_sync(0xffffffffu, o, x);
                }
                const float u = tok[NV * D] * (v - us);
#pragma unroll
                for (int i = 0; i < CHUNK; ++i)
                    if (row_of(i) < D) S[i] = fmaf(kr[i], u, S[i]);
                o = fmaf(tok[NV * D + 1], u, o);
                if (live && p == 0) o_raw[(size_t)(row0 + t0 + tt) * (a.heads * V) + h * V + col] = o;
                continue;
            }
            const float tv = take * v;                  // (gated memory, state space: the input's weight on this column's value)
            if (VEC && KIND == SSD) {
                // the state space layer's heads are tall (128 rows and more): a group's four rows are a short chain
                // of their own, and the groups' sums meet at the end (an order fixed by the sizes)
                float og[CHUNK / 4];
#pragma unroll
                for (int g = 0; g < CHUNK / 4; ++g) {
                    og[g] = 0.f;
                    const int r = 4 * (p + P * g);
                    if (r < D) {
                        const float4 q4 = *reinterpret_cast<const float4*>(tok + r);
                        const float4 k4 = *reinterpret_cast<const float4*>(tok + D + r);
                        const float s0 = fmaf(k4.x, tv, keep * S[4 * g]), s1 = fmaf(k4.y, tv, keep * S[4 * g + 1]);
                        const float s2 = fmaf(k4.z, tv, keep * S[4 * g + 2]), s3 = fmaf(k4.w, tv, keep * S[4 * g + 3]);
                        S[4 * g] = s0; S[4 * g + 1] = s1; S[4 * g + 2] = s2; S[4 * g + 3] = s3;
                        og[g] = fmaf(s3, q4.w, fmaf(s2, q4.z, fmaf(s1, q4.y, s0 * q4.x)));
                    }
                }
#pragma unroll
                for (int g = 0; g < CHUNK / 4; ++g) o += og[g];
            } else if (VEC) {
#pragma unroll
                for (int g = 0; g < CHUNK / 4; ++g) {
                    const int r = 4 * (p + P * g);
                    if (r < D) {
                        float qq[4], kk[4], ww[4], aa[4];
                        *reinterpret_cast<float4*>(qq) = *reinterpret_cast<const float4*>(tok + r);
                        *reinterpret_cast<float4*>(kk) = *reinterpret_cast<const float4*>(tok + D + r);
                        if (DELTA || KIND == WKV) *reinterpret_cast<float4*>(ww) = *reinterpret_cast<const float4*>(tok + 2 * D + r);
                        if (DELTA) *reinterpret_cast<float4*>(aa) = *reinterpret_cast<const float4*>(tok + 3 * D + r);
#pragma unroll
                        for (int j = 0; j < 4; ++j) {
                            float s;
                            if (DELTA) s = fmaf(kk[j], v, fmaf(-aa[j], us, ww[j] * S[4 * g + j]));
                            else if (KIND == GATED_MEMORY || KIND == SSD) s = fmaf(kk[j], tv, keep * S[4 * g + j]);
                            else if (KIND == WKV) s = fmaf(kk[j], v, ww[j] * S[4 * g + j]);
                            else s = fmaf(kk[j], v, decay * S[4 * g + j]);
                            o = fmaf(KIND == WKV ? S[4 * g + j] : s, qq[j], o);      // wkv reads the old state
                            S[4 * g + j] = s;
                        }
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < CHUNK; ++i) {
                    if (p + P * i < D) {
                        float s;
                        if (DELTA) s = fmaf(base[D + P * i], v, fmaf(-base[3 * D + P * i], us, base[2 * D + P * i] * S[i]));
                        else if (KIND == GATED_MEMORY || KIND == SSD) s = fmaf(base[D + P * i], tv, keep * S[i]);
                        else if (KIND == WKV) s = fmaf(base[D + P * i], v, base[2 * D + P * i] * S[i]);
                        else s = fmaf(base[D + P * i], v, decay * S[i]);
                        o = fmaf(KIND == WKV ? S[i] : s, base[P * i], o);
                        S[i] = s;
                    }
                }
            }
#pragma unroll
            for (int x = P / 2; x > 0; x >>= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
            if (KIND == WKV) o = fmaf(tok[NV * D], v, o);                   // the current token's own pair, weighted by u
            if (KIND == GATED_MEMORY && col == a.v_dim + 1) o = m_run;      // the column after n's carries m_t to the finish
            if (live && p == 0) o_raw[(size_t)(row0 + t0 + tt) * (a.heads * V) + h * V + col] = o;
        }
        __syncthreads();                    // the buffer is free for the batch after the next
    }
#pragma unroll
    for (int i = 0; i < CHUNK; ++i)
        if (live && row_of(i) < D) S_slot[(size_t)row_of(i) * V + col] = S[i];
    if (KIND == GATED_MEMORY && tid == 0) *m_slot = m_run;
}

// (3) per-head root-mean-square division, weight, gate, scale
template <typename T, int KIND>
__global__ void __launch_bounds__(128)
recurrent_finish_kernel(const ScanArgs a, const float* __restrict__ o_raw, int tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long wg = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    if (wg >= (long long)tokens * a.heads) return;
    const size_t row = (size_t)(wg / a.heads);
    const int h = (int)(wg % a.heads), V = a.v_dim;
    const int VX = V + Rec<KIND>::XV;
    const float* o = o_raw + row * (a.heads * VX) + h * VX;
    const T* proj = static_cast<const T*>(a.proj);
    T* out = static_cast<T*>(a.out);
    // the gated memory divides by max(|n . q|, e^(-m)) + 1e-6 first
    const float den = KIND == GATED_MEMORY ? 1.0f / (fmaxf(fabsf(o[V]), expf(-o[V + 1])) + 1e-6f) : 1.f;
    float ss = 0.f;
    for (int c = lane; c < V; c += 32) {
        const float y = o[c] * den;
        ss = fmaf(y, y, ss);
    }
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)V + a.eps);
    for (int c = lane; c < V; c += 32) {
        const int hc = h * V + c;
        float y = o[c] * den * inv;
        if (a.norm_w != nullptr) y *= a.norm_w[KIND == GATED_DELTA ? c : hc];
        if (a.gate != 0) {
            const float g = KIND == GATED_DELTA ? a.g_raw[row * a.ld_g + hc] : to_f32(proj[row * a.ld_proj + a.g_off + hc]);
            y *= a.gate == 1 ? g * sigmoidf_(g) : sigmoidf_(g);
        }
        out[row * a.ld_out + hc] = from_f32<T>(y * a.out_scale);
    }
}

// The causal convolution of the state space layer and of the gated delta rule: a thread per (token, channel) sums
// taps inputs (the step's own rows, and before the portion's first token the rows the slot keeps, zeros at a
// sequence's start), adds the bias (if any) and applies silu; the result stays float32, [tokens, channels].
constexpr int MAX_TAPS = 16;
template <typename T>
__global__ void __launch_bounds__(256)
ssd_conv_kernel(const ScanArgs a, float* __restrict__ conv_out) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x, taps = a.taps;
    const int channels = a.channels;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int e = a.entry_of_token[row], first = a.q_start[e];
    const T* proj = static_cast<const T*>(a.proj);
    const float* kept = a.state + (size_t)a.slots[e] * (size_t)a.slot_stride + a.kept_off;      // [taps - 1][channels]
    float acc = a.conv_b != nullptr ? a.conv_b[c] : 0.f;
    for (int j = 0; j < taps; ++j) {
        const int r = row - (taps - 1 - j);                         // the row that meets tap j
        const float in = r >= first ? to_f32(proj[(size_t)r * a.ld_proj + a.xbc_off + c])
                                    : kept[(size_t)(taps - 1 + r - first) * channels + c];
        acc = fmaf(a.conv_w[(size_t)j * channels + c], in, acc);
    }
    conv_out[(size_t)row * channels + c] = acc / (1.0f + expf(-acc));
}

// The state space layer's token vectors.  A warp per (token, head) copies its group's C and B and its own
// x out of the convolved row and forms dt = softplus(dt_raw + bias) without a clamp: the record
// [C, B, (exp(-exp(A) dt), dt, 0, 0), x].
template <typename T>
__global__ void __launch_bounds__(128)
ssd_prepare_kernel(const ScanArgs a, const float* __restrict__ conv_out, float* __restrict__ vec, int tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long wg = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    if (wg >= (long long)tokens * a.heads) return;
    const int row = (int)(wg / a.heads), h = (int)(wg % a.heads);
    const int D = a.dim, V = a.v_dim;
    const int inner = a.heads * V, channels = inner + 2 * a.groups * D;
    const int g = h / (a.heads / a.groups);
    const float* cv = conv_out + (size_t)row * channels;
    const T* proj = static_cast<const T*>(a.proj);
    const int rec = 2 * D + 4 + V;
    float* dst = vec + ((size_t)h * tokens + row) * rec;
    for (int d = lane; d < D; d += 32) {
        dst[d] = cv[inner + a.groups * D + g * D + d];              // C: what reads the state
        dst[D + d] = cv[inner + g * D + d];                          // B: what writes it
    }
    for (int c = lane; c < V; c += 32) dst[2 * D + 4 + c] = cv[h * V + c];
    if (lane == 0) {
        const float raw = to_f32(proj[(size_t)row * a.ld_proj + a.dt_off + h]) + a.dt_bias[h];
        const float dt = fmaxf(raw, 0.f) + log1pf(expf(-fabsf(raw)));       // softplus, exact at both ends
        dst[2 * D] = expf(-expf(a.a_log[h]) * dt);
        dst[2 * D + 1] = dt;
        dst[2 * D + 2] = 0.f;
        dst[2 * D + 3] = 0.f;
    }
}

// Decay and step size of every (token, head), where the convolution's kernel does not form them.
template <typename T>
__global__ void __launch_bounds__(128)
ssd_dt_kernel(const ScanArgs a, float2* __restrict__ dts, int tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)tokens * a.heads) return;
    const int h = (int)(i % a.heads);
    const float raw = to_f32(static_cast<const T*>(a.proj)[(size_t)(i / a.heads) * a.ld_proj + a.dt_off + h]) + a.dt_bias[h];
    const float dt = fmaxf(raw, 0.f) + log1pf(expf(-fabsf(raw)));
    dts[i] = make_float2(expf(-expf(a.a_log[h]) * dt), dt);
}

// The gated delta rule's token vectors.  A warp per (token, head) makes the unit vectors of its group's q and k
// (q also times q_scale), the decay of every key channel and the write rate: the record
// [q, k, g, (beta, q . k, 0, 0), v].
template <typename T>
__global__ void __launch_bounds__(128)
gated_delta_prepare_kernel(const ScanArgs a, const float* __restrict__ conv_out, float* __restrict__ vec, int tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long wg = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    if (wg >= (long long)tokens * a.heads) return;
    const int row = (int)(wg / a.heads), h = (int)(wg % a.heads);
    const int D = a.dim, V = a.v_dim;
    const int g = h / (a.heads / a.groups);
    const float* qv = conv_out + (size_t)row * a.channels + g * D;
    const float* kv = qv + a.groups * D;
    const float* vv = conv_out + (size_t)row * a.channels + 2 * a.groups * D + h * V;
    const int rec = 3 * D + 4 + V;
    float* dst = vec + ((size_t)h * tokens + row) * rec;
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int d = lane; d < D; d += 32) {
        const float q = qv[d], k = kv[d];
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
        qk = fmaf(q, k, qk);
    }
    const float iq = a.q_scale / sqrtf(warp_sum(qq) + 1e-6f), ik = 1.0f / sqrtf(warp_sum(kk) + 1e-6f);
    qk = warp_sum(qk) * iq * ik;
    const float rate = expf(a.a_log[h]);
    const float* ar = a.a_raw + (size_t)row * a.ld_a + h * D;
    for (int d = lane; d < D; d += 32) {
        const float raw = ar[d] + a.dt_bias[h * D + d];
        const float sp = fmaxf(raw, 0.f) + log1pf(expf(-fabsf(raw)));       // softplus, exact at both ends
        dst[d] = qv[d] * iq;
        dst[D + d] = kv[d] * ik;
        dst[2 * D + d] = expf(-rate * sp);
    }
    for (int c = lane; c < V; c += 32) dst[3 * D + 4 + c] = vv[c];
    if (lane == 0) {
        dst[3 * D] = sigmoidf_(to_f32(static_cast<const T*>(a.proj)[(size_t)row * a.ld_proj + a.b_off + h]));
        dst[3 * D + 1] = qk;
        dst[3 * D + 2] = 0.f;
        dst[3 * D + 3] = 0.f;
    }
}

// After the scan: y = (o + D_h x) * silu(z), divided by the root mean square of its part of the row
// (norm_groups equal parts of heads * v_dim), times the weight.  A block per (token, part).
// keep: every entry brought one token, and the blocks of its row also move its kept inputs on.
template <typename T>
__global__ void __launch_bounds__(256)
ssd_finish_kernel(const ScanArgs a, const float* __restrict__ conv_out, const float* __restrict__ o_raw, int keep) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    if (keep) {
        const int e = blockIdx.x / a.norm_groups;               // (row e is entry e's)
        float* kept = a.state + (size_t)a.slots[e] * (size_t)a.slot_stride + a.kept_off;
        const T* in = static_cast<const T*>(a.proj) + (size_t)e * a.ld_proj + a.xbc_off;
        for (int c = (blockIdx.x % a.norm_groups) * blockDim.x + threadIdx.x; c < a.channels; c += a.norm_groups * blockDim.x) {
            for (int j = 0; j + 2 < a.taps; ++j) kept[(size_t)j * a.channels + c] = kept[(size_t)(j + 1) * a.channels + c];
            kept[(size_t)(a.taps - 2) * a.channels + c] = to_f32(in[c]);
        }
    }
    const size_t row = blockIdx.x / a.norm_groups;
    const int part = blockIdx.x % a.norm_groups, V = a.v_dim, inner = a.heads * V, n = inner / a.norm_groups;
    const int channels = inner + 2 * a.groups * a.dim;
    const T* proj = static_cast<const T*>(a.proj) + row * a.ld_proj;
    auto value = [&](int ch) {
        const float x = conv_out[row * channels + ch];
        const float z = to_f32(proj[a.z_off + ch]);
        return fmaf(a.d_skip[ch / V], x, o_raw[row * inner + ch]) * (z / (1.0f + expf(-z)));
    };
    // a thread's first values stay in registers between the two passes (all of them for parts of up to 1,024)
    constexpr int HELD = 8;
    float held[HELD];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < HELD; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
        held[k] = i < n ? value(part * n + i) : 0.f;
        ss = fmaf(held[k], held[k], ss);
    }
    for (int i = threadIdx.x + HELD * blockDim.x; i < n; i += blockDim.x) {
        const float y = value(part * n + i);
        ss = fmaf(y, y, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)n + a.eps);
    T* out = static_cast<T*>(a.out) + row * a.ld_out;
#pragma unroll
    for (int k = 0; k < HELD; ++k) {
        const int i = threadIdx.x + k * blockDim.x, ch = part * n + i;
        if (i < n) out[ch] = from_f32<T>(held[k] * inv * (a.norm_w ? a.norm_w[ch] : 1.f));
    }
    for (int i = threadIdx.x + HELD * blockDim.x; i < n; i += blockDim.x) {
        const int ch = part * n + i;
        out[ch] = from_f32<T>(value(ch) * inv * (a.norm_w ? a.norm_w[ch] : 1.f));
    }
}

// The slot keeps the last taps - 1 inputs of every convolved channel: the portion's last rows, and
// where the portion is shorter than that, the rows kept before move up.  A thread per (entry,
// channel) reads what it needs first and writes then.
template <typename T>
__global__ void __launch_bounds__(256)
ssd_conv_keep_kernel(const ScanArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x, first = a.q_start[e], n = a.q_start[e + 1] - first, keep = a.taps - 1;
    const int channels = a.channels;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (n <= 0 || c >= channels) return;
    const T* proj = static_cast<const T*>(a.proj);
    float* kept = a.state + (size_t)a.slots[e] * (size_t)a.slot_stride + a.kept_off;
    float rows[MAX_TAPS - 1];
#pragma unroll
    for (int r = 0; r < MAX_TAPS - 1; ++r) {
        if (r >= keep) break;
        const int k = n - keep + r;                                // row of the portion, or (negative) a row kept before
        rows[r] = k >= 0 ? to_f32(proj[(size_t)(first + k) * a.ld_proj + a.xbc_off + c]) : kept[(size_t)(keep + k) * channels + c];
    }
#pragma unroll
    for (int r = 0; r < MAX_TAPS - 1; ++r) {
        if (r >= keep) break;
        kept[(size_t)r * channels + c] = rows[r];
    }
}

// (P below 8 comes with at most 8 rows per thread, see launch_scan; rows that do not go by fours are rare, so two
// sizes of the unrolled loop serve them)
// The launch of a kernel whose blocks walk tokens: many tokens per entry make its blocks long-running, and those want
// to be spread over the SMs.
template <typename... KArgs, typename... Args>
int launch_walk(const ScanArgs& a, int tokens, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                Args&&... args) {
    if (tokens >= 8 * a.entries) return kipp_launch_spread(kernel, grid, block, smem, stream, static_cast<Args&&>(args)...);
    return kipp_launch(kernel, grid, block, smem, stream, 1, static_cast<Args&&>(args)...);
}

// ---------------------------------------------------------------------------
// The two recurrences whose scans are built for heads that go by fours (other sizes take the template above).  Both
// walk an entry's tokens in order with S in registers; what a token needs of shared memory is fetched into registers
// while the token before is worked on, so that only the recurrence itself is a chain.  The order of every sum
// depends on the sizes only.
//
// State space: a thread owns 4 columns x R rows (P threads per group of columns, rows in groups of four dealt out in
// turn), so that a token's C and B serve four columns per load; the four outputs' sums over P lanes meet in P's
// logarithm plus one shuffles (every exchange also halves the columns a lane is responsible for).  C, B and x come
// straight out of the convolved rows, decay and step size from dts [tokens][heads].
// Rows go through the arithmetic in pairs (float32 pairs in one instruction).
constexpr int SCAN_COLS = 4;
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)));
    return d;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)),
          "l"(reinterpret_cast<const unsigned long long&>(c)));
    return d;
}
__device__ __forceinline__ float2 both(float v) { return make_float2(v, v); }
struct TokenBatch {                          // two buffers of `tokens` tokens of `floats` floats
    int tokens, floats;
};
__host__ __device__ inline TokenBatch token_batch(int floats) {
    TokenBatch b;
    b.floats = floats;
    b.tokens = floats * 4 * 32 <= 22 * 1024 ? 32 : (22 * 1024) / (floats * 4);
    if (b.tokens < 1) b.tokens = 1;
    return b;
}
// EXACT: the P threads' rows are the head's, none too many.
template <int P, int R, int WARPS, bool EXACT>
__global__ void __launch_bounds__(32 * WARPS)
ssd_scan_kernel(const ScanArgs a, const float* __restrict__ conv, const float2* __restrict__ dts, float* __restrict__ o_raw, int v_slices) {
    extern __shared__ __align__(16) float smem[];
    constexpr int COLS = SCAN_COLS * 32 * WARPS / P, THREADS = 32 * WARPS;
    const int D = a.dim, V = a.v_dim;
    const TokenBatch tb = token_batch(2 * D + COLS + 4);
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, p = tid % P, slice = blockIdx.x % v_slices, eh = blockIdx.x / v_slices;
    const int e = eh / a.heads, h = eh % a.heads, g = h / (a.heads / a.groups);
    const int row0 = a.q_start[e], n_tok = a.q_start[e + 1] - row0;
    const int cl = tid / P * SCAN_COLS, col = slice * COLS + cl;
    const bool live = col < V;                                      // (V is a multiple of 4: a group is whole or absent)
    float* S_slot = a.state + (size_t)a.slots[e] * (size_t)a.slot_stride + (size_t)h * D * V;
    const int inner = a.heads * V;
    const float* b_at = conv + inner + (size_t)g * D;
    const float* c_at = conv + inner + (size_t)(a.groups + g) * D;
    // a token in a buffer: C [D], B [D], x [COLS], (decay, step size, -, -)
    auto fetch = [&](int t0, float* buf) {
        // (a warp takes whole tokens: nothing to divide)
        const int nb = min(tb.tokens, n_tok - t0), d4 = D / 4, per = 2 * d4 + COLS / 4;
        for (int t = tid >> 5; t < nb; t += WARPS) {
            const size_t at = (size_t)(row0 + t0 + t) * a.channels;
            const uint32_t to = smem_address(buf + (size_t)t * tb.floats);
            for (int c = tid & 31; c < per; c += 32) {
                const int x = slice * COLS + 4 * (c - 2 * d4);
                const bool ok = c < 2 * d4 || x < V;
                const float* src = c < d4 ? c_at + 4 * c : c < 2 * d4 ? b_at + 4 * (c - d4) : conv + (ok ? h * V + x : 0);
                cp_async16(to + 16 * c, src + at, ok ? 16 : 0);
            }
        }
        for (int t = tid; t < nb; t += THREADS)
            *reinterpret_cast<float2*>(buf + (size_t)t * tb.floats + 2 * D + COLS) = dts[(size_t)(row0 + t0 + t) * a.heads + h];
        cp_async_commit();
    };
    // row i of this thread: 4 (p + P (i / 4)) + i % 4; S[i / 2][c] holds rows i and i + 1 of column c
    float2 S[R / 2][SCAN_COLS];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int r = 4 * (p + P * (i >> 2)) + (i & 3);
        const float4 s4 = live && r < D ? *reinterpret_cast<const float4*>(S_slot + (size_t)r * V + col) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float e[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
        for (int c = 0; c < SCAN_COLS; ++c) (i & 1 ? S[i >> 1][c].y : S[i >> 1][c].x) = e[c];
    }
    float2 cv[R / 2], bv[R / 2], keep, tx[SCAN_COLS];
    auto take = [&](const float* tok) {
#pragma unroll
        for (int q = 0; q < R / 4; ++q) {
            const int r = 4 * (p + P * q);
            float4 c4 = make_float4(0.f, 0.f, 0.f, 0.f), b4 = c4;
            if (EXACT || r < D) {
                c4 = *reinterpret_cast<const float4*>(tok + r);
                b4 = *reinterpret_cast<const float4*>(tok + D + r);
            }
            cv[2 * q] = make_float2(c4.x, c4.y); cv[2 * q + 1] = make_float2(c4.z, c4.w);
            bv[2 * q] = make_float2(b4.x, b4.y); bv[2 * q + 1] = make_float2(b4.z, b4.w);
        }
        const float4 x4 = *reinterpret_cast<const float4*>(tok + 2 * D + cl);
        const float2 kd = *reinterpret_cast<const float2*>(tok + 2 * D + COLS);
        keep = both(kd.x);
        tx[0] = both(kd.y * x4.x); tx[1] = both(kd.y * x4.y); tx[2] = both(kd.y * x4.z); tx[3] = both(kd.y * x4.w);
    };
    fetch(0, smem);
    int buf = 0;
    for (int t0 = 0; t0 < n_tok; t0 += tb.tokens, buf ^= 1) {
        const int nb = min(tb.tokens, n_tok - t0);
        if (t0 + tb.tokens < n_tok) fetch(t0 + tb.tokens, smem + (size_t)(buf ^ 1) * tb.tokens * tb.floats);
        else cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const float* toks = smem + (size_t)buf * tb.tokens * tb.floats;
        take(toks);
        // a token's sums travel while the next token is worked on: the chain of shuffles is nobody's wait
        float last[SCAN_COLS] = {0.f, 0.f, 0.f, 0.f};
        float* out = o_raw + (size_t)(row0 + t0) * inner + h * V + col + 2 * (p & 1) + (p >> 1);      // lanes p < 4
        auto meet = [&](const float* o) {
            // lane p of a group of P ends up with column 2 (p & 1) + (p >> 1 & 1)
            const bool odd = p & 1, second = p & 2;
            float k0 = odd ? o[2] : o[0], k1 = odd ? o[3] : o[1];
            k0 += __shfl_xor_sync(0xffffffffu, odd ? o[0] : o[2], 1);
            k1 += __shfl_xor_sync(0xffffffffu, odd ? o[1] : o[3], 1);
            float y = (second ? k1 : k0) + __shfl_xor_sync(0xffffffffu, second ? k0 : k1, 2);
#pragma unroll
            for (int x = 4; x < P; x <<= 1) y += __shfl_xor_sync(0xffffffffu, y, x);
            return y;
        };
        const bool writes = live && p < SCAN_COLS;
        for (int t = 0; t < nb; ++t) {
            float2 o[SCAN_COLS];
            const float y = meet(last);
#pragma unroll
            for (int i = 0; i < R / 2; ++i)
#pragma unroll
                for (int c = 0; c < SCAN_COLS; ++c) {
                    S[i][c] = fma2(bv[i], tx[c], mul2(keep, S[i][c]));
                    o[c] = i == 0 ? mul2(cv[i], S[i][c]) : fma2(cv[i], S[i][c], o[c]);
                }
            take(toks + (size_t)min(t + 1, nb - 1) * tb.floats);
            if (writes && t > 0) {
                *out = y;
                out += inner;
            }
#pragma unroll
            for (int c = 0; c < SCAN_COLS; ++c) last[c] = o[c].x + o[c].y;
        }
        const float y = meet(last);
        if (writes) *out = y;
        __syncthreads();                    // the buffer is free for the batch after the next
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int r = 4 * (p + P * (i >> 2)) + (i & 3);
        auto at = [&](int c) { return i & 1 ? S[i >> 1][c].y : S[i >> 1][c].x; };
        if (live && r < D) *reinterpret_cast<float4*>(S_slot + (size_t)r * V + col) = make_float4(at(0), at(1), at(2), at(3));
    }
}

// The gated delta rule: a thread owns R rows of one column.  The decayed state meets k and q in one pass and both
// sums travel through the same shuffles; the token's own write then joins the output as (q . k) u.
template <int P, int R, int WARPS, bool EXACT>
__global__ void __launch_bounds__(32 * WARPS)
gated_delta_scan_kernel(const ScanArgs a, const float* __restrict__ vec, float* __restrict__ o_raw, int v_slices, int tokens) {
    extern __shared__ __align__(16) float smem[];
    constexpr int COLS = 32 * WARPS / P;
    const int D = a.dim, V = a.v_dim, nvd = 3 * D + 4, rec = nvd + V;
    const TokenBatch tb = token_batch(nvd + COLS);
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, p = tid % P, slice = blockIdx.x % v_slices, eh = blockIdx.x / v_slices;
    const int e = eh / a.heads, h = eh % a.heads;
    const int row0 = a.q_start[e], n_tok = a.q_start[e + 1] - row0;
    const int cl = tid / P, col = slice * COLS + cl;
    const bool live = col < V;
    float* S_slot = a.state + (size_t)a.slots[e] * (size_t)a.slot_stride + (size_t)h * D * V;
    const float* recs = vec + ((size_t)h * tokens + row0) * rec;
    auto fetch = [&](int t0, float* buf) {
        const int nb = min(tb.tokens, n_tok - t0), n4 = nvd / 4, per = n4 + COLS / 4;
        for (int t = tid >> 5; t < nb; t += WARPS) {
            const float* src = recs + (size_t)(t0 + t) * rec;
            const uint32_t to = smem_address(buf + (size_t)t * tb.floats);
            for (int c = tid & 31; c < per; c += 32) {
                const int x = slice * COLS + 4 * (c - n4);
                const bool ok = c < n4 || x < V;                    // (V is a multiple of 4 here)
                cp_async16(to + 16 * c, src + (c < n4 ? 4 * c : ok ? nvd + x : 0), ok ? 16 : 0);
            }
        }
        cp_async_commit();
    };
    float2 S[R / 2];                        // pairs of neighbouring rows
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int r = 4 * (p + P * (i >> 2)) + (i & 3);
        (i & 1 ? S[i >> 1].y : S[i >> 1].x) = live && r < D ? S_slot[(size_t)r * V + col] : 0.f;
    }
    struct Token { float2 q[R / 2], k[R / 2], g[R / 2]; float beta, qk, v; };
    auto take = [&](const float* tok, Token& n) {
#pragma unroll
        for (int q = 0; q < R / 4; ++q) {
            const int r = 4 * (p + P * q);
            float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f), k4 = q4, g4 = q4;
            if (EXACT || r < D) {
                q4 = *reinterpret_cast<const float4*>(tok + r);
                k4 = *reinterpret_cast<const float4*>(tok + D + r);
                g4 = *reinterpret_cast<const float4*>(tok + 2 * D + r);
            }
            n.q[2 * q] = make_float2(q4.x, q4.y); n.q[2 * q + 1] = make_float2(q4.z, q4.w);
            n.k[2 * q] = make_float2(k4.x, k4.y); n.k[2 * q + 1] = make_float2(k4.z, k4.w);
            n.g[2 * q] = make_float2(g4.x, g4.y); n.g[2 * q + 1] = make_float2(g4.z, g4.w);
        }
        n.beta = tok[3 * D];
        n.qk = tok[3 * D + 1];
        n.v = tok[nvd + cl];
    };
    fetch(0, smem);
    int buf = 0;
    for (int t0 = 0; t0 < n_tok; t0 += tb.tokens, buf ^= 1) {
        const int nb = min(tb.tokens, n_tok - t0);
        if (t0 + tb.tokens < n_tok) fetch(t0 + tb.tokens, smem + (size_t)(buf ^ 1) * tb.tokens * tb.floats);
        else cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const float* toks = smem + (size_t)buf * tb.tokens * tb.floats;
        float* out = o_raw + (size_t)(row0 + t0) * (a.heads * V) + h * V + col;
        const bool writes = live && p == 0;
        Token even, odd;
        // one token from `now`; `next` is fetched meanwhile (the last token of a batch fetches itself again)
        auto step = [&](int t, const Token& now, Token& next) {
            // (two sums per product, so that no chain is longer than a quarter of the rows)
            float2 us[2], os[2];
#pragma unroll
            for (int i = 0; i < R / 2; ++i) {
                S[i] = mul2(S[i], now.g[i]);
                us[i & 1] = i < 2 ? mul2(now.k[i], S[i]) : fma2(now.k[i], S[i], us[i & 1]);
            }
            float uy = (us[0].x + us[0].y) + (us[1].x + us[1].y);
#pragma unroll
            for (int x = P / 2; x > 0; x >>= 1) uy += __shfl_xor_sync(0xffffffffu, uy, x);
#pragma unroll
            for (int i = 0; i < R / 2; ++i) os[i & 1] = i < 2 ? mul2(now.q[i], S[i]) : fma2(now.q[i], S[i], os[i & 1]);
            float oy = (os[0].x + os[0].y) + (os[1].x + os[1].y);
#pragma unroll
            for (int x = P / 2; x > 0; x >>= 1) oy += __shfl_xor_sync(0xffffffffu, oy, x);
            take(toks + (size_t)min(t + 1, nb - 1) * tb.floats, next);
            const float u = now.beta * (now.v - uy);
            const float2 u2 = both(u);
#pragma unroll
            for (int i = 0; i < R / 2; ++i) S[i] = fma2(now.k[i], u2, S[i]);
            if (writes) *out = fmaf(now.qk, u, oy);
            out += a.heads * V;
        };
        take(toks, even);
        int t = 0;
        for (; t + 1 < nb; t += 2) {
            step(t, even, odd);
            step(t + 1, odd, even);
        }
        if (t < nb) step(t, even, odd);
        __syncthreads();                    // the buffer is free for the batch after the next
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int r = 4 * (p + P * (i >> 2)) + (i & 3);
        if (live && r < D) S_slot[(size_t)r * V + col] = i & 1 ? S[i >> 1].y : S[i >> 1].x;
    }
}

// The convolution for channels that go by eights (four in 32-bit) and up to 4 taps: a thread takes 16 bytes of
// channels over a run of CONV_RUN tokens and reads every input once (the last taps - 1 stay in registers; they come
// anew where a run or an entry starts).  The order of a channel's sum is ssd_conv_kernel's.  The last row of
// blocks forms the state space layer's decays and step sizes, dts [tokens][heads] (null: none).
constexpr int CONV_RUN = 8, CONV_THREADS = 128;
template <typename T, int TAPS>
__global__ void __launch_bounds__(CONV_THREADS)
conv_run_kernel(const ScanArgs a, float* __restrict__ conv_out, float2* __restrict__ dts, int tokens) {
    constexpr int VEC = 16 / (int)sizeof(T);
    pdl_launch_dependents();
    pdl_wait();
    const int r0 = blockIdx.x * CONV_RUN, r1 = min(tokens, r0 + CONV_RUN);
    const T* proj = static_cast<const T*>(a.proj);
    if (dts != nullptr && blockIdx.y == gridDim.y - 1) {
        for (int i = threadIdx.x; i < (r1 - r0) * a.heads; i += CONV_THREADS) {
            const int row = r0 + i / a.heads, h = i % a.heads;
            const float raw = to_f32(proj[(size_t)row * a.ld_proj + a.dt_off + h]) + a.dt_bias[h];
            const float dt = fmaxf(raw, 0.f) + log1pf(expf(-fabsf(raw)));       // softplus, exact at both ends
            dts[(size_t)row * a.heads + h] = make_float2(expf(-expf(a.a_log[h]) * dt), dt);
        }
        return;
    }
    const int c = (blockIdx.y * CONV_THREADS + threadIdx.x) * VEC;
    if (c >= a.channels) return;
    float w[VEC][TAPS], bias[VEC], in[TAPS][VEC];              // in[TAPS - 1]: the current token's
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        bias[i] = a.conv_b != nullptr ? a.conv_b[c + i] : 0.f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[i][j] = a.conv_w[(size_t)j * a.channels + c + i];
    }
    auto load = [&](int row, float* to) {
        const uint4 raw = *reinterpret_cast<const uint4*>(proj + (size_t)row * a.ld_proj + a.xbc_off + c);
        const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int i = 0; i < VEC; ++i) to[i] = to_f32(e[i]);
    };
    int end = r0;                                              // where the entry of the run's next token ends
    for (int row = r0; row < r1; ++row) {
        if (row == end || row == r0) {
            const int e = a.entry_of_token[row], first = a.q_start[e];
            end = a.q_start[e + 1];
            const float* kept = a.state + (size_t)a.slots[e] * (size_t)a.slot_stride + a.kept_off;     // [TAPS - 1][channels]
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) {
                const int r = row - (TAPS - 1 - j);
                if (r >= first) {
                    load(r, in[j]);
                } else {
#pragma unroll
                    for (int i = 0; i < VEC; ++i) in[j][i] = kept[(size_t)(TAPS - 1 + r - first) * a.channels + c + i];
                }
            }
        }
        load(row, in[TAPS - 1]);
        float y[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            float acc = bias[i];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) acc = fmaf(w[i][j], in[j][i], acc);
            y[i] = acc / (1.0f + expf(-acc));
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) in[j][i] = in[j + 1][i];
        }
#pragma unroll
        for (int i = 0; i < VEC; i += 4)
            *reinterpret_cast<float4*>(conv_out + (size_t)row * a.channels + c + i) = make_float4(y[i], y[i + 1], y[i + 2], y[i + 3]);
    }
}
template <typename T>
int launch_conv(const ScanArgs& a, float* conv_out, float2* dts, int tokens, bool run, cudaStream_t stream) {
    if (!run)
        return kipp_launch(ssd_conv_kernel<T>, dim3((unsigned)tokens, (unsigned)((a.channels + 255) / 256)), dim3(256), 0, stream, 1, a,
                           conv_out);
    constexpr int VEC = 16 / (int)sizeof(T);
    const dim3 grid((unsigned)((tokens + CONV_RUN - 1) / CONV_RUN),
                    (unsigned)((a.channels / VEC + CONV_THREADS - 1) / CONV_THREADS + (dts != nullptr ? 1 : 0)));
    auto go = [&](auto kernel) { return kipp_launch(kernel, grid, dim3(CONV_THREADS), 0, stream, 1, a, conv_out, dts, tokens); };
    switch (a.taps) {
    case 1: return go(conv_run_kernel<T, 1>);
    case 2: return go(conv_run_kernel<T, 2>);
    case 3: return go(conv_run_kernel<T, 3>);
    default: return go(conv_run_kernel<T, 4>);
    }
}
template <typename T> bool conv_run_ok(const ScanArgs& a) {
    constexpr int VEC = 16 / (int)sizeof(T);
    return a.taps <= 4 && a.channels % VEC == 0 && a.ld_proj % VEC == 0 && a.xbc_off % VEC == 0 && ((uintptr_t)a.proj & 15) == 0;
}
// Whether the scans built for heads that go by fours take this one.
inline bool scan_by_fours(const ScanArgs& a) {
    return a.dim % 4 == 0 && a.v_dim % 4 == 0 && a.dim <= 256 && a.slot_stride % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
}
// (32 columns a block)
template <int P, int R>
int launch_ssd_scan(const ScanArgs& a, const float* conv, const float2* dts, float* o_raw, int entries, int tokens, cudaStream_t stream) {
    constexpr int WARPS = P / 4, COLS = SCAN_COLS * 32 * WARPS / P;
    const TokenBatch tb = token_batch(2 * a.dim + COLS + 4);
    const int slices = (a.v_dim + COLS - 1) / COLS;
    return launch_walk(a, tokens, a.dim == P * R ? ssd_scan_kernel<P, R, WARPS, true> : ssd_scan_kernel<P, R, WARPS, false>,
                       dim3((unsigned)(entries * a.heads * slices)), dim3(32 * WARPS), (size_t)2 * tb.tokens * tb.floats * sizeof(float),
                       stream, a, conv, dts, o_raw, slices);
}
// (8 columns a block: the more blocks, the fewer warps share an SM, and a token's chain is what this scan is bound by)
template <int P, int R>
int launch_gated_delta_scan(const ScanArgs& a, const float* vec, float* o_raw, int entries, int tokens, cudaStream_t stream) {
    constexpr int WARPS = P / 4, COLS = 32 * WARPS / P;
    const TokenBatch tb = token_batch(3 * a.dim + 4 + COLS);
    const int slices = (a.v_dim + COLS - 1) / COLS;
    return launch_walk(a, tokens, a.dim == P * R ? gated_delta_scan_kernel<P, R, WARPS, true> : gated_delta_scan_kernel<P, R, WARPS, false>,
                       dim3((unsigned)(entries * a.heads * slices)), dim3(32 * WARPS), (size_t)2 * tb.tokens * tb.floats * sizeof(float),
                       stream, a, vec, o_raw, slices, tokens);
}

// ---------------------------------------------------------------------------
// Steps in which every entry brings ONE token: what the scans do in three or four launches, with lanes over the
// columns of S, so that the state, which is what such a step moves, is read and written in whole lines.  A thread owns
// the rows rg, rg + RG, ... of one column (RG row groups); the groups' sums meet in shared memory in order.  The state's
// loads are on their way while the convolution runs.
// One convolved channel of an entry's only token: silu of the sum over the kept inputs and the new one.  `keep`: the
// kept inputs move on (the caller owns the channel).
template <typename T>
__device__ __forceinline__ float conv_one(const ScanArgs& a, const T* __restrict__ proj, float* __restrict__ kept, int c, bool keep) {
    const int taps = a.taps;
    float acc = a.conv_b != nullptr ? a.conv_b[c] : 0.f;
    const float in = to_f32(proj[a.xbc_off + c]);
    for (int j = 0; j < taps - 1; ++j) {
        const float old = kept[(size_t)j * a.channels + c];
        acc = fmaf(a.conv_w[(size_t)j * a.channels + c], old, acc);
        if (keep && j > 0) kept[(size_t)(j - 1) * a.channels + c] = old;
    }
    acc = fmaf(a.conv_w[(size_t)(taps - 1) * a.channels + c], in, acc);
    if (keep && taps > 1) kept[(size_t)(taps - 2) * a.channels + c] = in;
    return acc / (1.0f + expf(-acc));
}
struct TokenShape {
    int cols, groups, rows;                  // threads along a row of S, row groups, rows per thread
};
inline TokenShape token_shape(int dim, int v_dim) {
    TokenShape t;
    t.cols = (v_dim + 31) / 32 * 32;
    t.groups = t.cols > 512 ? 1 : 512 / t.cols;
    if (t.groups > dim) t.groups = dim;
    if (t.groups > 16) t.groups = 16;
    t.rows = (dim + t.groups - 1) / t.groups;
    return t;
}
constexpr int TOKEN_ROWS = 32;
inline bool token_kernel_ok(const ScanArgs& a, int tokens) {
    const TokenShape t = token_shape(a.dim, a.v_dim);
    return tokens == a.entries && t.cols <= 512 && t.rows <= TOKEN_ROWS && a.dim <= 512;
}

// The gated delta rule: a block per (entry, q/k head) does the whole layer behind the projections for the heads of its
// group: convolution (and the kept inputs), unit vectors, decays, the recurrence, norm and gate.
template <typename T, int MR>
__global__ void __launch_bounds__(512, MR <= 16 ? 2 : 1)
gated_delta_token_kernel(const ScanArgs a, int cols, int groups) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float scratch[32];
    const int D = a.dim, V = a.v_dim, per = a.heads / a.groups;
    float *qs = smem, *ks = qs + D, *gs = ks + D, *vs = gs + D, *red = vs + V;           // red: [2][groups][cols]
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x / a.groups, kvh = blockIdx.x % a.groups, tid = threadIdx.x;
    const int row = a.q_start[e], col = tid % cols, rg = tid / cols;
    const T* proj = static_cast<const T*>(a.proj) + (size_t)row * a.ld_proj;
    float* slot = a.state + (size_t)a.slots[e] * (size_t)a.slot_stride;
    float* kept = slot + a.kept_off;
    const bool live = col < V;
    for (int hh = 0; hh < per; ++hh) {
        const int h = kvh * per + hh;
        float* S_slot = slot + (size_t)h * D * V;
        float S[MR];
#pragma unroll
        for (int i = 0; i < MR; ++i) {
            const int r = rg + groups * i;
            S[i] = live && r < D ? S_slot[(size_t)r * V + col] : 0.f;
        }
        if (hh == 0)
            for (int c = tid; c < 2 * D; c += blockDim.x) {
                const int ch = c < D ? kvh * D + c : (a.groups + kvh) * D + c - D;
                smem[c] = conv_one(a, proj, kept, ch, true);
            }
        for (int c = tid; c < V; c += blockDim.x) vs[c] = conv_one(a, proj, kept, 2 * a.groups * D + h * V + c, true);
        const float rate = expf(a.a_log[h]);
        for (int d = tid; d < D; d += blockDim.x) {
            const float raw = a.a_raw[(size_t)row * a.ld_a + h * D + d] + a.dt_bias[h * D + d];
            const float sp = fmaxf(raw, 0.f) + log1pf(expf(-fabsf(raw)));       // softplus, exact at both ends
            gs[d] = expf(-rate * sp);
        }
        const float beta = sigmoidf_(to_f32(proj[a.b_off + h]));
        __syncthreads();
        // every warp forms the three sums over the key channels itself
        float qq = 0.f, kk = 0.f, qk = 0.f;
        for (int d = tid & 31; d < D; d += 32) {
            qq = fmaf(qs[d], qs[d], qq);
            kk = fmaf(ks[d], ks[d], kk);
            qk = fmaf(qs[d], ks[d], qk);
        }
        const float iq = a.q_scale / sqrtf(warp_sum(qq) + 1e-6f), ik = 1.0f / sqrtf(warp_sum(kk) + 1e-6f);
        qk = warp_sum(qk) * iq * ik;
        float us = 0.f, os = 0.f;
#pragma unroll
        for (int i = 0; i < MR; ++i) {
            const int r = rg + groups * i;
            if (r < D) {
                S[i] *= gs[r];
                us = fmaf(ks[r] * ik, S[i], us);
                os = fmaf(qs[r] * iq, S[i], os);
            }
        }
        red[rg * cols + col] = us;
        red[(groups + rg) * cols + col] = os;
        __syncthreads();
        us = os = 0.f;
        for (int g = 0; g < groups; ++g) {
            us += red[g * cols + col];
            os += red[(groups + g) * cols + col];
        }
        const float u = live ? beta * (vs[col] - us) : 0.f;
#pragma unroll
        for (int i = 0; i < MR; ++i) {
            const int r = rg + groups * i;
            if (live && r < D) S_slot[(size_t)r * V + col] = fmaf(ks[r] * ik, u, S[i]);
        }
        const float o = live ? fmaf(qk, u, os) : 0.f;
        const float inv = 1.0f / sqrtf(block_sum(rg == 0 ? o * o : 0.f, scratch) / (float)V + a.eps);
        if (rg == 0 && live) {
            const float g = a.g_raw[(size_t)row * a.ld_g + h * V + col];
            const float y = o * inv * a.norm_w[col] * (a.gate == 1 ? g * sigmoidf_(g) : sigmoidf_(g));
            static_cast<T*>(a.out)[(size_t)row * a.ld_out + h * V + col] = from_f32<T>(y * a.out_scale);
        }
        __syncthreads();                    // the head's values and sums may be overwritten
    }
}

// The state space layer: a block per (entry, head) convolves its head's x and its group's B and C and updates the
// state; x and the output go where ssd_finish_kernel reads them (it also moves the kept inputs on then).
template <typename T, int MR>
__global__ void __launch_bounds__(512, MR <= 16 ? 2 : 1)
ssd_token_kernel(const ScanArgs a, float* __restrict__ conv_out, float* __restrict__ o_raw, int cols, int groups) {
    extern __shared__ __align__(16) float smem[];
    const int D = a.dim, V = a.v_dim;
    float *bs = smem, *cs = bs + D, *xs = cs + D, *red = xs + V;                          // red: [groups][cols]
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x / a.heads, h = blockIdx.x % a.heads, tid = threadIdx.x, g = h / (a.heads / a.groups);
    const int row = a.q_start[e], col = tid % cols, rg = tid / cols, inner = a.heads * V;
    const T* proj = static_cast<const T*>(a.proj) + (size_t)row * a.ld_proj;
    float* slot = a.state + (size_t)a.slots[e] * (size_t)a.slot_stride;
    float* S_slot = slot + (size_t)h * D * V;
    const bool live = col < V;
    float S[MR];
#pragma unroll
    for (int i = 0; i < MR; ++i) {
        const int r = rg + groups * i;
        S[i] = live && r < D ? S_slot[(size_t)r * V + col] : 0.f;
    }
    for (int c = tid; c < 2 * D + V; c += blockDim.x) {
        const int ch = c < D ? inner + g * D + c : c < 2 * D ? inner + (a.groups + g) * D + c - D : h * V + c - 2 * D;
        const float v = conv_one(a, proj, slot + a.kept_off, ch, false);
        smem[c] = v;
        if (c >= 2 * D) conv_out[(size_t)row * a.channels + ch] = v;
    }
    const float raw = to_f32(proj[a.dt_off + h]) + a.dt_bias[h];
    const float dt = fmaxf(raw, 0.f) + log1pf(expf(-fabsf(raw)));               // softplus, exact at both ends
    const float keep = expf(-expf(a.a_log[h]) * dt);
    __syncthreads();
    const float tx = live ? dt * xs[col] : 0.f;
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < MR; ++i) {
        const int r = rg + groups * i;
        if (live && r < D) {
            const float s = fmaf(bs[r], tx, keep * S[i]);
            o = fmaf(cs[r], s, o);
            S_slot[(size_t)r * V + col] = s;
        }
    }
    red[rg * cols + col] = o;
    __syncthreads();
    if (rg > 0 || !live) return;
    for (int q = 1; q < groups; ++q) o += red[q * cols + col];
    o_raw[(size_t)row * inner + h * V + col] = o;
}

template <typename T, int DELTA, int P, bool VEC>
int launch_scan_rows(const ScanArgs& b, const float* vec, float* o_raw, int slices, int tokens, dim3 grid, size_t smem,
                     cudaStream_t stream) {
    const int chunk = (b.dim + P - 1) / P;
#define KIPP_SCAN(C) return launch_walk(b, tokens, recurrent_scan_kernel<T, DELTA, P, C, VEC>, grid, dim3(VS * P), smem, stream, b, vec, o_raw, slices, tokens)
    if constexpr (P < 8) {
        if (chunk > 8) return KIPP_ERR_ARG;
        KIPP_SCAN(8);
    } else {
        if (chunk <= 8) KIPP_SCAN(8);
        if constexpr (VEC) {
            if (chunk <= 16) KIPP_SCAN(16);
            if (chunk <= 24) KIPP_SCAN(24);
        }
        KIPP_SCAN(32);
    }
#undef KIPP_SCAN
}
template <typename T, int DELTA, int P>
int launch_scan_chunk(const ScanArgs& b, const float* vec, float* o_raw, int slices, int tokens, dim3 grid, size_t smem,
                      cudaStream_t stream) {
    // groups of four rows per 16-byte load where the key size allows (every vector of a record then
    // starts on a 16-byte boundary)
    return b.dim % 4 == 0 ? launch_scan_rows<T, DELTA, P, true>(b, vec, o_raw, slices, tokens, grid, smem, stream)
                          : launch_scan_rows<T, DELTA, P, false>(b, vec, o_raw, slices, tokens, grid, smem, stream);
}

// scratch: float32 [heads][tokens][NV * dim + v_dim] for the records, then [tokens][heads * v_dim] for raw o
// conv_out: float32 [tokens, channels] for the convolved rows of the state space layer and the gated delta rule (null for the other kinds)
template <typename T, int DELTA>
int launch_scan(const ScanArgs& a, int entries, int tokens, float* scratch, cudaStream_t stream, float* conv_out = nullptr) {
    const int D = a.dim, V = a.v_dim + Rec<DELTA>::XV;
    constexpr int NV = Rec<DELTA>::NV, XG = Rec<DELTA>::XG;
    // threads per column: runs of 8 key rows where the head allows (short chains of dependent
    // multiply-adds, more warps per block), at most 8 threads (16 only where a head has more than 256 key rows)
    int P = 1;
    while (P < 8 && (D + P - 1) / P > 8) P *= 2;
    if ((D + P - 1) / P > MAX_CHUNK) P = 16;
    if ((DELTA == SSD || DELTA == GATED_DELTA) && D > 64 && KIPP_SSD_WIDE) P = 16;
    if ((D + P - 1) / P > MAX_CHUNK || scratch == nullptr) return KIPP_ERR_ARG;
    const size_t per_token = ((size_t)NV * D + XG + VS) * sizeof(float);
    int batch = (int)std::min<size_t>(32, (20 * 1024) / per_token);       // two buffers of at most 20 KB
    if (batch < 1) return KIPP_ERR_ARG;
    ScanArgs b = a;
    b.batch = batch;
    b.entries = entries;
    float* vec = scratch;
    float* o_raw = scratch + (size_t)tokens * a.heads * (NV * D + XG + V);
    const long long warps = (long long)tokens * a.heads;
    const dim3 wgrid((unsigned)((warps + 3) / 4));
    int rc = 0;
    constexpr bool CONV = DELTA == SSD || DELTA == GATED_DELTA;
    bool scanned = false;
    const bool one_token = CONV && token_kernel_ok(b, tokens);
    if constexpr (CONV) {
        if (conv_out == nullptr) return KIPP_ERR_ARG;
        if (one_token) {
            const TokenShape t = token_shape(D, V);
            const dim3 block((unsigned)(t.cols * t.groups));
            if constexpr (DELTA == GATED_DELTA) {
                const size_t bytes = ((size_t)3 * D + V + 2 * (size_t)t.groups * t.cols) * sizeof(float);
                return kipp_launch(t.rows <= 8    ? gated_delta_token_kernel<T, 8>
                                   : t.rows <= 16 ? gated_delta_token_kernel<T, 16>
                                                  : gated_delta_token_kernel<T, TOKEN_ROWS>,
                                   dim3((unsigned)(entries * a.groups)), block, bytes, stream, 1, b, t.cols, t.groups);
            }
            const size_t bytes = ((size_t)2 * D + V + (size_t)t.groups * t.cols) * sizeof(float);
            rc = kipp_launch(t.rows <= 8 ? ssd_token_kernel<T, 8> : t.rows <= 16 ? ssd_token_kernel<T, 16> : ssd_token_kernel<T, TOKEN_ROWS>, dim3((unsigned)(entries * a.heads)),
                             block, bytes, stream, 1, b, conv_out, o_raw, t.cols, t.groups);
            if (rc) return rc;
            scanned = true;
        }
    }
    const int channels = a.channels;
    if (scanned) {
    } else if constexpr (CONV) {
        const bool by_fours = scan_by_fours(b) && ((uintptr_t)conv_out & 15) == 0 && ((uintptr_t)scratch & 15) == 0;
        // the state space layer's scan reads the convolved rows themselves; decays and step sizes lie where the
        // records would
        const bool direct = DELTA == SSD && by_fours && channels % 4 == 0, run = conv_run_ok<T>(b) && (DELTA != SSD || direct);
        float2* dts = direct ? reinterpret_cast<float2*>(vec) : nullptr;
        rc = launch_conv<T>(b, conv_out, run ? dts : nullptr, tokens, run, stream);
        if (rc) return rc;
        if (DELTA == SSD && direct && !run) {
            rc = kipp_launch(ssd_dt_kernel<T>, dim3((unsigned)(((long long)tokens * a.heads + 127) / 128)), dim3(128), 0, stream, 1, b, dts,
                             tokens);
        } else if (!direct) {
            rc = kipp_launch(DELTA == SSD ? ssd_prepare_kernel<T> : gated_delta_prepare_kernel<T>, wgrid, dim3(128), 0, stream, 1, b,
                             (const float*)conv_out, vec, tokens);
        }
        if (rc) return rc;
        if (by_fours && (DELTA != SSD || direct)) {
            if constexpr (DELTA == SSD) {
                const float* cv = conv_out;
                if (D <= 32) rc = launch_ssd_scan<8, 4>(b, cv, dts, o_raw, entries, tokens, stream);
                else if (D <= 64) rc = launch_ssd_scan<16, 4>(b, cv, dts, o_raw, entries, tokens, stream);
                else if (D <= 128) rc = launch_ssd_scan<32, 4>(b, cv, dts, o_raw, entries, tokens, stream);
                else rc = launch_ssd_scan<32, 8>(b, cv, dts, o_raw, entries, tokens, stream);
            } else {
                if (D <= 32) rc = launch_gated_delta_scan<8, 4>(b, vec, o_raw, entries, tokens, stream);
                else if (D <= 64) rc = launch_gated_delta_scan<16, 4>(b, vec, o_raw, entries, tokens, stream);
                else if (D <= 128) rc = launch_gated_delta_scan<32, 4>(b, vec, o_raw, entries, tokens, stream);
                else rc = launch_gated_delta_scan<32, 8>(b, vec, o_raw, entries, tokens, stream);
            }
            scanned = true;
        }
    } else {
        rc = kipp_launch(recurrent_prepare_kernel<T, DELTA>, wgrid, dim3(128), 0, stream, 1, b, vec, tokens);
    }
    if (rc) return rc;
    const int slices = (V + VS - 1) / VS;
    const dim3 grid((unsigned)(entries * a.heads * slices));
    const size_t smem = 2 * per_token * batch;
    if (!scanned) switch (P) {
    case 1: rc = launch_scan_chunk<T, DELTA, 1>(b, vec, o_raw, slices, tokens, grid, smem, stream); break;
    case 2: rc = launch_scan_chunk<T, DELTA, 2>(b, vec, o_raw, slices, tokens, grid, smem, stream); break;
    case 4: rc = launch_scan_chunk<T, DELTA, 4>(b, vec, o_raw, slices, tokens, grid, smem, stream); break;
    case 8: rc = launch_scan_chunk<T, DELTA, 8>(b, vec, o_raw, slices, tokens, grid, smem, stream); break;
    default: rc = launch_scan_chunk<T, DELTA, 16>(b, vec, o_raw, slices, tokens, grid, smem, stream); break;
    }
    if (rc) return rc;
    if constexpr (DELTA == SSD) {
        const long long parts = (long long)tokens * b.norm_groups;
        if (parts > 0x7fffffffLL) return KIPP_ERR_ARG;
        const int per_part = a.heads * a.v_dim / b.norm_groups;
        rc = kipp_launch(ssd_finish_kernel<T>, dim3((unsigned)parts), dim3(one_token ? 256 : per_part >= 128 ? 128 : (per_part + 31) / 32 * 32), 0,
                         stream, 1, b, (const float*)conv_out, (const float*)o_raw, one_token && b.taps > 1 ? 1 : 0);
    } else {
        rc = kipp_launch(recurrent_finish_kernel<T, DELTA>, wgrid, dim3(128), 0, stream, 1, b, (const float*)o_raw, tokens);
    }
    if (rc || !CONV || b.taps <= 1 || one_token) return rc;
    return kipp_launch(ssd_conv_keep_kernel<T>, dim3((unsigned)entries, (unsigned)((channels + 255) / 256)), dim3(256), 0, stream,
                       1, b);
}

template <typename T>
__global__ void __launch_bounds__(128)
token_shift_mix_kernel(T* __restrict__ out, long long out_stride, const T* __restrict__ h, const float* __restrict__ mu,
                       const float* __restrict__ prev, long long slot_stride, const int* __restrict__ q_start,
                       const int* __restrict__ entry_of_token, const int* __restrict__ slots, int hidden, int n_mix) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, e = entry_of_token[t];
    const bool inside = t > q_start[e];
    const T* above = h + (size_t)(inside ? t - 1 : t) * hidden;
    const float* kept = prev + (size_t)slots[e] * slot_stride;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float hv = to_f32(h[(size_t)t * hidden + i]);
        const float d = (inside ? to_f32(above[i]) : kept[i]) - hv;
        for (int s = 0; s < n_mix; ++s)
            out[(size_t)s * out_stride + (size_t)t * hidden + i] = from_f32<T>(fmaf(d, mu[(size_t)s * hidden + i], hv));
    }
}
template <typename T>
__global__ void __launch_bounds__(128)
token_shift_keep_kernel(float* __restrict__ prev, long long slot_stride, const T* __restrict__ h,
                        const int* __restrict__ q_start, const int* __restrict__ slots, int hidden) {
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x, last = q_start[e + 1] - 1;
    if (last < q_start[e]) return;
    float* dst = prev + (size_t)slots[e] * slot_stride;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = to_f32(h[(size_t)last * hidden + i]);
}

template <typename T>
__global__ void tanh_rows_kernel(T* __restrict__ out, long long ld_out, const T* __restrict__ in, long long ld_in,
                                 int rows, int cols) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * cols) return;
    const long long r = i / cols, c = i % cols;
    out[r * ld_out + c] = from_f32<T>(tanhf(to_f32(in[r * ld_in + c])));
}
}  // namespace

// Whether the scan kernels take a head of these sizes.
extern "C" int kipp_recurrent_scan_ok(int dim, int v_dim, int kind) {
    if (dim <= 0 || v_dim <= 0 || dim > 16 * MAX_CHUNK || kind < 0 || kind > GATED_DELTA) return 0;
    return (((kind == DELTA_RULE ? 5 : kind == WKV || kind == GATED_DELTA ? 3 : 2) * (size_t)dim + 4 + VS) * sizeof(float)) <= 20 * 1024 ? 1 : 0;
}
// float32 values of scratch a scan of `tokens` tokens needs.
extern "C" long long kipp_recurrent_scratch_floats(int tokens, int heads, int dim, int v_dim, int kind) {
    const long long x = kind == GATED_MEMORY ? 4 : 0, g = kind == WKV || kind == SSD || kind == GATED_DELTA ? 4 : 0;
    return (long long)tokens * heads * ((kind == DELTA_RULE ? 5 : kind == WKV || kind == GATED_DELTA ? 3 : 2) * (long long)dim + x + g + 2 * ((long long)v_dim + x));
}
// float32 values of state one request slot of the gated memory holds: S with n's column and its
// padding, then one running maximum per head and slice of value columns.
extern "C" long long kipp_gated_memory_state_floats(int heads, int dim, int v_dim) {
    return (long long)heads * dim * (v_dim + 4) + (long long)heads * ((v_dim + 4 + VS - 1) / VS);
}

extern "C" int kipp_retention_scan(void* out, long long ld_out, const void* proj, long long ld_proj, int dtype,
                                   int q_off, int k_off, int v_off, int g_off, float* state, const float* decay,
                                   const float* cos_sin, int rot, const int* q_start, const int* slots, int entries,
                                   int tokens, int heads, int dim, int v_dim, float k_scale, float eps,
                                   float out_scale, int gate, float* scratch, void* stream) {
    if (entries <= 0 || tokens <= 0) return 0;
    if (!kipp_recurrent_scan_ok(dim, v_dim, 0) || heads <= 0 || rot < 0 || rot > dim || (rot & 1)) return KIPP_ERR_ARG;
    ScanArgs a = {};
    a.out = out; a.ld_out = ld_out; a.proj = proj; a.ld_proj = ld_proj;
    a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.g_off = g_off;
    a.decay = decay; a.cos_sin = rot > 0 ? cos_sin : nullptr; a.rot = rot; a.state = state;
    a.q_start = q_start; a.slots = slots; a.heads = heads; a.dim = dim; a.v_dim = v_dim;
    a.k_scale = k_scale; a.eps = eps; a.out_scale = out_scale; a.gate = gate;
    if (dtype == KIPP_DT_F32) return launch_scan<float, RETENTION>(a, entries, tokens, scratch, (cudaStream_t)stream);
    if (dtype == KIPP_DT_BF16) return launch_scan<bf16, RETENTION>(a, entries, tokens, scratch, (cudaStream_t)stream);
    return KIPP_ERR_DTYPE;
}

extern "C" int kipp_delta_rule_scan(void* out, long long ld_out, const void* proj, long long ld_proj, int dtype,
                                    int r_off, int k_off, int v_off, int g_off, int a_off, const void* w_raw,
                                    long long ld_w, const float* a_bias, const float* w_bias, const float* norm_w,
                                    float* state, const int* q_start, const int* slots, int entries, int tokens,
                                    int heads, int dim, float eps, float out_scale, int gate, float* scratch,
                                    void* stream) {
    if (entries <= 0 || tokens <= 0) return 0;
    if (!kipp_recurrent_scan_ok(dim, dim, 1) || heads <= 0 || a_bias == nullptr || w_bias == nullptr)
        return KIPP_ERR_ARG;
    ScanArgs a = {};
    a.out = out; a.ld_out = ld_out; a.proj = proj; a.ld_proj = ld_proj;
    a.q_off = r_off; a.k_off = k_off; a.v_off = v_off; a.g_off = g_off; a.a_off = a_off;
    a.w_raw = w_raw; a.ld_w = ld_w; a.a_bias = a_bias; a.w_bias = w_bias; a.norm_w = norm_w;
    a.state = state; a.q_start = q_start; a.slots = slots; a.heads = heads; a.dim = dim; a.v_dim = dim;
    a.k_scale = 1.f; a.eps = eps; a.out_scale = out_scale; a.gate = gate;
    if (dtype == KIPP_DT_F32) return launch_scan<float, DELTA_RULE>(a, entries, tokens, scratch, (cudaStream_t)stream);
    if (dtype == KIPP_DT_BF16) return launch_scan<bf16, DELTA_RULE>(a, entries, tokens, scratch, (cudaStream_t)stream);
    return KIPP_ERR_DTYPE;
}

// The gated matrix memory (see the head of this file): q, k [heads, dim], v and the output gate
// [heads, v_dim] and the two gates' pre-activations [heads] are columns of proj; the state of a slot
// is kipp_gated_memory_state_floats floats.
extern "C" int kipp_gated_memory_scan(void* out, long long ld_out, const void* proj, long long ld_proj, int dtype,
                                      int q_off, int k_off, int v_off, int g_off, int i_off, int f_off,
                                      const float* i_bias, const float* f_bias, const float* norm_w, float* state,
                                      const int* q_start, const int* slots, int entries, int tokens, int heads,
                                      int dim, int v_dim, float gate_cap, float q_scale, float eps, float out_scale,
                                      int gate, float* scratch, void* stream) {
    if (entries <= 0 || tokens <= 0) return 0;
    if (!kipp_recurrent_scan_ok(dim, v_dim, GATED_MEMORY) || heads <= 0 || i_bias == nullptr || f_bias == nullptr ||
        !(gate_cap > 0.f))
        return KIPP_ERR_ARG;
    ScanArgs a = {};
    a.out = out; a.ld_out = ld_out; a.proj = proj; a.ld_proj = ld_proj;
    a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.g_off = g_off; a.i_off = i_off; a.f_off = f_off;
    a.i_bias = i_bias; a.f_bias = f_bias; a.norm_w = norm_w; a.gate_cap = gate_cap; a.q_scale = q_scale;
    a.state = state; a.q_start = q_start; a.slots = slots; a.heads = heads; a.dim = dim; a.v_dim = v_dim;
    a.k_scale = 1.f; a.eps = eps; a.out_scale = out_scale; a.gate = gate;
    a.slot_stride = kipp_gated_memory_state_floats(heads, dim, v_dim);
    if (dtype == KIPP_DT_F32) return launch_scan<float, GATED_MEMORY>(a, entries, tokens, scratch, (cudaStream_t)stream);
    if (dtype == KIPP_DT_BF16) return launch_scan<bf16, GATED_MEMORY>(a, entries, tokens, scratch, (cudaStream_t)stream);
    return KIPP_ERR_DTYPE;
}

// The wkv recurrence (see the head of this file): r, k, v and the output gate [heads, dim] are columns of
// proj, the decay's pre-activation is w_raw [T, heads * dim]; `bonus` is u [heads * dim].  The state of a
// slot is `slot_stride` floats of which the first heads * dim * dim are S.
extern "C" int kipp_wkv_scan(void* out, long long ld_out, const void* proj, long long ld_proj, int dtype, int r_off,
                             int k_off, int v_off, int g_off, const void* w_raw, long long ld_w, const float* w_bias,
                             const float* bonus, const float* norm_w, float* state, long long slot_stride,
                             const int* q_start, const int* slots, int entries, int tokens, int heads, int dim,
                             float eps, float out_scale, int gate, float* scratch, void* stream) {
    if (entries <= 0 || tokens <= 0) return 0;
    if (!kipp_recurrent_scan_ok(dim, dim, WKV) || heads <= 0 || w_bias == nullptr || bonus == nullptr || w_raw == nullptr ||
        slot_stride < (long long)heads * dim * dim)
        return KIPP_ERR_ARG;
    ScanArgs a = {};
    a.out = out; a.ld_out = ld_out; a.proj = proj; a.ld_proj = ld_proj;
    a.q_off = r_off; a.k_off = k_off; a.v_off = v_off; a.g_off = g_off;
    a.w_raw = w_raw; a.ld_w = ld_w; a.w_bias = w_bias; a.bonus = bonus; a.norm_w = norm_w;
    a.state = state; a.slot_stride = slot_stride; a.q_start = q_start; a.slots = slots;
    a.heads = heads; a.dim = dim; a.v_dim = dim;
    a.k_scale = 1.f; a.eps = eps; a.out_scale = out_scale; a.gate = gate;
    if (dtype == KIPP_DT_F32) return launch_scan<float, WKV>(a, entries, tokens, scratch, (cudaStream_t)stream);
    if (dtype == KIPP_DT_BF16) return launch_scan<bf16, WKV>(a, entries, tokens, scratch, (cudaStream_t)stream);
    return KIPP_ERR_DTYPE;
}

// float32 values of state one request slot of the state space layer holds: S [heads, dim, v_dim], then the
// last taps - 1 inputs of the heads * v_dim + 2 * groups * dim convolved channels.
extern "C" long long kipp_ssd_state_floats(int heads, int groups, int dim, int v_dim, int taps) {
    return (long long)heads * dim * v_dim + (long long)(taps > 1 ? taps - 1 : 0) * ((long long)heads * v_dim + 2LL * groups * dim);
}

// The state space layer (see the head of this file).  proj [T, ...] holds z [heads * v_dim] at z_off, the
// channels to convolve [x | B | C] at xbc_off and dt [heads] at dt_off; conv_w [taps, channels] (the last
// tap meets the current token), conv_b [channels], dt_bias, a_log, d_skip [heads], norm_w [heads * v_dim]
// (or null) float32; `dim` is the size of B and C (the state's rows).  A slot is kipp_ssd_state_floats floats.
// conv_out: float32 [tokens, channels] of scratch for the convolved rows.  At most 16 taps.
extern "C" int kipp_ssd_max_taps() { return 16; }
extern "C" int kipp_ssd_scan(void* out, long long ld_out, const void* proj, long long ld_proj, int dtype, int z_off,
                             int xbc_off, int dt_off, const float* conv_w, const float* conv_b, int taps,
                             const float* dt_bias, const float* a_log, const float* d_skip, const float* norm_w,
                             int norm_groups, float* state, long long slot_stride, const int* q_start,
                             const int* entry_of_token, const int* slots, int entries, int tokens, int heads, int groups,
                             int dim, int v_dim, float eps, float* scratch, float* conv_out, void* stream) {
    if (entries <= 0 || tokens <= 0) return 0;
    if (!kipp_recurrent_scan_ok(dim, v_dim, SSD) || heads <= 0 || groups <= 0 || heads % groups || taps < 1 || taps > MAX_TAPS ||
        norm_groups <= 0 || (heads * v_dim) % norm_groups || conv_w == nullptr || conv_b == nullptr || dt_bias == nullptr ||
        a_log == nullptr || d_skip == nullptr || entry_of_token == nullptr ||
        slot_stride < kipp_ssd_state_floats(heads, groups, dim, v_dim, taps))
        return KIPP_ERR_ARG;
    ScanArgs a = {};
    a.out = out; a.ld_out = ld_out; a.proj = proj; a.ld_proj = ld_proj;
    a.z_off = z_off; a.xbc_off = xbc_off; a.dt_off = dt_off; a.taps = taps; a.groups = groups; a.norm_groups = norm_groups;
    a.conv_w = conv_w; a.conv_b = conv_b; a.dt_bias = dt_bias; a.a_log = a_log; a.d_skip = d_skip; a.norm_w = norm_w;
    a.state = state; a.slot_stride = slot_stride; a.q_start = q_start; a.entry_of_token = entry_of_token; a.slots = slots;
    a.heads = heads; a.dim = dim; a.v_dim = v_dim; a.eps = eps; a.k_scale = 1.f; a.out_scale = 1.f;
    a.channels = heads * v_dim + 2 * groups * dim; a.kept_off = (long long)heads * dim * v_dim;
    if (dtype == KIPP_DT_F32) return launch_scan<float, SSD>(a, entries, tokens, scratch, (cudaStream_t)stream, conv_out);
    if (dtype == KIPP_DT_BF16) return launch_scan<bf16, SSD>(a, entries, tokens, scratch, (cudaStream_t)stream, conv_out);
    return KIPP_ERR_DTYPE;
}

// float32 values of state one request slot of the gated delta rule holds: S [heads, dim, v_dim], then the last
// taps - 1 inputs of the 2 * kv_heads * dim + heads * v_dim convolved channels.
extern "C" long long kipp_gated_delta_state_floats(int heads, int kv_heads, int dim, int v_dim, int taps) {
    return (long long)heads * dim * v_dim + (long long)(taps > 1 ? taps - 1 : 0) * (2LL * kv_heads * dim + (long long)heads * v_dim);
}

// The gated delta rule (see the head of this file).  proj [T, ...] holds the channels to convolve [q: kv_heads * dim |
// k: kv_heads * dim | v: heads * v_dim] at qkv_off and the write rates' pre-activations [heads] at b_off; conv_w
// [taps, channels] (the last tap meets the current token); a_raw [T, heads * dim] and g_raw [T, heads * v_dim]
// float32 are the pre-activations of the decay and of the output's gate (1 silu, 2 sigmoid); dt_bias [heads * dim],
// a_log [heads], norm_w [v_dim] float32.  A slot is kipp_gated_delta_state_floats floats.  conv_out: float32
// [tokens, channels] of scratch.  At most 16 taps.
extern "C" int kipp_gated_delta_scan(void* out, long long ld_out, const void* proj, long long ld_proj, int dtype, int qkv_off,
                                     int b_off, const float* conv_w, int taps, const float* a_raw, long long ld_a,
                                     const float* dt_bias, const float* a_log, const float* g_raw, long long ld_g, int gate,
                                     const float* norm_w, float* state, long long slot_stride, const int* q_start,
                                     const int* entry_of_token, const int* slots, int entries, int tokens, int heads, int kv_heads,
                                     int dim, int v_dim, float q_scale, float eps, float out_scale, float* scratch, float* conv_out,
                                     void* stream) {
    if (entries <= 0 || tokens <= 0) return 0;
    if (!kipp_recurrent_scan_ok(dim, v_dim, GATED_DELTA) || heads <= 0 || kv_heads <= 0 || heads % kv_heads || taps < 1 ||
        taps > MAX_TAPS || conv_w == nullptr || a_raw == nullptr || g_raw == nullptr || dt_bias == nullptr || a_log == nullptr ||
        norm_w == nullptr || entry_of_token == nullptr || gate < 1 || gate > 2 || ld_a < (long long)heads * dim ||
        ld_g < (long long)heads * v_dim || slot_stride < kipp_gated_delta_state_floats(heads, kv_heads, dim, v_dim, taps))
        return KIPP_ERR_ARG;
    ScanArgs a = {};
    a.out = out; a.ld_out = ld_out; a.proj = proj; a.ld_proj = ld_proj;
    a.xbc_off = qkv_off; a.b_off = b_off; a.conv_w = conv_w; a.taps = taps; a.groups = kv_heads;
    a.a_raw = a_raw; a.ld_a = ld_a; a.dt_bias = dt_bias; a.a_log = a_log; a.g_raw = g_raw; a.ld_g = ld_g; a.gate = gate; a.norm_w = norm_w;
    a.state = state; a.slot_stride = slot_stride; a.q_start = q_start; a.entry_of_token = entry_of_token; a.slots = slots;
    a.heads = heads; a.dim = dim; a.v_dim = v_dim; a.q_scale = q_scale; a.eps = eps; a.k_scale = 1.f; a.out_scale = out_scale;
    a.channels = 2 * kv_heads * dim + heads * v_dim; a.kept_off = (long long)heads * dim * v_dim;
    if (dtype == KIPP_DT_F32) return launch_scan<float, GATED_DELTA>(a, entries, tokens, scratch, (cudaStream_t)stream, conv_out);
    if (dtype == KIPP_DT_BF16) return launch_scan<bf16, GATED_DELTA>(a, entries, tokens, scratch, (cudaStream_t)stream, conv_out);
    return KIPP_ERR_DTYPE;
}

// Token shift: out[s][t, :] = h[t, :] + (h'[t, :] - h[t, :]) * mu[s, :] for s < n_mix, with h' the row of
// the token before in the same sequence: the row above inside a step's portion, the row the
// sequence's slot keeps (prev[slot * slot_stride ...], float32, zeros at admission) for the portion's
// first token.  kipp_token_shift_keep then stores the portion's last row in the slot.
extern "C" int kipp_token_shift_mix(void* out, long long out_stride, const void* h, const float* mu, const float* prev,
                                    long long slot_stride, const int* q_start, const int* entry_of_token,
                                    const int* slots, int dtype, int tokens, int hidden, int n_mix, void* stream) {
    if (tokens <= 0) return 0;
    if (hidden <= 0 || n_mix <= 0 || n_mix > 8 || prev == nullptr || mu == nullptr) return KIPP_ERR_ARG;
    if (dtype == KIPP_DT_F32)
        return kipp_launch(token_shift_mix_kernel<float>, dim3((unsigned)tokens), dim3(128), 0, (cudaStream_t)stream, 1,
                           (float*)out, out_stride, (const float*)h, mu, prev, slot_stride, q_start, entry_of_token, slots,
                           hidden, n_mix);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(token_shift_mix_kernel<bf16>, dim3((unsigned)tokens), dim3(128), 0, (cudaStream_t)stream, 1,
                           (bf16*)out, out_stride, (const bf16*)h, mu, prev, slot_stride, q_start, entry_of_token, slots,
                           hidden, n_mix);
    return KIPP_ERR_DTYPE;
}
extern "C" int kipp_token_shift_keep(float* prev, long long slot_stride, const void* h, const int* q_start,
                                     const int* slots, int dtype, int entries, int hidden, void* stream) {
    if (entries <= 0) return 0;
    if (hidden <= 0 || prev == nullptr) return KIPP_ERR_ARG;
    if (dtype == KIPP_DT_F32)
        return kipp_launch(token_shift_keep_kernel<float>, dim3((unsigned)entries), dim3(128), 0, (cudaStream_t)stream, 1,
                           prev, slot_stride, (const float*)h, q_start, slots, hidden);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(token_shift_keep_kernel<bf16>, dim3((unsigned)entries), dim3(128), 0, (cudaStream_t)stream, 1,
                           prev, slot_stride, (const bf16*)h, q_start, slots, hidden);
    return KIPP_ERR_DTYPE;
}

// out[r, c] = tanh(in[r, c]) in the compute type (the bottleneck of a low-rank projection).
extern "C" int kipp_tanh_rows(void* out, long long ld_out, const void* in, long long ld_in, int dtype, int rows,
                              int cols, void* stream) {
    if (rows <= 0 || cols <= 0) return 0;
    const long long n = (long long)rows * cols;
    const dim3 grid((unsigned)((n + 255) / 256));
    if (dtype == KIPP_DT_F32)
        return kipp_launch(tanh_rows_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, 1, (float*)out, ld_out,
                           (const float*)in, ld_in, rows, cols);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(tanh_rows_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)stream, 1, (bf16*)out, ld_out,
                           (const bf16*)in, ld_in, rows, cols);
    return KIPP_ERR_DTYPE;
}
