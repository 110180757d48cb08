// Embedding gather, RMSNorm, layer norm, PolyNorm and element-wise activations.
//
// Reference counterparts: embed_kernel (cuda/kipp_kernels.cu:35) handles one
// token per launch, rms_norm_kernel (cuda/kipp_kernels.cu:44) one row in one
// block.  These take any number of tokens / rows per launch.
#include "common.cuh"
#include <algorithm>

// out[t, :] = float(table[ids[t], :]) * scale.  The residual stream is float32.
template <typename TW>
__global__ void embed_gather_kernel(float* __restrict__ out, const TW* __restrict__ table,
                                    const int* __restrict__ ids, int hidden, int vocab, float scale,
                                    int* __restrict__ status) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int id = ids[t];
    if (id < 0 || id >= vocab) {           // never read outside the table
        if (threadIdx.x == 0) atomicExch(status, 1);
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[(size_t)t * hidden + i] = 0.f;
        return;
    }
    const TW* row = table + (size_t)id * hidden;
    float* dst = out + (size_t)t * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = to_f32(row[i]) * scale;
}

extern "C" int kipp_embed_gather_scaled(float* out, const void* table, int table_dtype, const int* ids,
                                        int tokens, int hidden, int vocab, float scale, int* status, void* stream) {
    if (tokens <= 0) return 0;
    if (hidden <= 0 || vocab <= 0) return KIPP_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = hidden >= 1024 ? 256 : 128;
    if (table_dtype == KIPP_DT_F32)
        return kipp_launch(embed_gather_kernel<float>, dim3(tokens), dim3(threads), 0, s, 1, out,
                           (const float*)table, ids, hidden, vocab, scale, status);
    if (table_dtype == KIPP_DT_BF16)
        return kipp_launch(embed_gather_kernel<bf16>, dim3(tokens), dim3(threads), 0, s, 1, out,
                           (const bf16*)table, ids, hidden, vocab, scale, status);
    return KIPP_ERR_DTYPE;
}
extern "C" int kipp_embed_gather(float* out, const void* table, int table_dtype, const int* ids,
                                 int tokens, int hidden, int vocab, int* status, void* stream) {
    return kipp_embed_gather_scaled(out, table, table_dtype, ids, tokens, hidden, vocab, 1.0f, status, stream);
}

// y[r, i] = x[src(r), i] * rsqrt(mean(x[src(r), :]^2) + eps) * w[i]
// (src/kipp.c:2221-2231).  Sum of squares and scale in float32.  `rows`, when
// not null, gathers the input rows (used for the rows whose logits are wanted).
template <typename TO>
__global__ void rmsnorm_kernel(TO* __restrict__ out, const float* __restrict__ x,
                               const void* __restrict__ w, int w_dtype, const int* __restrict__ rows,
                               int size, float eps, float* __restrict__ ssq_out) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const float* src = x + (size_t)(rows ? rows[r] : r) * size;
    float ss = 0.f;
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        const float v = src[i];
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    // deferred form: x * w alone goes out, the sum of squares beside it (see kipp_rmsnorm_deferred)
    const float scale = ssq_out ? 1.0f : 1.0f / sqrtf(ss / (float)size + eps);
    if (ssq_out && threadIdx.x == 0) ssq_out[r] = ss;
    TO* dst = out + (size_t)r * size;
    for (int i = threadIdx.x; i < size; i += blockDim.x)
        dst[i] = from_f32<TO>(src[i] * scale * load_w(w, w_dtype, i));
}

// Vector path: size a multiple of 4 and at most 4096; each of 256 threads keeps
// its float4 pieces of the row in registers, so the row is read once.
template <typename TO>
__global__ void __launch_bounds__(256)
rmsnorm_vec_kernel(TO* __restrict__ out, const float* __restrict__ x, const void* __restrict__ w, int w_dtype,
                   const int* __restrict__ rows, int size, float eps, float* __restrict__ ssq_out) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const float4* src = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * size);
    const int n4 = size >> 2;
    float4 v[4];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int i = threadIdx.x + 256 * j;
        if (i < n4) {
            v[j] = src[i];
            ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
        }
    }
    ss = block_sum(ss, scratch);
    const float scale = ssq_out ? 1.0f : 1.0f / sqrtf(ss / (float)size + eps);
    if (ssq_out && threadIdx.x == 0) ssq_out[r] = ss;
    TO* dst = out + (size_t)r * size;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int i = threadIdx.x + 256 * j;
        if (i < n4) {
            const size_t e = (size_t)i * 4;
            const float a = v[j].x * scale * load_w(w, w_dtype, e), b = v[j].y * scale * load_w(w, w_dtype, e + 1);
            const float c = v[j].z * scale * load_w(w, w_dtype, e + 2), d = v[j].w * scale * load_w(w, w_dtype, e + 3);
            if (sizeof(TO) == 4) {
                *reinterpret_cast<float4*>(reinterpret_cast<float*>(dst) + e) = make_float4(a, b, c, d);
            } else {
                __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
                uint2 packed;
                packed.x = *reinterpret_cast<uint32_t*>(&lo);
                packed.y = *reinterpret_cast<uint32_t*>(&hi);
                *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(dst) + e) = packed;
            }
        }
    }
}

static int rmsnorm_launch(void* out, int out_dtype, const float* x, const void* w, int w_dtype, const int* rows,
                          int n_rows, int size, float eps, float* ssq_out, void* stream) {
    if (n_rows <= 0) return 0;
    if (size <= 0) return KIPP_ERR_ARG;
    if (w_dtype != KIPP_DT_F32 && w_dtype != KIPP_DT_BF16) return KIPP_ERR_DTYPE;
    cudaStream_t s = (cudaStream_t)stream;
    if (size % 4 == 0 && size <= 4096 && size >= 256 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)out & 15) == 0) {
        if (out_dtype == KIPP_DT_F32)
            return kipp_launch(rmsnorm_vec_kernel<float>, dim3(n_rows), dim3(256), 0, s, 1, (float*)out, x, w,
                               w_dtype, rows, size, eps, ssq_out);
        if (out_dtype == KIPP_DT_BF16)
            return kipp_launch(rmsnorm_vec_kernel<bf16>, dim3(n_rows), dim3(256), 0, s, 1, (bf16*)out, x, w,
                               w_dtype, rows, size, eps, ssq_out);
        return KIPP_ERR_DTYPE;
    }
    int threads = size >= 2048 ? 512 : (size >= 512 ? 256 : 64);
    if (out_dtype == KIPP_DT_F32)
        return kipp_launch(rmsnorm_kernel<float>, dim3(n_rows), dim3(threads), 0, s, 1, (float*)out, x, w, w_dtype,
                           rows, size, eps, ssq_out);
    if (out_dtype == KIPP_DT_BF16)
        return kipp_launch(rmsnorm_kernel<bf16>, dim3(n_rows), dim3(threads), 0, s, 1, (bf16*)out, x, w, w_dtype,
                           rows, size, eps, ssq_out);
    return KIPP_ERR_DTYPE;
}

extern "C" int kipp_rmsnorm(void* out, int out_dtype, const float* x, const void* w, int w_dtype,
                            const int* rows, int n_rows, int size, float eps, void* stream) {
    return rmsnorm_launch(out, out_dtype, x, w, w_dtype, rows, n_rows, size, eps, nullptr, stream);
}

// The norm with its per-row factor left to whoever reads the result: out[r, i] = x[row r, i] * w[i]
// (rounded to out's type) and ssq_out[r] = sum of x[row r, :]^2, so that
// rmsnorm(x)[r] = out[r] / sqrt(ssq_out[r] / size + eps).  A matrix product that follows applies
// the factor to its own result rows in float32 (kipp_gemm_tc_fold); a residual add that leaves
// x * w itself (the same kernel library) rounds the same values the same way, so both routes to
// the product's input agree to the bit.
extern "C" int kipp_rmsnorm_deferred(void* out, int out_dtype, float* ssq_out, const float* x, const void* w,
                                     int w_dtype, const int* rows, int n_rows, int size, void* stream) {
    if (ssq_out == nullptr) return KIPP_ERR_ARG;
    return rmsnorm_launch(out, out_dtype, x, w, w_dtype, rows, n_rows, size, 0.f, ssq_out, stream);
}

// ---------------------------------------------------------------------------
// PolyNorm activation over each row of z [rows, n]:
//   y = c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3,
// powers taken element by element, N(x) = x / sqrt(mean(x^2) + eps) over the
// row.  The three mean squares (of z, z^2 and z^3) and the polynomial are
// float32; z arrives and y leaves in the compute type.  One block per row.
template <typename T>
__global__ void __launch_bounds__(256)
polynorm_kernel(T* __restrict__ out, long long ld_out, const T* __restrict__ z, long long ld_z,
                const float* __restrict__ coef, int n, float eps) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const T* src = z + (size_t)blockIdx.x * ld_z;
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = to_f32(src[i]);
        const float v2 = v * v, v3 = v2 * v;
        s2 += v2;
        s4 = fmaf(v2, v2, s4);
        s6 = fmaf(v3, v3, s6);
    }
    s2 = block_sum(s2, scratch);
    s4 = block_sum(s4, scratch);
    s6 = block_sum(s6, scratch);
    const float inv_n = 1.0f / (float)n;
    const float r1 = coef[0] / sqrtf(s2 * inv_n + eps), r2 = coef[1] / sqrtf(s4 * inv_n + eps);
    const float r3 = coef[2] / sqrtf(s6 * inv_n + eps), c3 = coef[3];
    T* dst = out + (size_t)blockIdx.x * ld_out;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = to_f32(src[i]);
        const float v2 = v * v;
        dst[i] = from_f32<T>(fmaf(r1, v, fmaf(r2, v2, fmaf(r3, v2 * v, c3))));
    }
}

extern "C" int kipp_polynorm(void* out, long long ld_out, const void* z, long long ld_z, int dtype,
                             const float* coef, int rows, int n, float eps, void* stream) {
    if (rows <= 0) return 0;
    if (n <= 0 || coef == nullptr) return KIPP_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = n >= 1024 ? 256 : 128;
    if (dtype == KIPP_DT_F32)
        return kipp_launch(polynorm_kernel<float>, dim3(rows), dim3(threads), 0, s, 1, (float*)out, ld_out,
                           (const float*)z, ld_z, coef, n, eps);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(polynorm_kernel<bf16>, dim3(rows), dim3(threads), 0, s, 1, (bf16*)out, ld_out,
                           (const bf16*)z, ld_z, coef, n, eps);
    return KIPP_ERR_DTYPE;
}

// x += y over n float32 values (the embedding output fed back into the residual stream).
__global__ void add_f32_kernel(float* __restrict__ x, const float* __restrict__ y, long long n) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] += y[i];
}

extern "C" int kipp_add_f32(float* x, const float* y, long long n, void* stream) {
    if (n <= 0) return 0;
    const long long blocks = (n + 255) / 256;
    if (blocks > 0x7fffffffLL) return KIPP_ERR_ARG;
    return kipp_launch(add_f32_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, 1, x, y, n);
}

// ---------------------------------------------------------------------------
// Layer norm with weight and bias: y[r, i] = (x[src(r), i] - mean) / sqrt(var + eps) * w[i] + b[i],
// var = the mean of the squared deviations (two passes over the row, which a block keeps in
// shared memory), all of it float32.  `rows`, when not null, gathers the input rows; b may be null.
template <typename TO>
__global__ void __launch_bounds__(256)
layernorm_kernel(TO* __restrict__ out, const float* __restrict__ x, const float* __restrict__ w,
                 const float* __restrict__ b, const int* __restrict__ rows, int size, float eps) {
    extern __shared__ float row[];
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const float* src = x + (size_t)(rows ? rows[r] : r) * size;
    float s = 0.f;
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        const float v = src[i];
        row[i] = v;
        s += v;
    }
    const float mean = block_sum(s, scratch) / (float)size;
    float ss = 0.f;
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        const float d = row[i] - mean;
        ss = fmaf(d, d, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)size + eps);
    TO* dst = out + (size_t)r * size;
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        const float y = (row[i] - mean) * inv * w[i];
        dst[i] = from_f32<TO>(b ? y + b[i] : y);
    }
}

extern "C" int kipp_layernorm(void* out, int out_dtype, const float* x, const float* w, const float* b,
                              const int* rows, int n_rows, int size, float eps, void* stream) {
    if (n_rows <= 0) return 0;
    if (size <= 0 || size > 48 * 1024 / 4 || w == nullptr) return KIPP_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = size >= 1024 ? 256 : 128;
    const size_t smem = (size_t)size * sizeof(float);
    if (out_dtype == KIPP_DT_F32)
        return kipp_launch(layernorm_kernel<float>, dim3(n_rows), dim3(threads), smem, s, 1, (float*)out, x, w, b, rows,
                           size, eps);
    if (out_dtype == KIPP_DT_BF16)
        return kipp_launch(layernorm_kernel<bf16>, dim3(n_rows), dim3(threads), smem, s, 1, (bf16*)out, x, w, b, rows,
                           size, eps);
    return KIPP_ERR_DTYPE;
}

// ---------------------------------------------------------------------------
// Activations applied element by element to z [rows, n] in the compute type, arithmetic in
// float32: 0 relu, 1 the square of relu, 2 gelu with the tanh form
// 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), 3 silu.
template <typename T>
__global__ void activation_kernel(T* __restrict__ out, long long ld_out, const T* __restrict__ z, long long ld_z,
                                  int rows, int n, int kind) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * n) return;
    const long long r = i / n, c = i % n;
    out[r * ld_out + c] = from_f32<T>(kipp_activation(to_f32(z[r * ld_z + c]), kind));
}

extern "C" int kipp_activation(void* out, long long ld_out, const void* z, long long ld_z, int dtype, int rows,
                               int n, int kind, void* stream) {
    if (rows <= 0 || n <= 0) return 0;
    if (kind < 0 || kind > 3) return KIPP_ERR_ARG;
    const long long total = (long long)rows * n, blocks = (total + 255) / 256;
    if (blocks > 0x7fffffffLL) return KIPP_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == KIPP_DT_F32)
        return kipp_launch(activation_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, s, 1, (float*)out, ld_out,
                           (const float*)z, ld_z, rows, n, kind);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(activation_kernel<bf16>, dim3((unsigned)blocks), dim3(256), 0, s, 1, (bf16*)out, ld_out,
                           (const bf16*)z, ld_z, rows, n, kind);
    return KIPP_ERR_DTYPE;
}

// ---------------------------------------------------------------------------
// A second embedding table addressed by a hash of the token pair: x[t, :] += table[row(t), :] with
// row = (previous token * mul_prev + token * mul_cur) mod buckets, and row = buckets (the table's
// extra last row) for the token at position 0 of its sequence.  The previous token of a step's
// first token is the one the sequence's slot keeps (last_token[slot * stride], written by
// kipp_keep_last_token after this kernel: the token before is part of a sequence's state).
template <typename TW>
__global__ void hashed_pair_add_kernel(float* __restrict__ x, const TW* __restrict__ table,
                                       const int* __restrict__ ids, const int* __restrict__ positions,
                                       const int* __restrict__ entry_of_token, const int* __restrict__ q_start,
                                       const int* __restrict__ slots, const int* __restrict__ last_token,
                                       long long stride, int hidden, int vocab, long long buckets, long long mul_prev,
                                       long long mul_cur, int* __restrict__ status) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int id = ids[t], e = entry_of_token[t];
    long long row = buckets;
    if (positions[t] > 0) {
        const int prev = t > q_start[e] ? ids[t - 1] : last_token[(size_t)slots[e] * stride];
        if (id < 0 || id >= vocab || prev < 0 || prev >= vocab) {      // never read outside the table
            if (threadIdx.x == 0) atomicExch(status, 1);
            return;
        }
        row = ((long long)prev * mul_prev + (long long)id * mul_cur) % buckets;
    }
    const TW* src = table + (size_t)row * hidden;
    float* dst = x + (size_t)t * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] += to_f32(src[i]);
}

extern "C" int kipp_hashed_pair_add(float* x, const void* table, int table_dtype, const int* ids, const int* positions,
                                    const int* entry_of_token, const int* q_start, const int* slots,
                                    const int* last_token, long long stride, int tokens, int hidden, int vocab,
                                    long long buckets, long long mul_prev, long long mul_cur, int* status, void* stream) {
    if (tokens <= 0) return 0;
    if (hidden <= 0 || vocab <= 0 || buckets <= 0 || mul_prev < 0 || mul_cur < 0 || last_token == nullptr || stride <= 0)
        return KIPP_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = hidden >= 1024 ? 256 : 128;
    if (table_dtype == KIPP_DT_F32)
        return kipp_launch(hashed_pair_add_kernel<float>, dim3(tokens), dim3(threads), 0, s, 1, x, (const float*)table, ids,
                           positions, entry_of_token, q_start, slots, last_token, stride, hidden, vocab, buckets, mul_prev,
                           mul_cur, status);
    if (table_dtype == KIPP_DT_BF16)
        return kipp_launch(hashed_pair_add_kernel<bf16>, dim3(tokens), dim3(threads), 0, s, 1, x, (const bf16*)table, ids,
                           positions, entry_of_token, q_start, slots, last_token, stride, hidden, vocab, buckets, mul_prev,
                           mul_cur, status);
    return KIPP_ERR_DTYPE;
}

// last_token[slots[e] * stride] = the last token entry e brings in this step.
__global__ void keep_last_token_kernel(int* __restrict__ last_token, long long stride, const int* __restrict__ ids,
                                       const int* __restrict__ q_start, const int* __restrict__ slots, int entries) {
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x * blockDim.x + threadIdx.x;
    if (e < entries && q_start[e + 1] > q_start[e]) last_token[(size_t)slots[e] * stride] = ids[q_start[e + 1] - 1];
}

extern "C" int kipp_keep_last_token(int* last_token, long long stride, const int* ids, const int* q_start,
                                    const int* slots, int entries, void* stream) {
    if (entries <= 0) return 0;
    if (last_token == nullptr || stride <= 0) return KIPP_ERR_ARG;
    return kipp_launch(keep_last_token_kernel, dim3((unsigned)((entries + 127) / 128)), dim3(128), 0, (cudaStream_t)stream, 1,
                       last_token, stride, ids, q_start, slots, entries);
}

// ---------------------------------------------------------------------------
// x[r, :] += mult * y[r, :] * rsqrt(mean(y[r, :]^2) + eps) * w: the RMS norm of a sublayer's OUTPUT
// joins the residual stream, all of it float32 (w keeps its storage type).  `copy` (or null) takes
// the new x rounded to bfloat16: the input of the sublayer that reads the stream next.
__global__ void __launch_bounds__(256)
rmsnorm_scaled_add_kernel(float* __restrict__ x, const float* __restrict__ y, const void* __restrict__ w, int w_dtype,
                          int size, float eps, float mult, bf16* __restrict__ copy, int vec) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const float* src = y + (size_t)blockIdx.x * size;
    float* dst = x + (size_t)blockIdx.x * size;
    bf16* cp = copy ? copy + (size_t)blockIdx.x * size : nullptr;
    float ss = 0.f;
    if (vec) {
        // four neighbouring values per thread and step; the order of a row's sum depends on its size only
        for (int i = 4 * threadIdx.x; i < size; i += 4 * blockDim.x) {
            const float4 v = *reinterpret_cast<const float4*>(src + i);
            ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
        }
    } else {
        for (int i = threadIdx.x; i < size; i += blockDim.x) ss = fmaf(src[i], src[i], ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)size + eps);
    auto weight = [&](int i) {
        return w_dtype == KIPP_DT_F32 ? static_cast<const float*>(w)[i] : to_f32(static_cast<const bf16*>(w)[i]);
    };
    if (vec) {
        for (int i = 4 * threadIdx.x; i < size; i += 4 * blockDim.x) {
            const float4 v = *reinterpret_cast<const float4*>(src + i);
            float4 o = *reinterpret_cast<const float4*>(dst + i);
            o.x += mult * (v.x * inv * weight(i));
            o.y += mult * (v.y * inv * weight(i + 1));
            o.z += mult * (v.z * inv * weight(i + 2));
            o.w += mult * (v.w * inv * weight(i + 3));
            *reinterpret_cast<float4*>(dst + i) = o;
            if (cp) {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(o.x, o.y), hi = __floats2bfloat162_rn(o.z, o.w);
                uint2 pk;
                pk.x = *reinterpret_cast<const uint32_t*>(&lo);
                pk.y = *reinterpret_cast<const uint32_t*>(&hi);
                *reinterpret_cast<uint2*>(cp + i) = pk;
            }
        }
    } else {
        for (int i = threadIdx.x; i < size; i += blockDim.x) {
            const float o = dst[i] + mult * (src[i] * inv * weight(i));
            dst[i] = o;
            if (cp) cp[i] = __float2bfloat16_rn(o);
        }
    }
}

extern "C" int kipp_rmsnorm_scaled_add(float* x, const float* y, const void* w, int w_dtype, int rows, int size, float eps,
                                       float mult, void* copy_bf16, void* stream) {
    if (rows <= 0) return 0;
    if (size <= 0 || !(eps > 0.f) || (w_dtype != KIPP_DT_F32 && w_dtype != KIPP_DT_BF16)) return KIPP_ERR_ARG;
    const int vec = size % 4 == 0 && (((uintptr_t)x | (uintptr_t)y) & 15) == 0 && ((uintptr_t)copy_bf16 & 7) == 0;
    return kipp_launch(rmsnorm_scaled_add_kernel, dim3((unsigned)rows), dim3(size >= 1024 ? 256 : 128), 0, (cudaStream_t)stream,
                       1, x, y, w, w_dtype, size, eps, mult, (bf16*)copy_bf16, vec);
}

// x[r, :] += mult * y[r, :] * rsqrt(mean(y^2) + eps_y) * w_y, and of the new x h[r, :] = x * rsqrt(mean(x^2) + eps_h) * w_h:
// the norm of a sublayer's OUTPUT joins the stream and the norm of the next sublayer's INPUT leaves the same pass
// (blocks with a norm on either side of every sublayer).  All float32, h in the compute type; w keeps its storage
// type.  clear: y is left zeroed for the sublayer that adds its output into it next.  A block per row; a thread keeps
// its first 4 KEPT values in registers between the three passes over a row, what lies beyond them is read again.
namespace {
constexpr int NORM_KEPT = 4;
__device__ __forceinline__ float4 weights4(const void* w, int w_dtype, int i) {
    if (w_dtype == KIPP_DT_F32) return *reinterpret_cast<const float4*>(static_cast<const float*>(w) + i);
    const uint2 v = *reinterpret_cast<const uint2*>(static_cast<const bf16*>(w) + i);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                       __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ float squares4(float4 v, float ss) {
    ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss);
    return fmaf(v.w, v.w, ss);
}
__device__ __forceinline__ void store4(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
__device__ __forceinline__ void store4(bf16* dst, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 pk;
    pk.x = *reinterpret_cast<const uint32_t*>(&lo);
    pk.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(dst) = pk;
}

template <typename TO>
__global__ void __launch_bounds__(512)
norm_add_norm_kernel(float* __restrict__ x, float* __restrict__ y, int clear, const void* __restrict__ w_y, int w_y_dtype,
                     float eps_y, float mult, const void* __restrict__ w_h, int w_h_dtype, float eps_h, TO* __restrict__ h,
                     int size, int vec) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    float* yr = y + (size_t)blockIdx.x * size;
    float* xr = x + (size_t)blockIdx.x * size;
    TO* hr = h + (size_t)blockIdx.x * size;
    const int tid = threadIdx.x, step = blockDim.x;
    if (!vec) {
        float ss = 0.f;
        for (int i = tid; i < size; i += step) ss = fmaf(yr[i], yr[i], ss);
        const float inv = mult / sqrtf(block_sum(ss, scratch) / (float)size + eps_y);
        ss = 0.f;
        for (int i = tid; i < size; i += step) {
            const float o = fmaf(yr[i] * inv, load_w(w_y, w_y_dtype, i), xr[i]);
            xr[i] = o;
            if (clear) yr[i] = 0.f;
            ss = fmaf(o, o, ss);
        }
        const float inv_h = 1.0f / sqrtf(block_sum(ss, scratch) / (float)size + eps_h);
        for (int i = tid; i < size; i += step) hr[i] = from_f32<TO>(xr[i] * inv_h * load_w(w_h, w_h_dtype, i));
        return;
    }
    float4 keep[NORM_KEPT], stream[NORM_KEPT];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NORM_KEPT; ++j) {
        const int i = 4 * (tid + j * step);
        keep[j] = i < size ? *reinterpret_cast<const float4*>(yr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        stream[j] = i < size ? *reinterpret_cast<const float4*>(xr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss = squares4(keep[j], ss);
    }
    for (int i = 4 * (tid + NORM_KEPT * step); i < size; i += 4 * step) ss = squares4(*reinterpret_cast<const float4*>(yr + i), ss);
    const float inv = mult / sqrtf(block_sum(ss, scratch) / (float)size + eps_y);
    auto joined = [&](float4 v, float4 o, int i) {
        const float4 w = weights4(w_y, w_y_dtype, i);
        o.x = fmaf(v.x * inv, w.x, o.x); o.y = fmaf(v.y * inv, w.y, o.y);
        o.z = fmaf(v.z * inv, w.z, o.z); o.w = fmaf(v.w * inv, w.w, o.w);
        *reinterpret_cast<float4*>(xr + i) = o;
        if (clear) *reinterpret_cast<float4*>(yr + i) = make_float4(0.f, 0.f, 0.f, 0.f);
        return o;
    };
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < NORM_KEPT; ++j) {
        const int i = 4 * (tid + j * step);
        if (i < size) {
            keep[j] = joined(keep[j], stream[j], i);
            ss = squares4(keep[j], ss);
        }
    }
    for (int i = 4 * (tid + NORM_KEPT * step); i < size; i += 4 * step)
        ss = squares4(joined(*reinterpret_cast<const float4*>(yr + i), *reinterpret_cast<const float4*>(xr + i), i), ss);
    const float inv_h = 1.0f / sqrtf(block_sum(ss, scratch) / (float)size + eps_h);
    auto normed = [&](float4 o, int i) {
        const float4 w = weights4(w_h, w_h_dtype, i);
        store4(hr + i, make_float4(o.x * inv_h * w.x, o.y * inv_h * w.y, o.z * inv_h * w.z, o.w * inv_h * w.w));
    };
#pragma unroll
    for (int j = 0; j < NORM_KEPT; ++j) {
        const int i = 4 * (tid + j * step);
        if (i < size) normed(keep[j], i);
    }
    for (int i = 4 * (tid + NORM_KEPT * step); i < size; i += 4 * step) normed(*reinterpret_cast<const float4*>(xr + i), i);
}
}  // namespace

extern "C" int kipp_norm_add_norm(float* x, float* y, int clear, const void* w_y, int w_y_dtype, float eps_y, float mult,
                                  const void* w_h, int w_h_dtype, float eps_h, void* h, int h_dtype, int rows, int size,
                                  void* stream) {
    if (rows <= 0) return 0;
    if (size <= 0 || !(eps_y > 0.f) || !(eps_h > 0.f) || (w_y_dtype != KIPP_DT_F32 && w_y_dtype != KIPP_DT_BF16) ||
        (w_h_dtype != KIPP_DT_F32 && w_h_dtype != KIPP_DT_BF16))
        return KIPP_ERR_ARG;
    const int vec = size % 4 == 0 && (((uintptr_t)x | (uintptr_t)y | (uintptr_t)h | (uintptr_t)w_y | (uintptr_t)w_h) & 15) == 0;
    const dim3 grid((unsigned)rows), block(size >= 4096 ? 512 : size >= 1024 ? 256 : 128);
    cudaStream_t s = (cudaStream_t)stream;
    if (h_dtype == KIPP_DT_F32)
        return kipp_launch(norm_add_norm_kernel<float>, grid, block, 0, s, 1, x, y, clear, w_y, w_y_dtype, eps_y, mult, w_h, w_h_dtype,
                           eps_h, (float*)h, size, vec);
    if (h_dtype == KIPP_DT_BF16)
        return kipp_launch(norm_add_norm_kernel<bf16>, grid, block, 0, s, 1, x, y, clear, w_y, w_y_dtype, eps_y, mult, w_h, w_h_dtype,
                           eps_h, (bf16*)h, size, vec);
    return KIPP_ERR_DTYPE;
}

// One pass over the residual stream: x[r, :] += mult * sum_b y_b[r, :] * rsqrt(mean(y_b^2) + eps_b) * w_b for up to two
// outputs y_b that join it normed, and of the new x up to two norms h_q[r, :] = x * rsqrt(mean(x^2) + eps_q) * w_q (what
// sublayers of the next block read) and its rounded copy.  All float32, h and the copy in the compute type; weights keep
// their storage type.  A block per row; a thread keeps its first 4 JOIN_KEPT values of every array in registers between
// the passes over a row, what lies beyond them is read again.  (The layout is the host's Ops::Join.)
namespace {
struct JoinArgs {
    float* x;
    const float* y[2];
    const void* w_y[2];
    void* h[2];
    const void* w_h[2];
    void* copy;
    int w_y_dtype[2], w_h_dtype[2];
    float eps_y[2], eps_h[2];
    float mult;
    int size;
};
constexpr int JOIN_KEPT = 2;

// four values of a row at column i (fewer at the end of a row that does not go by fours: VEC false)
template <bool VEC> __device__ __forceinline__ float4 load_four(const float* p, int i, int n) {
    if (VEC) return *reinterpret_cast<const float4*>(p + i);
    return make_float4(p[i], i + 1 < n ? p[i + 1] : 0.f, i + 2 < n ? p[i + 2] : 0.f, i + 3 < n ? p[i + 3] : 0.f);
}
template <bool VEC> __device__ __forceinline__ float4 weight_four(const void* w, int dtype, int i, int n) {
    if (VEC) return weights4(w, dtype, i);
    return make_float4(load_w(w, dtype, i), i + 1 < n ? load_w(w, dtype, i + 1) : 0.f, i + 2 < n ? load_w(w, dtype, i + 2) : 0.f,
                       i + 3 < n ? load_w(w, dtype, i + 3) : 0.f);
}
template <bool VEC, typename TO> __device__ __forceinline__ void store_four(TO* p, int i, int n, float4 v) {
    if (VEC) {
        store4(p + i, v);
        return;
    }
    const float e[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int k = 0; k < 4; ++k)
        if (i + k < n) p[i + k] = from_f32<TO>(e[k]);
}

template <typename TO, int NY, bool VEC>
__global__ void __launch_bounds__(512)
stream_join_kernel(const JoinArgs a) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int n = a.size, tid = threadIdx.x, step = 4 * blockDim.x;
    const size_t row = (size_t)blockIdx.x * n;
    float* xr = a.x + row;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 xs[JOIN_KEPT], ys[NY > 0 ? NY : 1][JOIN_KEPT];
    float inv[NY > 0 ? NY : 1];
#pragma unroll
    for (int j = 0; j < JOIN_KEPT; ++j) {
        const int i = 4 * tid + j * step;
        xs[j] = i < n ? load_four<VEC>(xr, i, n) : zero;
#pragma unroll
        for (int b = 0; b < NY; ++b) ys[b][j] = i < n ? load_four<VEC>(a.y[b] + row, i, n) : zero;
    }
#pragma unroll
    for (int b = 0; b < NY; ++b) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < JOIN_KEPT; ++j) ss = squares4(ys[b][j], ss);
        for (int i = 4 * tid + JOIN_KEPT * step; i < n; i += step) ss = squares4(load_four<VEC>(a.y[b] + row, i, n), ss);
        inv[b] = a.mult / sqrtf(block_sum(ss, scratch) / (float)n + a.eps_y[b]);
    }
    auto joined = [&](float4 x, const float4* y, int i) {
#pragma unroll
        for (int b = 0; b < NY; ++b) {
            const float4 w = weight_four<VEC>(a.w_y[b], a.w_y_dtype[b], i, n);
            x.x = fmaf(y[b].x * inv[b], w.x, x.x); x.y = fmaf(y[b].y * inv[b], w.y, x.y);
            x.z = fmaf(y[b].z * inv[b], w.z, x.z); x.w = fmaf(y[b].w * inv[b], w.w, x.w);
        }
        if (NY > 0) store_four<VEC>(xr, i, n, x);
        if (a.copy != nullptr) store_four<VEC>(static_cast<TO*>(a.copy) + row, i, n, x);
        return x;
    };
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < JOIN_KEPT; ++j) {
        const int i = 4 * tid + j * step;
        if (i < n) {
            float4 y[NY > 0 ? NY : 1];
#pragma unroll
            for (int b = 0; b < NY; ++b) y[b] = ys[b][j];
            xs[j] = joined(xs[j], y, i);
            ss = squares4(xs[j], ss);
        }
    }
    for (int i = 4 * tid + JOIN_KEPT * step; i < n; i += step) {
        float4 y[NY > 0 ? NY : 1];
#pragma unroll
        for (int b = 0; b < NY; ++b) y[b] = load_four<VEC>(a.y[b] + row, i, n);
        ss = squares4(joined(load_four<VEC>(xr, i, n), y, i), ss);
    }
    if (a.h[0] == nullptr) return;
    const float mean = block_sum(ss, scratch) / (float)n;
#pragma unroll
    for (int q = 0; q < 2; ++q) {
        if (a.h[q] == nullptr) continue;
        TO* hr = static_cast<TO*>(a.h[q]) + row;
        const float f = 1.0f / sqrtf(mean + a.eps_h[q]);
        auto normed = [&](float4 x, int i) {
            const float4 w = weight_four<VEC>(a.w_h[q], a.w_h_dtype[q], i, n);
            store_four<VEC>(hr, i, n, make_float4(x.x * f * w.x, x.y * f * w.y, x.z * f * w.z, x.w * f * w.w));
        };
#pragma unroll
        for (int j = 0; j < JOIN_KEPT; ++j) {
            const int i = 4 * tid + j * step;
            if (i < n) normed(xs[j], i);
        }
        for (int i = 4 * tid + JOIN_KEPT * step; i < n; i += step) normed(load_four<VEC>(xr, i, n), i);
    }
}

template <typename TO>
int launch_stream_join(const JoinArgs& a, int ny, bool vec, int rows, cudaStream_t s) {
    const dim3 grid((unsigned)rows), block(std::min(512, std::max(64, (a.size / (4 * JOIN_KEPT) + 31) / 32 * 32)));
#define KIPP_JOIN(N) \
    return vec ? kipp_launch(stream_join_kernel<TO, N, true>, grid, block, 0, s, 1, a) : kipp_launch(stream_join_kernel<TO, N, false>, grid, block, 0, s, 1, a)
    if (ny == 0) KIPP_JOIN(0);
    if (ny == 1) KIPP_JOIN(1);
    KIPP_JOIN(2);
#undef KIPP_JOIN
}

// g[t, k] = gelu(z[t, k]) * e with e the token's row of the table from column `off` on; zeros from dim up to ld_g
template <typename T>
__global__ void token_side_gate_kernel(T* __restrict__ g, long long ld_g, const float* __restrict__ z, long long ld_z,
                                       const T* __restrict__ table, long long ld_table, int off, const int* __restrict__ ids,
                                       int tokens, int dim, int vocab) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= tokens * ld_g) return;
    const long long t = i / ld_g;
    const int k = (int)(i % ld_g), id = ids[t];
    float v = 0.f;
    if (k < dim && id >= 0 && id < vocab)                  // (the embedding stage reports ids outside the vocabulary)
        v = kipp_activation(z[t * ld_z + k], 2) * to_f32(table[(size_t)id * ld_table + off + k]);
    g[i] = from_f32<T>(v);
}
}  // namespace

extern "C" int kipp_stream_join(const void* join, int dtype, int rows, void* stream) {
    if (rows <= 0) return 0;
    if (join == nullptr) return KIPP_ERR_ARG;
    const JoinArgs a = *static_cast<const JoinArgs*>(join);
    if (a.x == nullptr || a.size <= 0 || (a.y[0] == nullptr && a.y[1] != nullptr) || (a.h[0] == nullptr && a.h[1] != nullptr))
        return KIPP_ERR_ARG;
    const int ny = a.y[1] != nullptr ? 2 : a.y[0] != nullptr ? 1 : 0;
    uintptr_t at = (uintptr_t)a.x | (uintptr_t)a.copy;
    for (int b = 0; b < 2; ++b) {
        if (a.y[b] != nullptr && (a.w_y[b] == nullptr || !(a.eps_y[b] > 0.f) || (a.w_y_dtype[b] != KIPP_DT_F32 && a.w_y_dtype[b] != KIPP_DT_BF16)))
            return KIPP_ERR_ARG;
        if (a.h[b] != nullptr && (a.w_h[b] == nullptr || !(a.eps_h[b] > 0.f) || (a.w_h_dtype[b] != KIPP_DT_F32 && a.w_h_dtype[b] != KIPP_DT_BF16)))
            return KIPP_ERR_ARG;
        at |= (uintptr_t)a.y[b] | (uintptr_t)a.h[b] | (a.y[b] ? (uintptr_t)a.w_y[b] : 0) | (a.h[b] ? (uintptr_t)a.w_h[b] : 0);
    }
    const bool vec = a.size % 4 == 0 && (at & 15) == 0;
    if (dtype == KIPP_DT_F32) return launch_stream_join<float>(a, ny, vec, rows, (cudaStream_t)stream);
    if (dtype == KIPP_DT_BF16) return launch_stream_join<bf16>(a, ny, vec, rows, (cudaStream_t)stream);
    return KIPP_ERR_DTYPE;
}

extern "C" int kipp_token_side_gate(void* g, long long ld_g, const float* z, long long ld_z, const void* table, long long ld_table,
                                    int off, int dtype, const int* ids, int tokens, int dim, int vocab, void* stream) {
    if (tokens <= 0) return 0;
    if (dim <= 0 || ld_g < dim || ld_z < dim || off < 0 || off + dim > ld_table || vocab <= 0) return KIPP_ERR_ARG;
    const dim3 grid((unsigned)((tokens * ld_g + 255) / 256));
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == KIPP_DT_F32)
        return kipp_launch(token_side_gate_kernel<float>, grid, dim3(256), 0, s, 1, (float*)g, ld_g, z, ld_z, (const float*)table,
                           ld_table, off, ids, tokens, dim, vocab);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(token_side_gate_kernel<bf16>, grid, dim3(256), 0, s, 1, (bf16*)g, ld_g, z, ld_z, (const bf16*)table,
                           ld_table, off, ids, tokens, dim, vocab);
    return KIPP_ERR_DTYPE;
}

// x *= scale over n float32 values (logits of a head with a scale).
__global__ void scale_f32_kernel(float* __restrict__ x, long long n, float scale) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] *= scale;
}

extern "C" int kipp_scale_f32(float* x, long long n, float scale, void* stream) {
    if (n <= 0) return 0;
    const long long blocks = (n + 255) / 256;
    if (blocks > 0x7fffffffLL) return KIPP_ERR_ARG;
    return kipp_launch(scale_f32_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, 1, x, n, scale);
}

// ---------------------------------------------------------------------------------------------
// Hyper-connections: the residual stream as S copies x_1 .. x_S, each [tokens, size] float32, `stride`
// floats apart.  One launch does, per token row, up to two things in float32:
//   update (y given)    x_t <- sum_s mix[s * S + t] x_s + mult * out[t] * y      for every t, from the old x_s
//   read (in_w given)   u = sum_s in_w[s] x_s;  h = u * rsqrt(mean(u^2) + eps) * norm_w, in the compute type
// so that the kernel between two sublayers writes the streams once and hands the next sublayer its
// input.  With S = 1 and mix = in = out = 1 this is the plain residual add and pre-norm.
namespace {
constexpr int MAX_STREAMS = 8;
struct HyperArgs {
    float* x; long long stride; int S;
    float* y; int clear_y;
    const float* mix; const float* out_w; float mult;
    const float* in_w; const void* norm_w; int norm_w_dtype; float eps;
    void* h;
    int size;
};

// VEC: values per thread and step (4 where the row's size and the pointers allow 16-byte accesses); MS: the
// most copies this instance holds (4 keeps a thread's values in few enough registers for blocks of 512)
template <typename T, int VEC, int MS>
__global__ void __launch_bounds__(MS <= 4 ? 512 : 256)
hyper_connection_kernel(const HyperArgs a) {
    extern __shared__ __align__(16) float u_row[];        // [size] when the read phase runs
    __shared__ float scratch[32];
    __shared__ float c_mix[MAX_STREAMS * MAX_STREAMS], c_out[MAX_STREAMS], c_in[MAX_STREAMS];
    pdl_launch_dependents();
    pdl_wait();
    const int S = a.S, size = a.size;
    if (threadIdx.x < S * S && a.y != nullptr) c_mix[threadIdx.x] = a.mix ? a.mix[threadIdx.x] : (threadIdx.x % (S + 1) == 0 ? 1.f : 0.f);
    if (threadIdx.x < S) {
        c_out[threadIdx.x] = a.y != nullptr ? a.mult * (a.out_w ? a.out_w[threadIdx.x] : 1.f) : 0.f;
        c_in[threadIdx.x] = a.in_w ? a.in_w[threadIdx.x] : 1.f;
    }
    __syncthreads();
    const bool read = a.h != nullptr;
    float* row = a.x + (size_t)blockIdx.x * size;
    float* yr = a.y ? a.y + (size_t)blockIdx.x * size : nullptr;
    float ss = 0.f;
    for (int i = VEC * threadIdx.x; i < size; i += VEC * blockDim.x) {
        float xs[MS][VEC];
#pragma unroll
        for (int s = 0; s < MS; ++s) {
            if (s >= S) continue;
            if (VEC == 4) *reinterpret_cast<float4*>(xs[s]) = *reinterpret_cast<const float4*>(row + (size_t)s * a.stride + i);
            else xs[s][0] = row[(size_t)s * a.stride + i];
        }
        if (yr != nullptr) {
            float y[VEC], nx[MS][VEC];
            if (VEC == 4) *reinterpret_cast<float4*>(y) = *reinterpret_cast<const float4*>(yr + i);
            else y[0] = yr[i];
            if (a.clear_y) {                            // the next sublayer adds its output into zeros
                if (VEC == 4) *reinterpret_cast<float4*>(yr + i) = make_float4(0.f, 0.f, 0.f, 0.f);
                else yr[i] = 0.f;
            }
#pragma unroll
            for (int t = 0; t < MS; ++t) {
                if (t >= S) continue;
#pragma unroll
                for (int v = 0; v < VEC; ++v) {
                    float acc = 0.f;
#pragma unroll
                    for (int s = 0; s < MS; ++s)
                        if (s < S) acc = fmaf(c_mix[s * S + t], xs[s][v], acc);
                    nx[t][v] = fmaf(c_out[t], y[v], acc);
                }
            }
#pragma unroll
            for (int t = 0; t < MS; ++t) {
                if (t >= S) continue;
#pragma unroll
                for (int v = 0; v < VEC; ++v) xs[t][v] = nx[t][v];
                if (VEC == 4) *reinterpret_cast<float4*>(row + (size_t)t * a.stride + i) = *reinterpret_cast<const float4*>(nx[t]);
                else row[(size_t)t * a.stride + i] = nx[t][0];
            }
        }
        if (read) {
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                float u = 0.f;
#pragma unroll
                for (int s = 0; s < MS; ++s)
                    if (s < S) u = fmaf(c_in[s], xs[s][v], u);
                u_row[i + v] = u;
                ss = fmaf(u, u, ss);
            }
        }
    }
    if (!read) return;
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)size + a.eps);
    T* h = static_cast<T*>(a.h) + (size_t)blockIdx.x * size;
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        const float w = a.norm_w_dtype == KIPP_DT_F32 ? static_cast<const float*>(a.norm_w)[i]
                                                      : to_f32(static_cast<const bf16*>(a.norm_w)[i]);
        h[i] = from_f32<T>(u_row[i] * inv * w);
    }
}

__global__ void sum_streams_kernel(float* __restrict__ out, const float* __restrict__ x, long long stride, int S,
                                   long long n) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    float acc = 0.f;
    for (int s = 0; s < S; ++s) acc += x[(size_t)s * stride + i];
    out[i] = acc;
}
}  // namespace

extern "C" int kipp_hyper_connection_max_streams() { return MAX_STREAMS; }

// y null: no update; h null: no read.  mix [S, S] indexed [from, to], out_w [S], in_w [S] float32 (null: identity / ones).
// clear_y: y is set to zero once it is read (the buffer the next sublayer adds its output into).
extern "C" int kipp_hyper_connection(float* x, long long stride, int streams, float* y, int clear_y, const float* mix,
                                     const float* out_w, float mult, const float* in_w, const void* norm_w,
                                     int norm_w_dtype, float eps, void* h, int h_dtype, int rows, int size, void* stream) {
    if (rows <= 0) return 0;
    if (size <= 0 || streams <= 0 || streams > MAX_STREAMS || x == nullptr) return KIPP_ERR_ARG;
    if (h != nullptr && (norm_w == nullptr || !(eps > 0.f) || (norm_w_dtype != KIPP_DT_F32 && norm_w_dtype != KIPP_DT_BF16)))
        return KIPP_ERR_ARG;
    if ((size_t)size * sizeof(float) > 160 * 1024) return KIPP_ERR_ARG;
    HyperArgs a;
    a.x = x; a.stride = stride; a.S = streams; a.y = y; a.clear_y = clear_y; a.mix = mix; a.out_w = out_w; a.mult = mult;
    a.in_w = in_w; a.norm_w = norm_w; a.norm_w_dtype = norm_w_dtype; a.eps = eps; a.h = h; a.size = size;
    const size_t smem = h != nullptr ? (size_t)size * sizeof(float) : 0;
    const bool vec = size % 4 == 0 && stride % 4 == 0 && (((uintptr_t)x | (uintptr_t)y) & 15) == 0;
    // a thread's steps wait for one another (loads behind stores to the same row): with few rows as few steps
    // as the block allows; with rows enough to fill the GPU several times over, small blocks (measured at
    // 2,048 rows of 4 x 2,048: 36 us with 128 threads, 55 us with 512)
    const int per = vec ? 4 : 1;
    const int wide = std::min(streams <= 4 ? 512 : 256, std::max(64, (size / per + 31) / 32 * 32));
    const dim3 grid((unsigned)rows), block((unsigned)(rows >= 1024 ? std::min(128, wide) : wide));
    auto go = [&](auto kernel) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        return kipp_launch(kernel, grid, block, smem, (cudaStream_t)stream, 1, a);
    };
    const bool f32 = h == nullptr || h_dtype == KIPP_DT_F32;
    if (!f32 && h_dtype != KIPP_DT_BF16) return KIPP_ERR_DTYPE;
    if (streams <= 4) {
        if (f32) return vec ? go(hyper_connection_kernel<float, 4, 4>) : go(hyper_connection_kernel<float, 1, 4>);
        return vec ? go(hyper_connection_kernel<bf16, 4, 4>) : go(hyper_connection_kernel<bf16, 1, 4>);
    }
    if (f32) return vec ? go(hyper_connection_kernel<float, 4, MAX_STREAMS>) : go(hyper_connection_kernel<float, 1, MAX_STREAMS>);
    if (h_dtype == KIPP_DT_BF16)
        return vec ? go(hyper_connection_kernel<bf16, 4, MAX_STREAMS>) : go(hyper_connection_kernel<bf16, 1, MAX_STREAMS>);
    return KIPP_ERR_DTYPE;
}

// out[i] = sum_s x[s * stride + i] over n float32 values.
extern "C" int kipp_sum_streams(float* out, const float* x, long long stride, int streams, long long n, void* stream) {
    if (n <= 0) return 0;
    if (streams <= 0) return KIPP_ERR_ARG;
    const long long blocks = (n + 255) / 256;
    if (blocks > 0x7fffffffLL) return KIPP_ERR_ARG;
    return kipp_launch(sum_streams_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, 1, out, x, stride,
                       streams, n);
}

// ---------------------------------------------------------------------------------------------
// A gated feed-forward's activation: g = min(gate + bg, limit), u = clamp(up + bu, -limit, limit),
// out = act(g) (u + up_add) with act(g) = g sigmoid(alpha g) (act -1), or gelu in its tanh form (act 2), in
// float32 from the projection's stored values.  gate of element i
// is proj[r, gate_off + i * step], up proj[r, up_off + i * step].  limit <= 0: no limits.  row_gate given:
// the whole row is also multiplied by sigmoid(row_gate[r]) (a gate per token on the part's output:
// applied here, before the linear down projection).
namespace {
template <typename T>
__global__ void glu_limited_kernel(T* __restrict__ out, long long ld_out, const T* __restrict__ proj, long long ld_proj,
                                   int rows, int n, int gate_off, int up_off, int step, const float* __restrict__ bias_gate,
                                   const float* __restrict__ bias_up, int bias_step, int act, float limit, float alpha,
                                   float up_add, const float* __restrict__ row_gate) {
    pdl_launch_dependents();
    pdl_wait();
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)rows * n) return;
    const long long r = idx / n;
    const int i = (int)(idx % n);
    const T* pr = proj + r * ld_proj;
    float g = to_f32(pr[gate_off + (long long)i * step]), u = to_f32(pr[up_off + (long long)i * step]);
    if (bias_gate != nullptr) g += bias_gate[(long long)i * bias_step];
    if (bias_up != nullptr) u += bias_up[(long long)i * bias_step];
    if (limit > 0.f) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
    }
    float v = g / (1.0f + expf(act == 2 ? gelu_tanh_exponent(g) : -alpha * g)) * (u + up_add);
    if (row_gate != nullptr) v *= 1.0f / (1.0f + expf(-row_gate[r]));
    out[r * ld_out + i] = from_f32<T>(v);
}

__global__ void add_row_bias_kernel(float* __restrict__ x, const float* __restrict__ bias, long long n, int size) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] += bias[i % size];
}

__global__ void softcap_f32_kernel(float* __restrict__ x, long long n, float cap) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] = cap * tanhf(x[i] / cap);
}
}  // namespace

extern "C" int kipp_glu_limited(void* out, long long ld_out, const void* proj, long long ld_proj, int dtype, int rows, int n,
                                int gate_off, int up_off, int step, const float* bias_gate, const float* bias_up,
                                int bias_step, int act, float limit, float alpha, float up_add, const float* row_gate,
                                void* stream) {
    if (rows <= 0 || n <= 0) return 0;
    if (step <= 0 || gate_off < 0 || up_off < 0 || (act != -1 && act != 2)) return KIPP_ERR_ARG;
    const long long total = (long long)rows * n, blocks = (total + 255) / 256;
    if (blocks > 0x7fffffffLL) return KIPP_ERR_ARG;
    if (dtype == KIPP_DT_F32)
        return kipp_launch(glu_limited_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, 1, (float*)out,
                           ld_out, (const float*)proj, ld_proj, rows, n, gate_off, up_off, step, bias_gate, bias_up, bias_step,
                           act, limit, alpha, up_add, row_gate);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(glu_limited_kernel<bf16>, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, 1, (bf16*)out,
                           ld_out, (const bf16*)proj, ld_proj, rows, n, gate_off, up_off, step, bias_gate, bias_up, bias_step,
                           act, limit, alpha, up_add, row_gate);
    return KIPP_ERR_DTYPE;
}

// out[r] = w . h[r, :] in float32 (w float32 [size]; h in `dtype`): a block per row, the order of the sum
// fixed by the size.
namespace {
template <typename T>
__global__ void __launch_bounds__(128)
row_dot_kernel(float* __restrict__ out, const T* __restrict__ h, long long ldh, const float* __restrict__ w, int rows, int size) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const T* row = h + (size_t)blockIdx.x * ldh;
    float acc = 0.f;
    for (int i = threadIdx.x; i < size; i += blockDim.x) acc = fmaf(w[i], to_f32(row[i]), acc);
    acc = block_sum(acc, scratch);
    if (threadIdx.x == 0) out[blockIdx.x] = acc;
}
}  // namespace
extern "C" int kipp_row_dot(float* out, const void* h, long long ldh, int dtype, const float* w, int rows, int size, void* stream) {
    if (rows <= 0) return 0;
    if (size <= 0 || w == nullptr) return KIPP_ERR_ARG;
    const dim3 grid((unsigned)rows);
    if (dtype == KIPP_DT_F32)
        return kipp_launch(row_dot_kernel<float>, grid, dim3(128), 0, (cudaStream_t)stream, 1, out, (const float*)h, ldh, w, rows, size);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(row_dot_kernel<bf16>, grid, dim3(128), 0, (cudaStream_t)stream, 1, out, (const bf16*)h, ldh, w, rows, size);
    return KIPP_ERR_DTYPE;
}

// x[r, :] += bias over rows of `size` float32 values.
extern "C" int kipp_add_row_bias(float* x, const float* bias, int rows, int size, void* stream) {
    if (rows <= 0 || size <= 0) return 0;
    const long long n = (long long)rows * size, blocks = (n + 255) / 256;
    if (blocks > 0x7fffffffLL || bias == nullptr) return KIPP_ERR_ARG;
    return kipp_launch(add_row_bias_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, 1, x, bias, n, size);
}

// x <- cap * tanh(x / cap) over n float32 values (logits with a soft cap).
extern "C" int kipp_softcap_f32(float* x, long long n, float cap, void* stream) {
    if (n <= 0) return 0;
    const long long blocks = (n + 255) / 256;
    if (blocks > 0x7fffffffLL || !(cap > 0.f)) return KIPP_ERR_ARG;
    return kipp_launch(softcap_f32_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, 1, x, n, cap);
}
