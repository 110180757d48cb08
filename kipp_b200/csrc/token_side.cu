// The gate of a token side (what a layer's own embedding of a token adds to the residual stream) for steps of few
// tokens: g = gelu_tanh(W_gate x) * e in one launch, e the columns [off, off + dim) of the token's row of a table.  Larger
// steps make it of a rounded copy of the stream, a product and an element-wise kernel (token_side_gate, elementwise.cu).
//
// A block takes 8 rows of W_gate and 16 tokens; the width is dealt out to its 8 warps in groups of 32, whose sums meet
// in shared memory in order.  The products run on mma.sync m16n8k16 with the tokens as M; x is rounded to bfloat16 on
// the way into the registers, as the larger steps' copy rounds it.  A lane reads 16 bytes of a weight row (8
// neighbouring columns) and the same columns of its token's rows, so the k order inside a group of 32 is a permuted
// one, the same on both sides.  The first groups' weights are fetched before the kernel before this one has ended:
// nothing of a step writes weights.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int THREADS = 256, WARPS = THREADS / 32, TOKENS = 16, AHEAD = 8;

__device__ __forceinline__ void mma_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// eight neighbouring values of the stream as bfloat16 pairs
__device__ __forceinline__ uint4 rounded(const float* p) {
    const float4 u = *reinterpret_cast<const float4*>(p), v = *reinterpret_cast<const float4*>(p + 4);
    const __nv_bfloat162 b[4] = {__floats2bfloat162_rn(u.x, u.y), __floats2bfloat162_rn(u.z, u.w), __floats2bfloat162_rn(v.x, v.y),
                                 __floats2bfloat162_rn(v.z, v.w)};
    return *reinterpret_cast<const uint4*>(b);
}

__global__ void __launch_bounds__(THREADS)
token_side_few_kernel(bf16* __restrict__ g, long long ld_g, const float* __restrict__ x, const bf16* __restrict__ w_gate,
                      const bf16* __restrict__ table, long long ld_table, int off, const int* __restrict__ ids, int tokens, int width,
                      int dim, int vocab) {
    __shared__ float red[WARPS][TOKENS][8];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
    const int n0 = blockIdx.x * 8, t0 = blockIdx.y * TOKENS, nt = min(TOKENS, tokens - t0), groups = width / 32;
    const uint4 none = make_uint4(0u, 0u, 0u, 0u);
    const bf16* wr = w_gate + (size_t)min(n0 + gid, dim - 1) * width + tig * 8;      // (rows beyond the last are not stored)
    pdl_launch_dependents();
    uint4 w[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) w[i] = warp + WARPS * i < groups ? *reinterpret_cast<const uint4*>(wr + (warp + WARPS * i) * 32) : none;
    pdl_wait();
    const float* lo_row = x + (size_t)(t0 + min(gid, nt - 1)) * width + tig * 8;
    const float* hi_row = x + (size_t)(t0 + min(gid + 8, nt - 1)) * width + tig * 8;
    const bool has_hi = nt > 8;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    auto group = [&](int kc, const uint4& wv) {
        const uint4 lo = rounded(lo_row + kc * 32), hi = has_hi ? rounded(hi_row + kc * 32) : none;
        const uint32_t first[4] = {lo.x, hi.x, lo.y, hi.y}, second[4] = {lo.z, hi.z, lo.w, hi.w};
        mma_16816(acc, first, wv.x, wv.y);
        mma_16816(acc, second, wv.z, wv.w);
    };
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
        if (warp + WARPS * i < groups) group(warp + WARPS * i, w[i]);
#pragma unroll 4
    for (int kc = warp + WARPS * AHEAD; kc < groups; kc += WARPS) group(kc, *reinterpret_cast<const uint4*>(wr + kc * 32));
    red[warp][gid][tig * 2] = acc[0];
    red[warp][gid][tig * 2 + 1] = acc[1];
    red[warp][gid + 8][tig * 2] = acc[2];
    red[warp][gid + 8][tig * 2 + 1] = acc[3];
    __syncthreads();
    const int t = tid >> 3, n = n0 + (tid & 7);
    if (t >= nt || n >= ld_g) return;
    float v = 0.f;
    if (n < dim) {
        float z = 0.f;
#pragma unroll
        for (int i = 0; i < WARPS; ++i) z += red[i][t][tid & 7];
        const int id = ids[t0 + t];                            // (the embedding stage reports ids outside the vocabulary)
        if (id >= 0 && id < vocab) v = kipp_activation(z, 2) * to_f32(table[(size_t)id * ld_table + off + n]);
    }
    g[(size_t)(t0 + t) * ld_g + n] = __float2bfloat16_rn(v);
}
}  // namespace

// Whether the kernel takes this width (bfloat16 weights only).
extern "C" int kipp_token_side_few_ok(int width) { return width > 0 && width % 32 == 0; }

// g bfloat16 [tokens, ld_g] with zeros from dim on; x float32 [tokens, width]; w_gate bfloat16 [dim, width].
extern "C" int kipp_token_side_few(void* g, long long ld_g, const float* x, const void* w_gate, const void* table, long long ld_table,
                                   int off, const int* ids, int tokens, int width, int dim, int vocab, void* stream) {
    if (tokens <= 0) return 0;
    if (!kipp_token_side_few_ok(width) || dim <= 0 || ld_g < dim || off < 0 || off + dim > ld_table || vocab <= 0) return KIPP_ERR_ARG;
    if ((((uintptr_t)x | (uintptr_t)w_gate) & 15) != 0) return -3;
    const dim3 grid((unsigned)((ld_g + 7) / 8), (unsigned)((tokens + TOKENS - 1) / TOKENS));
    return kipp_launch(token_side_few_kernel, grid, dim3(THREADS), 0, (cudaStream_t)stream, 1, (bf16*)g, ld_g, x, (const bf16*)w_gate,
                       (const bf16*)table, ld_table, off, ids, tokens, width, dim, vocab);
}
