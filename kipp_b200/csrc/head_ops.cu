// Work on the heads of a projection that the plain per-head norm + rotation kernel does not
// cover, and products that run head by head.
//
// kipp_head_segments: the columns of a projection row are cut into SEGMENTS of heads; each
// segment says where its heads lie, what is done to them and where they go:
//   bias       a float32 vector added first (the projection's bias);
//   norm       division of the head by its root mean square (eps inside the root), times a
//              weight of the head's size; or (norm_all) division of ALL heads of the segment by the
//              root mean square of the whole run of heads x dim columns, times a weight of that size;
//              or (unit_norm) the division alone, without a weight;
//   rotation   of the dims [rot_off, rot_off + rot) of the head: pair (i, i + rot/2) turns by the
//              angle of the step's (cos, sin) table for the token; or (interleaved) pair (2i, 2i + 1);
//   target     a row of an activation buffer (queries), or the token's slot in the key or value
//              pages, where several heads of a segment may share one page row side by side
//              (two score maps of one key head; a latent and a rotated part that form one key).
// A warp takes one (token, head); all arithmetic is float32.  With this one kernel a mixer
// states its layout as data: keys made of parts, biases, rotation of a head's tail.
//
// kipp_head_matmul: out[t, h, :] = W_h a[t, h, :] for every head h, W_h [n, k] row-major, with
// float32 accumulation, optionally each element times the sigmoid of a gate of its own, all heads in one launch: in bfloat16 on the tensor cores (mma.sync); in
// 32-bit, or where rows do not start on 16-byte boundaries, few tokens by a kernel that reads the
// weights once and more tokens in tiles on the CUDA cores.  (Products with a latent: keys absorbed into queries, values expanded after the
// weighted sum.)
//
// kipp_latent_expand: the keys and values of every head out of cached latents, for prompt kernels that read them as
// keys and values of heads of their own: see the kernel.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int MAX_SEGMENTS = 4;

struct HeadSegment {
    int src_off, heads, dim, src_stride;     // columns of the projection row: head i at src_off + i * src_stride
    int rot_off, rot;                        // rotated dims of a head (rot 0: none)
    int target;                              // 0 activation rows, 1 key pages, 2 value pages
    int dst_off, dst_stride;                 // activation: head i at dst_off + i * dst_stride of the token's row
    int heads_per_row;                       // pages: this many heads side by side in one page row
    int norm_all;                            // 1: one mean square over all heads of the segment, norm_w [heads * dim]
    int interleaved;                         // 1: the rotation pairs dim 2i with dim 2i + 1
    int unit_norm;                           // 1: the norm's division without a weight (norm_w null)
    const float* bias;                       // [heads * dim] or null
    const float* norm_w;                     // [dim] ([heads * dim] with norm_all) or null
    const float* cos_sin;                    // [tokens, rot / 2, 2] or null
    void* dst;                               // activation buffer of the compute type (target 0)
    long long ld_dst;
};

struct SegmentArgs {
    HeadSegment seg[MAX_SEGMENTS];
    int n_segments, total_heads;
    const void* src; long long ld_src;
    void* k_pages; void* v_pages;
    int k_row, v_row, n_kv;                  // elements of a page row, rows (kv heads) per slot
    const int* positions; const int* entry_of_token; const int* block_table;
    int table_width, page_size, tokens, write_cache;
    float eps;
    int vec;                                 // every row of every segment starts on 16 bytes and holds whole 16-byte pieces
};

template <typename T>
__global__ void __launch_bounds__(128)
head_segments_kernel(const SegmentArgs a, int* __restrict__ status) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long wg = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    if (wg >= (long long)a.tokens * a.total_heads) return;
    const int t = (int)(wg / a.total_heads);
    int hh = (int)(wg % a.total_heads), si = 0;
    while (si + 1 < a.n_segments && hh >= a.seg[si].heads) { hh -= a.seg[si].heads; ++si; }
    const HeadSegment& g = a.seg[si];
    const int D = g.dim;
    const T* src = static_cast<const T*>(a.src) + (size_t)t * a.ld_src + g.src_off + (size_t)hh * g.src_stride;
    const float* bias = g.bias ? g.bias + (size_t)hh * D : nullptr;

    T* dst;
    bool into_cache = false;
    if (g.target == 0) {
        dst = static_cast<T*>(g.dst) + (size_t)t * g.ld_dst + g.dst_off + (size_t)hh * g.dst_stride;
    } else {
        if (!(a.write_cache & 1)) return;
        const int pos = a.positions[t], slot = pos / a.page_size;
        const int page = slot < a.table_width ? a.block_table[(size_t)a.entry_of_token[t] * a.table_width + slot] : -1;
        if (page < 0) {                       // unmapped page: refuse, never write
            if (lane == 0) atomicExch(status, 2);
            return;
        }
        const int row = hh / g.heads_per_row, within = hh % g.heads_per_row;
        const int row_len = g.target == 1 ? a.k_row : a.v_row;
        T* base = static_cast<T*>(g.target == 1 ? a.k_pages : a.v_pages);
        dst = base + (((size_t)page * a.n_kv + row) * a.page_size + pos % a.page_size) * row_len + g.dst_off +
              (size_t)within * D;
        into_cache = true;
    }

    float inv = 1.f;
    const float* norm_w = g.norm_w;
    const bool divided = g.norm_w != nullptr || g.unit_norm;
    if (divided && g.norm_all) {
        // every warp of the token sums the whole run of heads in the same order
        const T* all = static_cast<const T*>(a.src) + (size_t)t * a.ld_src + g.src_off;
        const int n = g.heads * D;
        constexpr int VEC = 16 / (int)sizeof(T);
        float ss = 0.f;
        if (g.bias == nullptr && n % VEC == 0 && ((uintptr_t)all & 15) == 0) {
            // 16 bytes per lane and step (the same lanes take the same elements for every head's warp)
            for (int i = VEC * lane; i < n; i += 32 * VEC) {
                const uint4 raw = *reinterpret_cast<const uint4*>(all + i);
                const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
                for (int j = 0; j < VEC; ++j) {
                    const float v = to_f32(e[j]);
                    ss = fmaf(v, v, ss);
                }
            }
        } else {
            for (int i = lane; i < n; i += 32) {
                const float v = to_f32(all[i]) + (g.bias ? g.bias[i] : 0.f);
                ss = fmaf(v, v, ss);
            }
        }
        inv = 1.0f / sqrtf(warp_sum(ss) / (float)n + a.eps);
        if (norm_w != nullptr) norm_w += (size_t)hh * D;
    } else if (divided) {
        float ss = 0.f;
        if (a.vec && bias == nullptr) {
            constexpr int VEC = 16 / (int)sizeof(T);
            for (int i = VEC * lane; i < D; i += 32 * VEC) {
                const uint4 raw = *reinterpret_cast<const uint4*>(src + i);
                const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
                for (int j = 0; j < VEC; ++j) {
                    const float v = to_f32(e[j]);
                    ss = fmaf(v, v, ss);
                }
            }
        } else {
            for (int i = lane; i < D; i += 32) {
                const float v = to_f32(src[i]) + (bias ? bias[i] : 0.f);
                ss = fmaf(v, v, ss);
            }
        }
        inv = 1.0f / sqrtf(warp_sum(ss) / (float)D + a.eps);
    }
    const int half = g.rot / 2;
    const float2* cs = (g.cos_sin != nullptr && g.rot > 0) ? reinterpret_cast<const float2*>(g.cos_sin) + (size_t)t * half
                                                           : nullptr;
    auto value = [&](int i) {
        float v = to_f32(src[i]) + (bias ? bias[i] : 0.f);
        if (divided) v = v * inv;
        if (norm_w != nullptr) v *= norm_w[i];
        return v;
    };
    if (a.vec && bias == nullptr && cs == nullptr) {
        // nothing is rotated: 16 bytes per lane and step
        constexpr int VEC = 16 / (int)sizeof(T);
        for (int i = VEC * lane; i < D; i += 32 * VEC) {
            const uint4 raw = *reinterpret_cast<const uint4*>(src + i);
            const T* e = reinterpret_cast<const T*>(&raw);
            uint4 packed;
            T* to = reinterpret_cast<T*>(&packed);
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                float v = to_f32(e[j]);
                if (divided) v = v * inv;
                if (norm_w != nullptr) v *= norm_w[i + j];
                if (into_cache) {
                    if (a.write_cache & 2) v = __bfloat162float(__float2bfloat16_rn(v));
                    v = cache_value(v);
                }
                to[j] = from_f32<T>(v);
            }
            *reinterpret_cast<uint4*>(dst + i) = packed;
        }
        return;
    }
    for (int i = lane; i < D; i += 32) {
        float v = value(i);
        const int r = i - g.rot_off;
        if (cs != nullptr && r >= 0 && r < g.rot) {
            // first of a pair: u cos - v sin; second: v cos + u sin (u the first, v the second)
            const bool low = g.interleaved ? (r & 1) == 0 : r < half;
            const float2 c = cs[g.interleaved ? r >> 1 : (low ? r : r - half)];
            const float other = value(g.interleaved ? (low ? i + 1 : i - 1) : (low ? i + half : i - half));
            v = low ? v * c.x - other * c.y : v * c.x + other * c.y;
        }
        if (into_cache) {
            if (a.write_cache & 2) v = __bfloat162float(__float2bfloat16_rn(v));
            v = cache_value(v);
        }
        dst[i] = from_f32<T>(v);
    }
}

// ---------------------------------------------------------------------------
// the factor of element n of head h of token m: sigmoid(gate[m, h * N + n]), or 1
template <typename T>
__device__ __forceinline__ float gate_factor(const T* __restrict__ gate, long long ld_gate, int m, int h, int N, int n) {
    return gate == nullptr ? 1.f : 1.0f / (1.0f + expf(-to_f32(gate[(size_t)m * ld_gate + (size_t)h * N + n])));
}

constexpr int BM = 64, BN = 64, BK = 16, TM = 4, TN = 4;

template <typename T>
__global__ void __launch_bounds__(256)
head_matmul_kernel(T* __restrict__ C, const T* __restrict__ A, const T* __restrict__ W, int M, int N, int K,
                   long long lda, long long a_head, long long w_head, long long ldc, long long c_head,
                   const T* __restrict__ gate, long long ld_gate) {
    __shared__ float As[BK][BM + 4];
    __shared__ float Ws[BK][BN + 4];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.z;
    A += (size_t)h * a_head;
    W += (size_t)h * w_head;
    C += (size_t)h * c_head;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
    float acc[TM][TN];
#pragma unroll
    for (int i = 0; i < TM; ++i)
#pragma unroll
        for (int j = 0; j < TN; ++j) acc[i][j] = 0.f;
    const int lrow = tid >> 2, lk = (tid & 3) * 4;
    for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int k = k0 + lk + i, am = m0 + lrow, wn = n0 + lrow;
            As[lk + i][lrow] = (am < M && k < K) ? to_f32(A[(size_t)am * lda + k]) : 0.f;
            Ws[lk + i][lrow] = (wn < N && k < K) ? to_f32(W[(size_t)wn * K + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; ++k) {
            float x[TM], y[TN];
#pragma unroll
            for (int i = 0; i < TM; ++i) x[i] = As[k][ty * TM + i];
#pragma unroll
            for (int j = 0; j < TN; ++j) y[j] = Ws[k][tx * TN + j];
#pragma unroll
            for (int i = 0; i < TM; ++i)
#pragma unroll
                for (int j = 0; j < TN; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < TM; ++i) {
        const int m = m0 + ty * TM + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < TN; ++j) {
            const int n = n0 + tx * TN + j;
            if (n < N) C[(size_t)m * ldc + n] = from_f32<T>(acc[i][j] * gate_factor(gate, ld_gate, m, h, N, n));
        }
    }
}

// Few tokens: the product is bound by reading W once.  A warp takes one output feature of one
// head for up to MT tokens; lanes stride over k (the same order for every token).
constexpr int MT = 8;
template <typename T>
__global__ void __launch_bounds__(256)
head_matvec_kernel(T* __restrict__ C, const T* __restrict__ A, const T* __restrict__ W, int M, int N, int K,
                   long long lda, long long a_head, long long w_head, long long ldc, long long c_head,
                   const T* __restrict__ gate, long long ld_gate) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const int n = blockIdx.x * 8 + (threadIdx.x >> 5), h = blockIdx.z, m0 = blockIdx.y * MT;
    if (n >= N) return;
    const T* w = W + (size_t)h * w_head + (size_t)n * K;
    const T* a = A + (size_t)h * a_head + (size_t)m0 * lda;
    const int rows = min(MT, M - m0);
    float acc[MT];
#pragma unroll
    for (int i = 0; i < MT; ++i) acc[i] = 0.f;
    for (int k = lane; k < K; k += 32) {
        const float wv = to_f32(w[k]);
#pragma unroll
        for (int i = 0; i < MT; ++i)
            if (i < rows) acc[i] = fmaf(to_f32(a[(size_t)i * lda + k]), wv, acc[i]);
    }
#pragma unroll
    for (int i = 0; i < MT; ++i) {
        const float s = warp_sum(acc[i]);
        if (i < rows && lane == 0) C[(size_t)h * c_head + (size_t)(m0 + i) * ldc + n] = from_f32<T>(s * gate_factor(gate, ld_gate, m0 + i, h, N, n));
    }
}

// In bfloat16: the same product on the tensor cores (mma.sync m16n8k16), all heads in one launch.  A block of 4 warps takes 64 tokens x 64 features of one head; K is walked in steps of 32
// through four stages of shared memory (16-byte asynchronous copies, zeros beyond M, N and K); a warp owns 16
// tokens x 64 features.  The sum over k runs in the same order for every token.
constexpr int HM = 64, HN = 64, HK = 32, HLD = HK + 8, H_STAGES = 4;
__device__ __forceinline__ void mma_bf16_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__global__ void __launch_bounds__(128)
head_matmul_mma_kernel(bf16* __restrict__ C, const bf16* __restrict__ A, const bf16* __restrict__ W, int M, int N, int K,
                       long long lda, long long a_head, long long w_head, long long ldc, long long c_head,
                       const bf16* __restrict__ gate, long long ld_gate) {
    __shared__ __align__(16) bf16 A_stage[H_STAGES][HM * HLD];
    __shared__ __align__(16) bf16 W_stage[H_STAGES][HN * HLD];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.z;
    A += (size_t)h * a_head;
    W += (size_t)h * w_head;
    C += (size_t)h * c_head;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
    const int m0 = blockIdx.y * HM, n0 = blockIdx.x * HN;
    float acc[HN / 8][4];
#pragma unroll
    for (int j = 0; j < HN / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    // 64 rows x 4 chunks of 8 elements for each operand: 256 chunks, two per thread and operand
    auto fetch = [&](int k0, int stage) {
#pragma unroll
        for (int i = tid; i < HM * (HK / 8); i += 128) {
            const int r = i >> 2, c = (i & 3) * 8;
            const bool ka = k0 + c < K;
            const bool oa = ka && m0 + r < M, ow = ka && n0 + r < N;
            cp_async16(smem_address(A_stage[stage] + r * HLD + c), oa ? A + (size_t)(m0 + r) * lda + k0 + c : A, oa ? 16 : 0);
            cp_async16(smem_address(W_stage[stage] + r * HLD + c), ow ? W + (size_t)(n0 + r) * K + k0 + c : W, ow ? 16 : 0);
        }
    };
#pragma unroll
    for (int s = 0; s < H_STAGES - 1; ++s) {
        if (s * HK < K) fetch(s * HK, s);
        cp_async_commit();
    }
    for (int k0 = 0, s = 0; k0 < K; k0 += HK, s = (s + 1) % H_STAGES) {
        cp_async_wait<H_STAGES - 2>();
        __syncthreads();                                            // this step's tiles are there, those of the step before are read
        if (k0 + (H_STAGES - 1) * HK < K) fetch(k0 + (H_STAGES - 1) * HK, (s + H_STAGES - 1) % H_STAGES);
        cp_async_commit();
        const bf16 *As = A_stage[s], *Ws = W_stage[s];
#pragma unroll
        for (int ks = 0; ks < HK; ks += 16) {
            const bf16* ar = As + (warp * 16 + gid) * HLD + ks + tig * 2;
            uint32_t a[4];
            a[0] = *reinterpret_cast<const uint32_t*>(ar);
            a[1] = *reinterpret_cast<const uint32_t*>(ar + 8 * HLD);
            a[2] = *reinterpret_cast<const uint32_t*>(ar + 8);
            a[3] = *reinterpret_cast<const uint32_t*>(ar + 8 * HLD + 8);
#pragma unroll
            for (int j = 0; j < HN / 8; ++j) {
                const bf16* wr = Ws + (j * 8 + gid) * HLD + ks + tig * 2;
                mma_bf16_16816(acc[j], a, *reinterpret_cast<const uint32_t*>(wr), *reinterpret_cast<const uint32_t*>(wr + 8));
            }
        }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int m = m0 + warp * 16 + gid + 8 * half;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < HN / 8; ++j) {
            const int n = n0 + j * 8 + tig * 2;
            if (n + 1 < N) {
                *reinterpret_cast<__nv_bfloat162*>(C + (size_t)m * ldc + n) =
                    __floats2bfloat162_rn(acc[j][2 * half] * gate_factor(gate, ld_gate, m, h, N, n),
                                          acc[j][2 * half + 1] * gate_factor(gate, ld_gate, m, h, N, n + 1));
            } else if (n < N) {
                C[(size_t)m * ldc + n] = __float2bfloat16_rn(acc[j][2 * half] * gate_factor(gate, ld_gate, m, h, N, n));
            }
        }
    }
}

// The keys and values of every head from the latents a step's entries have cached (bfloat16).  A cached row holds a
// token's latent c [rank] and a key part [rot] all heads share; head h's key is [W_uk,h c | shared part], its value
// W_uv,h c.  They go to a pool of their own in pages of 64 tokens, keys [page][head][64][dim + rot] and values
// [page][head][64][v_dim], where token t of entry e lies in page e * pages_per_entry + t / 64 (that table is written too);
// rows of a page beyond the entry's last token are zeros.  A block of 8 warps (2 x 4) takes 128 tokens x 128
// features on mma.sync, K in steps of 32 through three stages of asynchronous copies; the tile leaves through shared
// memory in 16-byte pieces.  One more block per tile copies the shared key part into every head's keys.
constexpr int EM = 128, EN = 128, EK = 32, ELD = EK + 8, E_STAGES = 3, E_THREADS = 256, E_PAGE = 64;
constexpr size_t E_SMEM = (size_t)E_STAGES * (EM + EN) * ELD * 2;
static_assert(E_SMEM >= (size_t)EM * (EN + 8) * 2, "the result tile fits where the stages were");
struct ExpandArgs {
    const bf16* pages;                       // [page][page_size][row] latents
    const int* block_table; int table_width, page_size, row;
    const int* q_start; const int* context_len;
    const bf16* w_k; const bf16* w_v;        // [heads * dim, rank], [heads * v_dim, rank]
    int rank, dim, rot, v_dim, heads;
    bf16* k_out; bf16* v_out; int* table_out;
    int pages_per_entry, k_tiles, v_tiles;
    int* status;
};
__device__ __forceinline__ void ldmatrix4(uint32_t* r, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__global__ void __launch_bounds__(E_THREADS)
latent_expand_kernel(const ExpandArgs a) {
    extern __shared__ __align__(16) bf16 tile_mem[];
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.z, t0 = blockIdx.y * EM, tid = threadIdx.x;
    const int len = a.context_len[e] + a.q_start[e + 1] - a.q_start[e];
    const int rows_end = (len + E_PAGE - 1) / E_PAGE * E_PAGE;          // rows to write: whole pages
    const int ft = blockIdx.x;
    if (ft == a.k_tiles + a.v_tiles && blockIdx.y == 0)
        for (int j = tid; j < a.pages_per_entry; j += E_THREADS) a.table_out[(size_t)e * a.pages_per_entry + j] = e * a.pages_per_entry + j;
    if (t0 >= rows_end) return;
    const int* table = a.block_table + (size_t)e * a.table_width;
    const int k_row = a.dim + a.rot;
    // the cached row of token t, or null where the entry has no such token
    auto cached = [&](int t) -> const bf16* {
        if (t >= len) return nullptr;
        const int slot = t / a.page_size, page = slot < a.table_width ? table[slot] : -1;
        if (page < 0) {
            atomicExch(a.status, 3);                                    // a needed key is not mapped
            return nullptr;
        }
        return a.pages + ((size_t)page * a.page_size + t % a.page_size) * a.row;
    };
    auto out_row = [&](bf16* base, int t, int h, int width) {
        return base + ((((size_t)e * a.pages_per_entry + t / E_PAGE) * a.heads + h) * E_PAGE + t % E_PAGE) * width;
    };
    if (ft == a.k_tiles + a.v_tiles) {                                  // the shared key part
        const int chunks = a.rot / 8;
        for (int i = tid; i < EM * chunks; i += E_THREADS) {
            const int t = t0 + i / chunks, c = i % chunks;
            if (t >= rows_end) break;
            const bf16* src = cached(t);
            const uint4 v = src != nullptr ? *reinterpret_cast<const uint4*>(src + a.rank + c * 8) : make_uint4(0u, 0u, 0u, 0u);
            for (int h = 0; h < a.heads; ++h) *reinterpret_cast<uint4*>(out_row(a.k_out, t, h, k_row) + a.dim + c * 8) = v;
        }
        return;
    }
    const bool keys = ft < a.k_tiles;
    const int per_head = keys ? a.dim : a.v_dim, features = a.heads * per_head, n0 = (keys ? ft : ft - a.k_tiles) * EN;
    const bf16* w = keys ? a.w_k : a.w_v;
    // 128 rows x 4 chunks of 8 elements per operand and stage: two of each per thread, rows lr and lr + 64
    const int lr = tid >> 2, lc = (tid & 3) * 8;
    const bf16* a_src[2];
    const bf16* w_src[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        a_src[i] = cached(t0 + lr + 64 * i);
        w_src[i] = n0 + lr + 64 * i < features ? w + (size_t)(n0 + lr + 64 * i) * a.rank : nullptr;
    }
    auto fetch = [&](int k0, int stage) {
        bf16* as = tile_mem + (size_t)stage * (EM + EN) * ELD;
        bf16* ws = as + EM * ELD;
        const bool in = k0 + lc < a.rank;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const bool oa = in && a_src[i] != nullptr, ow = in && w_src[i] != nullptr;
            cp_async16(smem_address(as + (lr + 64 * i) * ELD + lc), oa ? a_src[i] + k0 + lc : a.pages, oa ? 16 : 0);
            cp_async16(smem_address(ws + (lr + 64 * i) * ELD + lc), ow ? w_src[i] + k0 + lc : w, ow ? 16 : 0);
        }
    };
    const int lane = tid & 31, warp = tid >> 5, wm = (warp >> 2) * 64, wn = (warp & 3) * 32, gid = lane >> 2, tig = lane & 3;
    float acc[4][4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
    const int steps = (a.rank + EK - 1) / EK;
#pragma unroll
    for (int s = 0; s < E_STAGES - 1; ++s) {
        if (s < steps) fetch(s * EK, s);
        cp_async_commit();
    }
    for (int s = 0; s < steps; ++s) {
        cp_async_wait<E_STAGES - 2>();
        __syncthreads();
        if (s + E_STAGES - 1 < steps) fetch((s + E_STAGES - 1) * EK, (s + E_STAGES - 1) % E_STAGES);
        cp_async_commit();
        const bf16* as = tile_mem + (size_t)(s % E_STAGES) * (EM + EN) * ELD;
        const bf16* ws = as + EM * ELD;
#pragma unroll
        for (int ks = 0; ks < EK; ks += 16) {
            uint32_t af[4][4], bf[2][4];
#pragma unroll
            for (int i = 0; i < 4; ++i) ldmatrix4(af[i], smem_address(as + (wm + i * 16 + (lane & 15)) * ELD + ks + (lane >> 4) * 8));
            // two groups of 8 features per load: rows (lane & 7) + 8 (lane >> 4), k half by bit 3 of the lane
#pragma unroll
            for (int j = 0; j < 2; ++j)
                ldmatrix4(bf[j], smem_address(ws + (wn + j * 16 + (lane & 7) + (lane >> 4) * 8) * ELD + ks + ((lane >> 3) & 1) * 8));
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) mma_bf16_16816(acc[i][j], af[i], bf[j >> 1][2 * (j & 1)], bf[j >> 1][2 * (j & 1) + 1]);
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    constexpr int CLD = EN + 8;
    bf16* ct = tile_mem;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half)
                *reinterpret_cast<__nv_bfloat162*>(ct + (wm + i * 16 + gid + 8 * half) * CLD + wn + j * 8 + tig * 2) =
                    __floats2bfloat162_rn(acc[i][j][2 * half], acc[i][j][2 * half + 1]);
    __syncthreads();
    for (int i = tid; i < EM * (EN / 8); i += E_THREADS) {
        const int r = i / (EN / 8), n = n0 + i % (EN / 8) * 8, t = t0 + r;
        if (t >= rows_end || n >= features) continue;                   // (heads are multiples of 8: a piece lies in one head)
        bf16* dst = keys ? out_row(a.k_out, t, n / per_head, k_row) : out_row(a.v_out, t, n / per_head, a.v_dim);
        *reinterpret_cast<uint4*>(dst + n % per_head) = *reinterpret_cast<const uint4*>(ct + r * CLD + i % (EN / 8) * 8);
    }
}

// out[h][n][k] = in[h][k][n]: the matrices of every head transposed (at bind time).
template <typename T>
__global__ void transpose_heads_kernel(T* __restrict__ out, const T* __restrict__ in, int rows, int cols) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * cols) return;
    const size_t base = (size_t)blockIdx.y * rows * cols;
    const int r = (int)(i / cols), c = (int)(i % cols);
    out[base + (size_t)c * rows + r] = in[base + i];
}

template <typename T>
int launch_head_matmul(void* C, const void* A, const void* W, int M, int N, int K, int heads, long long lda,
                       long long a_head, long long w_head, long long ldc, long long c_head, const void* gate, long long ld_gate,
                       cudaStream_t s) {
    // the tensor-core kernel: bfloat16 at any number of tokens (a decoded token and a prompt's token
    // then sum in the same order), rows of both operands on 16-byte boundaries, results on 4-byte ones
    if (sizeof(T) == 2 && K % 8 == 0 && lda % 8 == 0 && a_head % 8 == 0 && w_head % 8 == 0 && ldc % 2 == 0 &&
        c_head % 2 == 0 && (((uintptr_t)A | (uintptr_t)W) & 15) == 0 && ((uintptr_t)C & 3) == 0) {
        const dim3 grid((unsigned)((N + HN - 1) / HN), (unsigned)((M + HM - 1) / HM), (unsigned)heads);
        if (grid.y > 65535) return KIPP_ERR_ARG;
        return kipp_launch(head_matmul_mma_kernel, grid, dim3(128), 0, s, 1, (bf16*)C, (const bf16*)A, (const bf16*)W, M, N, K,
                           lda, a_head, w_head, ldc, c_head, (const bf16*)gate, ld_gate);
    }
    if (M <= 2 * MT) {
        const dim3 grid((unsigned)((N + 7) / 8), (unsigned)((M + MT - 1) / MT), (unsigned)heads);
        return kipp_launch(head_matvec_kernel<T>, grid, dim3(256), 0, s, 1, (T*)C, (const T*)A, (const T*)W, M, N, K, lda,
                           a_head, w_head, ldc, c_head, (const T*)gate, ld_gate);
    }
    const dim3 grid((unsigned)((N + BN - 1) / BN), (unsigned)((M + BM - 1) / BM), (unsigned)heads);
    if (grid.y > 65535) return KIPP_ERR_ARG;
    return kipp_launch(head_matmul_kernel<T>, grid, dim3(256), 0, s, 1, (T*)C, (const T*)A, (const T*)W, M, N, K, lda,
                       a_head, w_head, ldc, c_head, (const T*)gate, ld_gate);
}
}  // namespace

// `segments` points at n_segments HeadSegment records (host memory; the layout is the host
// core's HeadSegment, kernels.hpp).  write_cache: bit 0 write keys and values, bit 1 round them to
// bfloat16 first (32-bit cache).
extern "C" int kipp_head_segments(const void* src, long long ld_src, int dtype, const void* segments, int n_segments,
                                  void* k_pages, void* v_pages, int k_row, int v_row, int n_kv, const int* positions,
                                  const int* entry_of_token, const int* block_table, int table_width, int page_size,
                                  int tokens, int write_cache, float eps, int* status, void* stream) {
    if (tokens <= 0 || n_segments <= 0) return 0;
    if (n_segments > MAX_SEGMENTS || segments == nullptr || page_size <= 0) return KIPP_ERR_ARG;
    SegmentArgs a = {};
    const HeadSegment* seg = static_cast<const HeadSegment*>(segments);
    for (int i = 0; i < n_segments; ++i) {
        const HeadSegment& g = seg[i];
        if (g.heads <= 0 || g.dim <= 0 || g.rot < 0 || (g.rot & 1) || g.rot_off < 0 || g.rot_off + g.rot > g.dim ||
            g.target < 0 || g.target > 2 || (g.target == 0 && g.dst == nullptr) || (g.target != 0 && g.heads_per_row <= 0) ||
            (g.rot > 0 && g.cos_sin == nullptr) || (g.norm_all && g.src_stride != g.dim))
            return KIPP_ERR_ARG;
        if (g.target == 1 && (k_pages == nullptr || g.dst_off + g.heads_per_row * g.dim > k_row)) return KIPP_ERR_ARG;
        if (g.target == 2 && (v_pages == nullptr || g.dst_off + g.heads_per_row * g.dim > v_row)) return KIPP_ERR_ARG;
        if (g.target != 0 && (g.heads + g.heads_per_row - 1) / g.heads_per_row > n_kv) return KIPP_ERR_ARG;
        a.seg[i] = g;
        a.total_heads += g.heads;
    }
    a.n_segments = n_segments;
    // whether every head starts on 16 bytes on both sides and holds whole 16-byte pieces
    const int piece = dtype == KIPP_DT_F32 ? 4 : 8;
    uintptr_t bases = (uintptr_t)src | (uintptr_t)k_pages | (uintptr_t)v_pages;
    long long lengths = ld_src | (long long)(k_pages ? k_row : 0) | (v_pages ? v_row : 0);
    for (int i = 0; i < n_segments; ++i) {
        const HeadSegment& g = a.seg[i];
        bases |= (uintptr_t)g.dst;
        lengths |= (long long)g.src_off | g.src_stride | g.dim | g.dst_off | (g.target == 0 ? g.dst_stride | g.ld_dst : 0);
    }
    a.vec = (bases & 15) == 0 && lengths % piece == 0;
    a.src = src; a.ld_src = ld_src; a.k_pages = k_pages; a.v_pages = v_pages;
    a.k_row = k_row; a.v_row = v_row; a.n_kv = n_kv;
    a.positions = positions; a.entry_of_token = entry_of_token; a.block_table = block_table;
    a.table_width = table_width; a.page_size = page_size; a.tokens = tokens; a.write_cache = write_cache; a.eps = eps;
    const long long warps = (long long)tokens * a.total_heads, blocks = (warps + 3) / 4;
    if (blocks > 0x7fffffffLL) return KIPP_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == KIPP_DT_F32)
        return kipp_launch(head_segments_kernel<float>, dim3((unsigned)blocks), dim3(128), 0, s, 1, a, status);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(head_segments_kernel<bf16>, dim3((unsigned)blocks), dim3(128), 0, s, 1, a, status);
    return KIPP_ERR_DTYPE;
}

// C[t, h, 0:N] = W_h A[t, h, 0:K]: row t of head h of A at A + h * a_head + t * lda, W_h at
// W + h * w_head as [N, K], the result at C + h * c_head + t * ldc; all in `dtype`.  gate (or null), of the same
// type: the element is also multiplied by sigmoid(gate[t * ld_gate + h * N + n]).
extern "C" int kipp_head_matmul_gated(void* C, const void* A, const void* W, int dtype, int M, int N, int K, int heads,
                                      long long lda, long long a_head, long long w_head, long long ldc, long long c_head,
                                      const void* gate, long long ld_gate, void* stream) {
    if (M <= 0 || N <= 0 || heads <= 0) return 0;
    if (K <= 0 || heads > 65535 || (gate != nullptr && ld_gate < (long long)heads * N)) return KIPP_ERR_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == KIPP_DT_F32)
        return launch_head_matmul<float>(C, A, W, M, N, K, heads, lda, a_head, w_head, ldc, c_head, gate, ld_gate, s);
    if (dtype == KIPP_DT_BF16)
        return launch_head_matmul<bf16>(C, A, W, M, N, K, heads, lda, a_head, w_head, ldc, c_head, gate, ld_gate, s);
    return KIPP_ERR_DTYPE;
}
extern "C" int kipp_head_matmul(void* C, const void* A, const void* W, int dtype, int M, int N, int K, int heads,
                                long long lda, long long a_head, long long w_head, long long ldc, long long c_head,
                                void* stream) {
    return kipp_head_matmul_gated(C, A, W, dtype, M, N, K, heads, lda, a_head, w_head, ldc, c_head, nullptr, 0, stream);
}

// Whether kipp_latent_expand takes these sizes: every row and head goes by 16-byte pieces.
extern "C" int kipp_latent_expand_ok(int rank, int dim, int rot, int v_dim, int heads) {
    return rank > 0 && dim > 0 && rot >= 0 && v_dim > 0 && heads > 0 && rank % 8 == 0 && dim % 8 == 0 && rot % 8 == 0 && v_dim % 8 == 0;
}
extern "C" int kipp_latent_expand_page() { return E_PAGE; }

// See latent_expand_kernel.  pages_per_entry pages of kipp_latent_expand_page() tokens hold the longest context the
// block table can name.
extern "C" int kipp_latent_expand(const void* pages, const int* block_table, int table_width, int page_size, int row,
                                  const int* q_start, const int* context_len, int entries, const void* w_k, const void* w_v,
                                  int rank, int dim, int rot, int v_dim, int heads, void* k_out, void* v_out, int* table_out,
                                  int pages_per_entry, int* status, void* stream) {
    if (entries <= 0) return 0;
    if (!kipp_latent_expand_ok(rank, dim, rot, v_dim, heads) || row != rank + rot || page_size <= 0 || table_width <= 0 ||
        (long long)pages_per_entry * E_PAGE < (long long)table_width * page_size || entries > 65535)
        return KIPP_ERR_ARG;
    if ((((uintptr_t)pages | (uintptr_t)w_k | (uintptr_t)w_v | (uintptr_t)k_out | (uintptr_t)v_out) & 15) != 0) return -3;
    ExpandArgs a = {};
    a.pages = (const bf16*)pages; a.block_table = block_table; a.table_width = table_width; a.page_size = page_size; a.row = row;
    a.q_start = q_start; a.context_len = context_len; a.w_k = (const bf16*)w_k; a.w_v = (const bf16*)w_v;
    a.rank = rank; a.dim = dim; a.rot = rot; a.v_dim = v_dim; a.heads = heads;
    a.k_out = (bf16*)k_out; a.v_out = (bf16*)v_out; a.table_out = table_out; a.pages_per_entry = pages_per_entry; a.status = status;
    a.k_tiles = (heads * dim + EN - 1) / EN;
    a.v_tiles = (heads * v_dim + EN - 1) / EN;
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(latent_expand_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)E_SMEM);
        if (e != cudaSuccess) { cudaGetLastError(); return (int)e; }
        configured = true;
    }
    const int tiles = (pages_per_entry * E_PAGE + EM - 1) / EM;
    if (tiles > 65535) return KIPP_ERR_ARG;
    return kipp_launch(latent_expand_kernel, dim3((unsigned)(a.k_tiles + a.v_tiles + 1), (unsigned)tiles, (unsigned)entries),
                       dim3(E_THREADS), E_SMEM, (cudaStream_t)stream, 1, a);
}

// out[h] = in[h]^T for `heads` row-major matrices of [rows, cols] in `dtype`.
extern "C" int kipp_transpose_heads(void* out, const void* in, int dtype, int heads, int rows, int cols, void* stream) {
    if (heads <= 0 || rows <= 0 || cols <= 0) return 0;
    if (heads > 65535) return KIPP_ERR_ARG;
    const long long n = (long long)rows * cols;
    const dim3 grid((unsigned)((n + 255) / 256), (unsigned)heads);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == KIPP_DT_F32)
        return kipp_launch(transpose_heads_kernel<float>, grid, dim3(256), 0, s, 1, (float*)out, (const float*)in, rows, cols);
    if (dtype == KIPP_DT_BF16)
        return kipp_launch(transpose_heads_kernel<bf16>, grid, dim3(256), 0, s, 1, (bf16*)out, (const bf16*)in, rows, cols);
    return KIPP_ERR_DTYPE;
}
