// Rows [q | k | v] -> the queries and, in the paged pool, the keys and values, for layers whose positions do not enter the
// scores through a rotation, with a norm over each q head and each k head:
//
//     x / sqrt(mean(x^2) + eps) [* w]          (w: one weight per column of a head, shared by the heads; optional)
//
// and, optionally, values mixed with another layer's values of the same token: v <- (1 - lambda) v + lambda v_other.
// Statistics, the norm and the mix are 32-bit, with one rounding to the storage type T. One block per token; a head's
// elements lie over L lanes (a power of two), ITEMS chunks of VEC elements a lane.
#include <math.h>

#include "common.cuh"

namespace {
enum : int { TK_K_HEAD_NORM = 15 };
constexpr int HN_THREADS = 256;

struct HeadNorm {
    const void* qkv;
    int64_t stride;
    const float *wq, *wk;
    float eps;
    const void* other;           // [T, >= Hkv Dv] rows `other_stride` apart, or null
    int64_t other_stride;
    float keep, take;            // 1 - lambda, lambda
    const int *positions, *tok_seq, *block_table;
    int bt_stride;
    void *q_out, *pool;
    int H, Hkv, D, Dv, P, Dp, L;
};

template <typename T, int VEC>
struct __align__(sizeof(T) * VEC) HnChunk {
    T v[VEC];
};
}  // namespace

template <typename T, int VEC, int ITEMS>
__global__ void __launch_bounds__(HN_THREADS)
qkv_head_norm_write_kernel(const HeadNorm a) {
    using Chunk = HnChunk<T, VEC>;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const T* row = (const T*)a.qkv + (size_t)t * a.stride;
    const bool write = a.pool != nullptr;
    const int pos = a.positions[t];
    const int page = write ? TK_PAGE(TK_K_HEAD_NORM, a.block_table[(size_t)a.tok_seq[t] * a.bt_stride + pos / a.P]) : 0;
    T* pool = (T*)a.pool;
    const int lane = threadIdx.x % a.L, per_pass = HN_THREADS / a.L, heads = a.H + (write ? a.Hkv : 0);
    for (int h0 = 0; h0 < heads; h0 += per_pass) {
        const int h = h0 + threadIdx.x / a.L;
        const bool mine = h < heads;
        const T* src = row + (size_t)h * a.D;                 // the k heads follow the q heads
        Chunk c[ITEMS];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < ITEMS; ++k) {
            const int i = (lane + k * a.L) * VEC;
            if (mine && i < a.D) {
                c[k] = *reinterpret_cast<const Chunk*>(src + i);
#pragma unroll
                for (int e = 0; e < VEC; ++e) ss = fmaf(to_f<T>(c[k].v[e]), to_f<T>(c[k].v[e]), ss);
            }
        }
        for (int o = a.L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (!mine) continue;
        const float rstd = 1.0f / sqrtf(ss / (float)a.D + a.eps);
        const bool is_q = h < a.H;
        const float* w = is_q ? a.wq : a.wk;
        T* dst = is_q ? (T*)a.q_out + ((size_t)t * a.H + h) * a.D
                      : pool + (((size_t)page * 2 * a.Hkv + (h - a.H)) * a.P + pos % a.P) * a.Dp;
#pragma unroll
        for (int k = 0; k < ITEMS; ++k) {
            const int i = (lane + k * a.L) * VEC;
            if (i >= a.D) continue;
#pragma unroll
            for (int e = 0; e < VEC; ++e)
                c[k].v[e] = from_f<T>(to_f<T>(c[k].v[e]) * rstd * (w != nullptr ? w[i + e] : 1.0f));
            *reinterpret_cast<Chunk*>(dst + i) = c[k];
        }
    }
    if (!write) return;
    const T* v = row + (size_t)(a.H + a.Hkv) * a.D;
    const T* other = a.other != nullptr ? (const T*)a.other + (size_t)t * a.other_stride : nullptr;
    for (int i = threadIdx.x * VEC; i < a.Hkv * a.Dv; i += HN_THREADS * VEC) {
        Chunk c = *reinterpret_cast<const Chunk*>(v + i);
        if (other != nullptr) {
            const Chunk f = *reinterpret_cast<const Chunk*>(other + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e)
                c.v[e] = from_f<T>(fmaf(a.take, to_f<T>(f.v[e]), a.keep * to_f<T>(c.v[e])));
        }
        *reinterpret_cast<Chunk*>(pool + (((size_t)(page * 2 + 1) * a.Hkv + i / a.Dv) * a.P + pos % a.P) * a.Dp + i % a.Dv) = c;
    }
}

// qkv: [T, >= (H + Hkv) D + Hkv Dv] rows `stride` apart; wq, wk: float32 [D] or null; other: [T, >= Hkv Dv] rows
// `other_stride` apart or null (the mix's other values, in the storage type); q_out: [T, H, D]; pool (null: queries only):
// [pages, 2, Hkv, P, Dp] with Dp >= max(D, Dv).
TK_API int tk_qkv_head_norm_write(const void* qkv, int64_t stride, const float* wq, const float* wk, float eps,
                                  const void* other, int64_t other_stride, float keep, float take, const int* positions,
                                  const int* tok_seq, const int* block_table, int bt_stride, void* q_out, void* pool,
                                  int tokens, int H, int Hkv, int D, int Dv, int P, int Dp, int dtype, cudaStream_t stream) {
    TK_CHECK_ARG(tokens >= 0 && H > 0 && Hkv > 0 && D > 0 && D <= 256 && Dv > 0, "qkv_head_norm_write: bad sizes");
    TK_CHECK_ARG(pool == nullptr || (block_table != nullptr && P > 0 && Dp >= D && Dp >= Dv),
                 "qkv_head_norm_write: cache rows of %d for keys of %d and values of %d", Dp, D, Dv);
    TK_CHECK_ARG(other == nullptr || pool != nullptr, "qkv_head_norm_write: values to mix without a cache to write");
    if (tokens == 0) return 0;
    HeadNorm a{qkv, stride, wq, wk, eps, other, other_stride, keep, take, positions, tok_seq, block_table, bt_stride,
               q_out, pool, H, Hkv, D, Dv, P, Dp, 1};
    const int es = dtype == TK_BF16 ? 2 : 4, vec = 16 / es;
    const bool wide = D % vec == 0 && Dv % vec == 0 && stride % vec == 0 && other_stride % vec == 0 &&
                      (pool == nullptr || Dp % vec == 0) &&
                      (((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)pool | (uintptr_t)other) & 15) == 0;
    const int chunks = ceil_div(D, wide ? vec : 1);
    while (a.L < 32 && a.L < chunks) a.L *= 2;
#define TK_HN(TT, VEC, ITEMS) \
    tk_launch(qkv_head_norm_write_kernel<TT, VEC, ITEMS>, dim3(tokens), dim3(HN_THREADS), 0, stream, a)
    if (dtype == TK_F32) {
        if (wide) TK_HN(float, 4, 2);
        else TK_HN(float, 1, 8);
    } else if (dtype == TK_BF16) {
        if (wide) TK_HN(__nv_bfloat16, 8, 1);
        else TK_HN(__nv_bfloat16, 1, 8);
    } else {
        TK_CHECK_ARG(false, "qkv_head_norm_write: unknown dtype %d", dtype);
    }
#undef TK_HN
    TK_CHECK_LAUNCH("qkv_head_norm_write");
    return 0;
}
