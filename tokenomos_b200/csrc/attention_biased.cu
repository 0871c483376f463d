// Paged softmax attention with a soft cap on the scores and a learned bias by distance, on the tensor cores
// (bfloat16, warp-level mma.sync m16n8k16):
//
//     s_ij = cap tanh((q_i . k_j) scale / cap) + bias[h][min(i - j, L - 1)],   softmax over first_seen(i, window) <= j <= i
//
// (cap 0: none; a sliding window, chunks or every earlier position: see first_seen). With a sink the softmax's denominator
// has one more term, a key of score 0 without a value. Keys and values may differ in size (D and Dv up to 128,
// multiples of 8; the cache row Dp holds either); the tiles in shared memory are 64 or 128 wide, columns past D
// or Dv are zeros. Scores, bias, maxima and sums are 32-bit; a weight is rounded to bfloat16 where it meets the
// values. The CUDA-core form for any sizes and 32-bit storage is attn_generic's.
//   prompt portions: a CTA takes up to 64 rows (64 / G tokens of one sequence, G heads each), four warps of 16
//     rows, and walks the keys in tiles of 64 through a double-buffered cp.async pipeline.
//   single tokens: a token's G heads are the (padded) 16 rows of all four warps; warp w takes keys 16 w .. 16 w + 15
//     of every tile; `nsplit` CTAs share a token's keys and a second kernel merges their shares.
// The bias of a tile's distances (at most 63 + the tile's tokens of them) is staged beside its keys, per head.
// With the cap as tanh(z) = 1 - 2 / (1 + e^(2 z)), a score in base-2 logarithms and up to a constant of the row is
//     s2 = bias log2(e) - k2 / (1 + 2^(c1 dot)),    c1 = 2 scale log2(e) / cap,  k2 = 2 cap log2(e),
// which lies between -k2 and 0 around the bias (a sink, of score 0, is at -k2 / 2 there): where that range is narrow
// enough for 32-bit powers of two (BOUNDED, decided by the caller from cap and bias, or, without a cap, from the lengths
// of queries and keys) no running maximum is needed and shares simply add up.
//
// In front of it: the write of the step's keys and values with a norm over a token's whole query row and whole key
// row (not per head), for layers whose positions enter through the scores alone.
#include <math.h>

#include "paged_tiles.cuh"

namespace {
enum : int { TK_K_ATTN_BIASED = 14 };

struct BiasedOptions {
    float scale, cap;
    const float* bias;       // [H, L] times log2(e), or null
    int L, window, D, Dv, Dp, sink;
};



__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(dst), "l"(src));
}

// Copies of 64 rows of W columns (D of them real) out of pages with rows Dp apart, NT threads; the page numbers of
// a tile are looked up while the tile before it is in flight.
template <int W, int NT>
struct PitchLoader {
    static constexpr int CH = W / 8, STEP = NT / CH, PER = 64 / STEP;
    static_assert(STEP % 8 == 0, "a thread's rows share their swizzle");
    int r0, p_shift, P, Dp;
    uint32_t dst;
    bool real;
    size_t head_off, page_stride;
    int page[PER];

    __device__ __forceinline__ void init(int tid, int kvh, int Hkv, int page_size, int shift, int D, int pitch) {
        const int c = tid % CH;
        r0 = tid / CH;
        dst = tile_off<W>(r0, c);
        real = c * 8 < D;
        P = page_size, p_shift = shift, Dp = pitch;
        head_off = (size_t)kvh * P * Dp + (size_t)c * 8;
        page_stride = (size_t)2 * Hkv * P * Dp;
    }
    __device__ __forceinline__ int block_of(int j) const { return p_shift >= 0 ? j >> p_shift : j / P; }
    __device__ __forceinline__ void lookup(const int* bt_row, int j0, int j_first, int j_last) {
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int j = min(max(j0 + r0 + k * STEP, j_first), j_last);     // always a held position
            page[k] = TK_PAGE(TK_K_ATTN_BIASED, bt_row[block_of(j)]);
        }
    }
    // `delta`: 0 for keys, the distance to the values for values
    __device__ __forceinline__ void issue(uint32_t tile, const __nv_bfloat16* pool, size_t delta, int j0, int j_first,
                                          int j_last) const {
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int j = j0 + r0 + k * STEP;
            const bool valid = real && j >= j_first && j <= j_last;
            const __nv_bfloat16* src = pool;
            if (valid) src = pool + (size_t)page[k] * page_stride + head_off + delta + (size_t)(j - block_of(j) * P) * Dp;
            cp_async16(tile + dst + (uint32_t)(k * STEP * W * 2), src, valid);
        }
    }
};

// Rows of a warp: the two a lane works for (g and g + 8)
struct BiasedRows {
    int pos[2];              // positions, -1: padding
    int first[2];            // the first positions they see
    const float* bias[2];    // the staged bias at the tile's first key: bias[-key]
};

template <int DK, int DV, int NK, bool BOUNDED, bool MASK>
__device__ __forceinline__ void biased_block(const uint32_t (&qf)[DK / 16][4], uint32_t ktile, uint32_t vtile, int k0, int j0,
                                             const BiasedRows& rows, bool capped, float c1, float k2,
                                             float (&m)[2], float (&l)[2], float (&o)[DV / 8][4]) {
    const int lane = threadIdx.x & 31;
    const int t = lane & 3, mi = lane >> 3, r = lane & 7;
    float s[NK / 8][4];
#pragma unroll
    for (int n = 0; n < NK / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
#pragma unroll
    for (int np = 0; np < NK / 16; ++np) {
        const int key = k0 + np * 16 + r + 8 * (mi >> 1);
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
            uint32_t b[4];
            ldmatrix_x4(b, ktile + tile_off<DK>(key, ks * 2 + (mi & 1)));
            mma16816(s[2 * np], qf[ks], b[0], b[1]);
            mma16816(s[2 * np + 1], qf[ks], b[2], b[3]);
        }
    }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < NK / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int key = k0 + n * 8 + 2 * t + (e & 1);
            // (a padding row's position is -1)
            const bool visible = !MASK || (j0 + key <= rows.pos[e >> 1] && j0 + key >= rows.first[e >> 1]);
            const float b = rows.bias[e >> 1][-key];
            const float v = capped ? fmaf(-k2, rcp_approx(1.f + fast_exp2(s[n][e] * c1)), b) : fmaf(s[n][e], c1, b);
            s[n][e] = visible ? v : -INFINITY;
            if constexpr (!BOUNDED) mx[e >> 1] = fmaxf(mx[e >> 1], s[n][e]);
        }
    float msafe[2] = {0.f, 0.f};
    if constexpr (!BOUNDED) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
            const float m_new = fmaxf(m[h], mx[h]);
            msafe[h] = m_new == -INFINITY ? 0.f : m_new;
            const float alpha = fast_exp2(m[h] - msafe[h]);
            m[h] = m_new;
            l[h] *= alpha;
#pragma unroll
            for (int n = 0; n < DV / 8; ++n) {
                o[n][2 * h] *= alpha;
                o[n][2 * h + 1] *= alpha;
            }
        }
    }
    uint32_t pf[NK / 16][4];
#pragma unroll
    for (int n = 0; n < NK / 8; ++n) {
        float p[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            p[e] = fast_exp2(BOUNDED ? s[n][e] : s[n][e] - msafe[e >> 1]);
            l[e >> 1] += p[e];
        }
        // the C layout of two neighbouring 8-key tiles is the A layout of one 16-key step
        pf[n >> 1][(n & 1) * 2 + 0] = pack_bf16(p[0], p[1]);
        pf[n >> 1][(n & 1) * 2 + 1] = pack_bf16(p[2], p[3]);
    }
#pragma unroll
    for (int ks = 0; ks < NK / 16; ++ks) {
        const int key = k0 + ks * 16 + r + 8 * (mi & 1);
#pragma unroll
        for (int dp = 0; dp < DV / 16; ++dp) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, vtile + tile_off<DV>(key, dp * 2 + (mi >> 1)));
            mma16816(o[2 * dp], pf[ks], b[0], b[1]);
            mma16816(o[2 * dp + 1], pf[ks], b[2], b[3]);
        }
    }
}

// Query fragments of 16 rows from global memory: row r is (token tok0 + r / G, head h0 + r % G); rows at or past
// `rows` and columns at or past D read as zero.
template <int DK>
__device__ __forceinline__ void biased_load_q(uint32_t (&qf)[DK / 16][4], const __nv_bfloat16* q, int row0, int rows,
                                              int tok0, int G, int H, int h0, int D) {
    const int lane = threadIdx.x & 31;
    const int g = lane >> 2, t = lane & 3;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = row0 + g + 8 * half;
        const bool ok = r < rows;
        const __nv_bfloat16* src = ok ? q + ((size_t)(tok0 + r / G) * H + h0 + r % G) * D : q;
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
            uint32_t lo = 0u, hi = 0u;
            if (ok && ks * 16 < D) lo = *reinterpret_cast<const uint32_t*>(src + ks * 16 + 2 * t);
            if (ok && ks * 16 + 8 < D) hi = *reinterpret_cast<const uint32_t*>(src + ks * 16 + 8 + 2 * t);
            qf[ks][half] = lo;
            qf[ks][half + 2] = hi;
        }
    }
}

template <int DK, int DV, bool SINGLE, bool BOUNDED>
__global__ void __launch_bounds__(128, (DK + DV <= 128 ? 4 : 2))
attn_biased_mma_kernel(const __nv_bfloat16* q, const __nv_bfloat16* pool, __nv_bfloat16* out, float* part_o, float* part_ml,
                       const int* positions, const int* tok_seq, const int* block_table, int bt_stride,
                       const int* tile_tok0, const int* tile_ntok, const int* singles, int n_units, int H, int Hkv, int P,
                       int p_shift, const BiasedOptions opt, int nsplit, int span) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(128) unsigned char smem_raw[];
    constexpr int K_BYTES = 64 * DK * 2, V_BYTES = 64 * DV * 2, STAGE = K_BYTES + V_BYTES;
    const uint32_t smem = (uint32_t)__cvta_generic_to_shared(smem_raw);      // [stage][K 64 x DK | V 64 x DV]
    float* bias_s = reinterpret_cast<float*>(smem_raw + 2 * STAGE);          // [stage][G][span], base-2 logarithms
    const uint32_t bias_at = smem + 2 * STAGE;
    const int G = H / Hkv;
    const int kvh = blockIdx.x % Hkv;
    // prompt tiles in reverse: a tile late in its sequence reads the most keys and starts first
    const int unit = SINGLE ? blockIdx.x / Hkv : n_units - 1 - blockIdx.x / Hkv;
    int tok0, ntok;
    if (SINGLE) {
        tok0 = singles != nullptr ? singles[unit] : unit;
        ntok = 1;
        if (tok0 < 0) return;        // an unused entry of a fixed-length list (captured steps)
    } else {
        tok0 = tile_tok0[unit];
        ntok = tile_ntok[unit];
        if (ntok <= 0) return;       // an unused entry of a fixed-length tile list (captured steps)
    }
    const int rows = ntok * G;
    const int seq = tok_seq[tok0];
    const int* bt_row = block_table + (size_t)seq * bt_stride;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2;
    const int pos_first = positions[tok0];
    const int pos_last = pos_first + ntok - 1;       // consecutive positions within a tile
    const int lo = first_seen(pos_first, opt.window);
    const int j_begin = (lo / 64) * 64;
    const int row0 = SINGLE ? 0 : warp * 16;
    if (opt.bias == nullptr)
        for (int i = tid; i < 2 * G * span; i += 128) bias_s[i] = 0.f;

    uint32_t qf[DK / 16][4];
    biased_load_q<DK>(qf, q, row0, rows, tok0, G, H, kvh * G, opt.D);
    BiasedRows br;
    int bias_off[2];                                 // where a row's bias starts within a stage
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int r = row0 + g + 8 * e;
        const bool ok = r < rows;
        br.pos[e] = ok ? pos_first + r / G : -1;
        br.first[e] = first_seen(br.pos[e], opt.window);
        bias_off[e] = (ok ? (r % G) * span + r / G : 0) + 63;
    }
    const bool capped = opt.cap > 0.f;
    const float c1 = capped ? 2.f * LOG2E * opt.scale / opt.cap : LOG2E * opt.scale;
    const float k2 = 2.f * LOG2E * opt.cap;
    // the warp's own key range: nothing above its last row's position, nothing a window hides
    const int w_last_row = min(rows, row0 + 16) - 1;
    const int w_pos_max = w_last_row >= row0 ? pos_first + w_last_row / G : -1;
    const int w_pos_min = pos_first + row0 / G;
    const int w_first_min = first_seen(w_pos_min, opt.window), w_first_max = first_seen(w_pos_max, opt.window);

    float m[2] = {BOUNDED ? 0.f : -INFINITY, BOUNDED ? 0.f : -INFINITY}, l[2] = {0.f, 0.f};
    if (opt.sink && (!SINGLE || (warp == 0 && blockIdx.y == 0))) {        // the sink joins a row's sum once
        const float at = capped ? -0.5f * k2 : 0.f;
        if constexpr (!BOUNDED) m[0] = m[1] = at;
        if ((lane & 3) == 0) l[0] = l[1] = BOUNDED ? fast_exp2(at) : 1.f;
    }
    float o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] = 0.f;

    // this CTA's share of the key tiles
    const int n_all = (pos_last - j_begin) / 64 + 1;
    const int per = (n_all + nsplit - 1) / nsplit;
    const int it0 = blockIdx.y * per, it1 = min(n_all, it0 + per);

    const size_t v_delta = (size_t)Hkv * P * opt.Dp;
    PitchLoader<DK, 128> kl;
    PitchLoader<DV, 128> vl;
    kl.init(tid, kvh, Hkv, P, p_shift, opt.D, opt.Dp);
    vl.init(tid, kvh, Hkv, P, p_shift, opt.Dv, opt.Dp);
    auto lookup = [&](int it) {
        kl.lookup(bt_row, j_begin + it * 64, lo, pos_last);
        if constexpr (DK != DV) vl.lookup(bt_row, j_begin + it * 64, lo, pos_last);
    };
    auto issue = [&](int it) {
        const int b = (it - it0) & 1, j0 = j_begin + it * 64;
        const uint32_t base = smem + (uint32_t)b * STAGE;
        kl.issue(base, pool, 0, j0, lo, pos_last);
        if constexpr (DK == DV) {
#pragma unroll
            for (int k = 0; k < PitchLoader<DK, 128>::PER; ++k) vl.page[k] = kl.page[k];
        }
        vl.issue(base + K_BYTES, pool, v_delta, j0, lo, pos_last);
        // bias of the tile's distances: entry i is distance i + pos_first - (j0 + 63)
        if (opt.bias != nullptr) {
            const uint32_t bs = bias_at + (uint32_t)(b * G * span) * 4;
            const int d0 = pos_first - j0 - 63;
            for (int h = warp; h < G; h += 4) {
                const float* src = opt.bias + (size_t)(kvh * G + h) * opt.L;
                for (int i = lane; i < span; i += 32)
                    cp_async4(bs + (uint32_t)(h * span + i) * 4, src + min(max(i + d0, 0), opt.L - 1));
            }
        }
        cp_async_commit();
        if (it + 1 < it1) lookup(it + 1);
    };
    if (it0 < it1) {
        lookup(it0);
        issue(it0);
    }
    for (int it = it0; it < it1; ++it) {
        cp_async_wait<0>();
        __syncthreads();
        if (it + 1 < it1) issue(it + 1);
        const int j0 = j_begin + it * 64, b = (it - it0) & 1;
        const uint32_t base = smem + (uint32_t)b * STAGE;
        br.bias[0] = bias_s + (size_t)b * G * span + bias_off[0];
        br.bias[1] = bias_s + (size_t)b * G * span + bias_off[1];
        if (SINGLE) {
            const int k0 = warp * 16;
            if (w_pos_max >= j0 + k0 && j0 + k0 + 15 >= w_first_min)
                biased_block<DK, DV, 16, BOUNDED, true>(qf, base, base + K_BYTES, k0, j0, br, capped, c1, k2, m, l, o);
        } else if (w_pos_max >= j0 && j0 + 63 >= w_first_min) {
            // (every key of an inner tile is seen by every row of the warp, padding rows aside, which nothing reads)
            if (j0 + 63 > w_pos_min || j0 < w_first_max)
                biased_block<DK, DV, 64, BOUNDED, true>(qf, base, base + K_BYTES, 0, j0, br, capped, c1, k2, m, l, o);
            else
                biased_block<DK, DV, 64, BOUNDED, false>(qf, base, base + K_BYTES, 0, j0, br, capped, c1, k2, m, l, o);
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    }
    const int t = lane & 3;
    if (!SINGLE) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = row0 + g + 8 * half;
            if (r >= rows) continue;
            const float inv = l[half] > 0.f ? 1.0f / l[half] : 0.f;
            __nv_bfloat16* dst = out + ((size_t)(tok0 + r / G) * H + kvh * G + r % G) * opt.Dv;
#pragma unroll
            for (int n = 0; n < DV / 8; ++n)
                if (n * 8 < opt.Dv)
                    *reinterpret_cast<uint32_t*>(dst + n * 8 + 2 * t) = pack_bf16(o[n][half * 2] * inv, o[n][half * 2 + 1] * inv);
        }
        return;
    }
    // single tokens: the four warps' shares meet in shared memory
    __syncthreads();                                  // every warp is done with the staged tiles
    float* sums = reinterpret_cast<float*>(smem_raw); // [4][16][DV], then [4][16] sums and [4][16] maxima
    float* ls = sums + 4 * 16 * DV;
    float* ms = ls + 64;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = warp * 16 + g + 8 * half;
        float* dst = sums + (size_t)r * DV;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n)
            *reinterpret_cast<float2*>(dst + n * 8 + 2 * t) = make_float2(o[n][half * 2], o[n][half * 2 + 1]);
        if (t == 0) {
            ls[r] = l[half];
            ms[r] = m[half];
        }
    }
    __syncthreads();
    for (int i = tid; i < rows * opt.Dv; i += 128) {
        const int r = i / opt.Dv, c = i % opt.Dv;
        float mm = 0.f, w[4] = {1.f, 1.f, 1.f, 1.f};
        if constexpr (!BOUNDED) {
            mm = fmaxf(fmaxf(ms[r], ms[16 + r]), fmaxf(ms[32 + r], ms[48 + r]));
            const float safe = mm == -INFINITY ? 0.f : mm;
#pragma unroll
            for (int k = 0; k < 4; ++k) w[k] = fast_exp2(ms[16 * k + r] - safe);
        }
        float v = 0.f, lt = 0.f;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            v = fmaf(w[k], sums[(size_t)(16 * k + r) * DV + c], v);
            lt = fmaf(w[k], ls[16 * k + r], lt);
        }
        const int head = kvh * G + r;
        if (nsplit == 1) {
            out[((size_t)tok0 * H + head) * opt.Dv + c] = __float2bfloat16(lt > 0.f ? v / lt : 0.f);
        } else {
            const size_t row = ((size_t)blockIdx.y * n_units + unit) * H + head;
            part_o[row * opt.Dv + c] = v;
            if (c == 0) {
                part_ml[2 * row] = mm;
                part_ml[2 * row + 1] = lt;
            }
        }
    }
}

// out rows of the listed tokens from their `nsplit` shares: one warp per (token, head)
__global__ void __launch_bounds__(128)
attn_biased_merge_kernel(const float* part_o, const float* part_ml, __nv_bfloat16* out, const int* singles, int n_units, int H,
                         int Dv, int nsplit) {
    pdl_launch_dependents();
    pdl_wait();
    const int w = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (w >= n_units * H) return;
    const int unit = w / H, head = w % H;
    const int tok = singles != nullptr ? singles[unit] : unit;
    if (tok < 0) return;             // an unused entry of a fixed-length list (captured steps)
    float mm = -INFINITY;
    for (int s = 0; s < nsplit; ++s) {
        const size_t row = ((size_t)s * n_units + unit) * H + head;
        if (part_ml[2 * row + 1] > 0.f) mm = fmaxf(mm, part_ml[2 * row]);
    }
    const float safe = mm == -INFINITY ? 0.f : mm;
    float acc[4] = {0.f, 0.f, 0.f, 0.f}, lt = 0.f;
    for (int s = 0; s < nsplit; ++s) {
        const size_t row = ((size_t)s * n_units + unit) * H + head;
        const float l = part_ml[2 * row + 1];
        const float f = l > 0.f ? fast_exp2(part_ml[2 * row] - safe) : 0.f;
        lt = fmaf(f, l, lt);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int c = lane + 32 * k;
            if (c < Dv) acc[k] = fmaf(f, part_o[row * Dv + c], acc[k]);
        }
    }
    const float inv = lt > 0.f ? 1.f / lt : 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        const int c = lane + 32 * k;
        if (c < Dv) out[((size_t)tok * H + head) * Dv + c] = __float2bfloat16(acc[k] * inv);
    }
}

int biased_shift(int P) {
    int s = 0;
    while ((1 << s) < P) ++s;
    return (1 << s) == P ? s : -1;
}
}  // namespace

// Whether the tensor-core form takes the shape: bfloat16, key and value sizes multiples of 8 up to 128, the cache row
// a multiple of 8, at most 16 query heads per key/value head.
TK_API int tk_attn_biased_mma_supported(int H, int Hkv, int D, int Dv, int Dp) {
    return H > 0 && Hkv > 0 && H % Hkv == 0 && H / Hkv <= 16 && D > 0 && Dv > 0 && D % 8 == 0 && Dv % 8 == 0 && D <= 128 &&
           Dv <= 128 && Dp % 8 == 0 && Dp >= D && Dp >= Dv;
}

TK_API int tk_attn_biased_mma_tokens(int H, int Hkv) { return 64 / (H / Hkv); }

// Prompt portions: tiles of tk_attn_biased_mma_tokens tokens (first token and count per tile). Single tokens (`n_single`
// > 0): the rows `singles` lists (null: rows 0 .. n_single - 1), each shared `nsplit` ways over its keys; part_o float32
// [nsplit, n_single, H, Dv] and part_ml [nsplit, n_single, H, 2] when nsplit > 1. bias: float32 [H, L] times log2(e), or null; bounded:
// the scores' reach, in base-2 logarithms, stays well inside a float's exponents. window: see first_seen.
TK_API int tk_attn_biased_mma(const void* q, const void* kv_pool, void* out, const int* positions, const int* tok_seq,
                              const int* block_table, int bt_stride, const int* tile_tok0, const int* tile_ntok, int n_tiles,
                              const int* singles, int n_single, int nsplit, float* part_o, float* part_ml, int H, int Hkv,
                              int D, int Dv, int Dp, int P, int window, float scale, float cap, const float* bias, int L,
                              int bounded, int sink, cudaStream_t stream) {
    TK_CHECK_ARG(tk_attn_biased_mma_supported(H, Hkv, D, Dv, Dp),
                 "attention: %d / %d heads of %d and %d are not the tensor-core form's", H, Hkv, D, Dv);
    TK_CHECK_ARG(P > 0 && n_tiles >= 0 && n_single >= 0 && cap >= 0.f && nsplit >= 1, "attention: bad sizes");
    TK_CHECK_ARG(nsplit == 1 || (part_o != nullptr && part_ml != nullptr), "attention: shares need scratch memory");
    TK_CHECK_ARG(bias == nullptr || L > 0, "attention: a distance bias of %d columns", L);
    const BiasedOptions opt{scale, cap, bias, max(L, 1), window, D, Dv, Dp, sink};
    const int G = H / Hkv, shift = biased_shift(P);
    auto q16 = (const __nv_bfloat16*)q;
    auto pool = (const __nv_bfloat16*)kv_pool;
    auto o16 = (__nv_bfloat16*)out;
#define TK_AB(DKK, DVV, SINGLE, BND, units, ns)                                                                         \
    do {                                                                                                                \
        const int span = 63 + (SINGLE ? 1 : 64 / G);                                                                    \
        const size_t smem = 2 * 64 * (size_t)(DKK + DVV) * 2 + 2 * (size_t)G * span * 4;                                \
        static size_t raised = 0;                                                                                       \
        if (smem > raised) {                                                                                            \
            cudaFuncSetAttribute(attn_biased_mma_kernel<DKK, DVV, SINGLE, BND>,                                         \
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                               \
            raised = smem;                                                                                              \
        }                                                                                                               \
        tk_launch(attn_biased_mma_kernel<DKK, DVV, SINGLE, BND>, dim3((units) * Hkv, ns), dim3(128), smem, stream, q16, \
                  pool, o16, part_o, part_ml, positions, tok_seq, block_table, bt_stride, tile_tok0, tile_ntok, singles, \
                  units, H, Hkv, P, shift, opt, ns, span);                                                              \
    } while (0)
#define TK_AB_D(SINGLE, BND, units, ns)                                         \
    do {                                                                        \
        if (D <= 64 && Dv <= 64) TK_AB(64, 64, SINGLE, BND, units, ns);         \
        else if (D <= 64) TK_AB(64, 128, SINGLE, BND, units, ns);               \
        else if (Dv <= 64) TK_AB(128, 64, SINGLE, BND, units, ns);              \
        else TK_AB(128, 128, SINGLE, BND, units, ns);                           \
    } while (0)
    if (n_tiles > 0) {
        if (bounded) TK_AB_D(false, true, n_tiles, 1);
        else TK_AB_D(false, false, n_tiles, 1);
        TK_CHECK_LAUNCH("attn_biased_mma");
    }
    if (n_single > 0) {
        if (bounded) TK_AB_D(true, true, n_single, nsplit);
        else TK_AB_D(true, false, n_single, nsplit);
        TK_CHECK_LAUNCH("attn_biased_mma");
        if (nsplit > 1) {
            tk_launch(attn_biased_merge_kernel, dim3((n_single * H + 3) / 4), dim3(128), 0, stream, (const float*)part_o,
                      (const float*)part_ml, o16, singles, n_single, H, Dv, nsplit);
            TK_CHECK_LAUNCH("attn_biased_merge");
        }
    }
#undef TK_AB_D
#undef TK_AB
    return 0;
}

// ---------------------------------------------------------------------------------------------
// Rows [q | k | v] -> the queries and, in the paged pool, the keys and values, with a norm over a token's whole q row
// (all heads at once) and over its whole k row: x / sqrt(mean(x^2) + eps) * w. One block per token.
// ---------------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
qkv_row_norm_write_kernel(const T* qkv, int64_t stride, const float* __restrict__ wq, const float* __restrict__ wk, float eps,
                          const int* positions, const int* tok_seq, const int* block_table, int bt_stride, T* q_out, T* pool,
                          int nq, int nk, int nv, int Hkv, int D, int Dv, int P, int Dp) {
    __shared__ float red[66];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const T* row = qkv + (size_t)t * stride;
    struct __align__(sizeof(T) * VEC) Chunk { T v[VEC]; };
    auto squares = [&](const T* x, int n) {
        float ss = 0.f;
        for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
            const Chunk c = *reinterpret_cast<const Chunk*>(x + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss = fmaf(to_f<T>(c.v[e]), to_f<T>(c.v[e]), ss);
        }
        return ss;
    };
    const T* k = row + nq;
    const T* v = k + nk;
    const bool write = pool != nullptr;
    const int pos = positions[t];
    const int page = write ? TK_PAGE(TK_K_ATTN_BIASED, block_table[(size_t)tok_seq[t] * bt_stride + pos / P]) : 0;
    const float2 ss = block_sum2(make_float2(squares(row, nq), write ? squares(k, nk) : 0.f), red);
    const float rq = 1.0f / sqrtf(ss.x / (float)nq + eps), rk = 1.0f / sqrtf(ss.y / (float)nk + eps);
    auto normed = [&](const T* x, int i, float rstd, const float* w) {
        Chunk c = *reinterpret_cast<const Chunk*>(x + i);
#pragma unroll
        for (int e = 0; e < VEC; ++e) c.v[e] = from_f<T>(to_f<T>(c.v[e]) * rstd * w[i + e]);
        return c;
    };
    for (int i = threadIdx.x * VEC; i < nq; i += blockDim.x * VEC)
        *reinterpret_cast<Chunk*>(q_out + (size_t)t * nq + i) = normed(row, i, rq, wq);
    if (!write) return;
    // [page][K | V][head][slot in page][Dp]
    T* kd = pool + (((size_t)page * 2 + 0) * Hkv * P + pos % P) * Dp;
    T* vd = pool + (((size_t)page * 2 + 1) * Hkv * P + pos % P) * Dp;
    for (int i = threadIdx.x * VEC; i < nk; i += blockDim.x * VEC)
        *reinterpret_cast<Chunk*>(kd + (size_t)(i / D) * P * Dp + i % D) = normed(k, i, rk, wk);
    for (int i = threadIdx.x * VEC; i < nv; i += blockDim.x * VEC)
        *reinterpret_cast<Chunk*>(vd + (size_t)(i / Dv) * P * Dp + i % Dv) = *reinterpret_cast<const Chunk*>(v + i);
}

// qkv: [T, >= H D + Hkv (D + Dv)] rows `stride` apart; wq: float32 [H D], wk: float32 [Hkv D]; q_out: [T, H, D]; pool (null:
// queries only): [pages, 2, Hkv, P, Dp] with Dp >= max(D, Dv).
TK_API int tk_qkv_row_norm_write(const void* qkv, int64_t stride, const float* wq, const float* wk, float eps,
                                 const int* positions, const int* tok_seq, const int* block_table, int bt_stride, void* q_out,
                                 void* pool, int tokens, int H, int Hkv, int D, int Dv, int P, int Dp, int dtype,
                                 cudaStream_t stream) {
    TK_CHECK_ARG(tokens >= 0 && H > 0 && Hkv > 0 && D > 0 && Dv > 0, "qkv_row_norm_write: bad sizes");
    TK_CHECK_ARG(pool == nullptr || (block_table != nullptr && wk != nullptr && P > 0 && Dp >= D && Dp >= Dv),
                 "qkv_row_norm_write: cache rows of %d for keys of %d and values of %d", Dp, D, Dv);
    if (tokens == 0) return 0;
    const int es = dtype == TK_BF16 ? 2 : 4, vec = 16 / es;
    const bool wide = D % vec == 0 && Dv % vec == 0 && stride % vec == 0 && (pool == nullptr || Dp % vec == 0) &&
                      (((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)pool) & 15) == 0;
#define TK_QN(TT, VEC)                                                                                                   \
    tk_launch(qkv_row_norm_write_kernel<TT, VEC>, dim3(tokens), dim3(256), 0, stream, (const TT*)qkv, stride, wq, wk, eps, \
              positions, tok_seq, block_table, bt_stride, (TT*)q_out, (TT*)pool, H * D, Hkv * D, Hkv * Dv, Hkv, D, Dv, P, Dp)
    if (dtype == TK_F32) {
        if (wide) TK_QN(float, 4);
        else TK_QN(float, 1);
    } else if (dtype == TK_BF16) {
        if (wide) TK_QN(__nv_bfloat16, 8);
        else TK_QN(__nv_bfloat16, 1);
    } else {
        TK_CHECK_ARG(false, "qkv_row_norm_write: unknown dtype %d", dtype);
    }
#undef TK_QN
    TK_CHECK_LAUNCH("qkv_row_norm_write");
    return 0;
}
