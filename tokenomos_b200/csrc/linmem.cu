// Linear memories: recurrent mixers whose state is a matrix S [D, V] per head (D key channels, V values), walked
// in token order with S in registers. Everything here is 32-bit arithmetic; the storage type T is only what q, k, v
// are read as. Two rules and three kinds of decay, each a template parameter:
//
//   additive:  S <- a S;  S <- S + k v^T;                               o = S^T q
//   delta:     S <- a S;  u = beta (v - S^T k);  S <- S + k u^T;        o = S^T q
//
//   a fixed per head (a constant of the layer), a per head and token, or a per key channel and token; the last two
//   are a = exp(-A[h] * softplus(z + bias)). beta = sigmoid(zb). With `unit`, k and q are first brought to unit
//   length, x / sqrt(sum(x^2) + 1e-6); with `act`, q, k and v first pass silu; with `freq`, the first 2 n columns of q and k
//   are rotated by position * freq[i] (pairs (i, i + n)); q is multiplied by q_scale.
//   Head h reads the q/k head h / (H / K).
//
// Eight lanes own a column of S: lane r of them has the rows 32 i + 4 r .. + 3 (i < R / 4), so that the state
// [H, V, D] and the staged rows of k, q and a are read 16 bytes a lane, 128 bytes a column. The read-out is formed
// from the decayed state and the step that is about to be written, o = (aS)^T q + (k . q) u, so that both sums
// over the rows, (aS)^T k and (aS)^T q, run side by side and only the first is on the path from token to token.
//
// A step continues from the stored S exactly where the step before left it, and a token's arithmetic is the same
// wherever the request was cut, to rounding; a sequence at position 0 starts from zeros whatever its state row holds.
//
// The additive rule with a fixed decay is linear in S, so a long portion need not be walked by one block per columns from
// end to end: it is cut into segments of LM_SEG tokens, a first pass walks all of them but the last side by side for what
// each adds to the state (no read-out), and in the second pass a segment's block starts from S' = a^LM_SEG S + (what the
// segment before added), formed over the segments before it, all in 32-bit like the walk itself.
#include <math.h>

#include "common.cuh"

namespace {
enum : int { TK_K_LINMEM = 13 };
constexpr int LM_COLS = 4;       // columns of a warp (times the columns per thread)
constexpr int LM_TOK = 16;       // tokens of a stage
constexpr int LM_STAGES = 3;
constexpr int LM_SEG = 256;      // tokens of a segment (whole stages)

enum : int { LM_ADD = 0, LM_DELTA = 1 };
enum : int { LM_FIXED = 0, LM_HEAD = 1, LM_CHANNEL = 2 };

struct LinMem {
    const void* qkv;
    int64_t stride;
    int q_off, k_off, v_off;
    const float* zb;             // [T, >= H] (delta)
    int64_t zb_stride;
    const float* za;             // [T, >= H] or [T, >= H D]
    int64_t za_stride;
    const float* bias;           // [H] or [H D]
    const float* A;              // [H]: exp(A_log), or the fixed decays
    float* state;                // [slots, H, V, D]
    const int* cu_seqlens;
    const int* seq_ctx;
    const int* seq_slot;
    float* y;                    // [T, H V]
    int H, K, D, V;
    float q_scale;
    int unit, act;
    const float* freq;           // [half] or null
    int half;
    const int* positions;        // [T], with freq
};

__device__ __forceinline__ float lm_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float lm_decay(float z, float A) { return expf(-A * (z > 20.f ? z : log1pf(expf(z)))); }

// Two 32-bit multiply-adds in one instruction (sm_100's packed form), each half rounded as the scalar one.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)),
          "l"(reinterpret_cast<unsigned long long&>(c)));
    return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("mul.rn.f32x2 %0, %1, %2;"
        : "=l"(reinterpret_cast<unsigned long long&>(d))
        : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)));
    return d;
}
__device__ __forceinline__ float2 two(float x) { return make_float2(x, x); }
__device__ __forceinline__ float sum8(float v) {      // over the eight lanes of a column
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    return v;
}

// A column's rows between registers and memory
template <int R>
__device__ __forceinline__ void lm_load(float2 (&S)[R / 2], const float* col, int r, int D, bool ok) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const int d = 32 * i + 4 * r;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (ok && d < D) {
            if (D % 4 == 0) {
                v = *reinterpret_cast<const float4*>(col + d);
            } else {
                v.x = col[d];
                if (d + 1 < D) v.y = col[d + 1];
                if (d + 2 < D) v.z = col[d + 2];
                if (d + 3 < D) v.w = col[d + 3];
            }
        }
        S[2 * i] = make_float2(v.x, v.y);
        S[2 * i + 1] = make_float2(v.z, v.w);
    }
}
template <int R>
__device__ __forceinline__ void lm_store(const float2 (&S)[R / 2], float* col, int r, int D, bool ok) {
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const int d = 32 * i + 4 * r;
        if (!ok || d >= D) continue;
        if (D % 4 == 0) {
            *reinterpret_cast<float4*>(col + d) = make_float4(S[2 * i].x, S[2 * i].y, S[2 * i + 1].x, S[2 * i + 1].y);
        } else {
            col[d] = S[2 * i].x;
            if (d + 1 < D) col[d + 1] = S[2 * i].y;
            if (d + 2 < D) col[d + 2] = S[2 * i + 1].x;
            if (d + 3 < D) col[d + 3] = S[2 * i + 1].y;
        }
    }
}

// One token for one column: S moves on, the column's output comes back (on all eight lanes). k, q, a: this lane's
// first row of the staged vectors.
template <int R, int RULE, int DECAY>
__device__ __forceinline__ float lm_step(float2 (&S)[R / 2], const float* k, const float* q, const float* ga, float a,
                                         float v, float beta, float kq) {
    float2 kk[R / 2];
    float2 pk0 = two(0.f), pk1 = two(0.f), pq0 = two(0.f), pq1 = two(0.f);
#pragma unroll
    for (int i = 0; i < R / 4; ++i) {
        const float4 k4 = *reinterpret_cast<const float4*>(k + 32 * i);
        const float4 q4 = *reinterpret_cast<const float4*>(q + 32 * i);
        kk[2 * i] = make_float2(k4.x, k4.y);
        kk[2 * i + 1] = make_float2(k4.z, k4.w);
        if constexpr (DECAY == LM_CHANNEL) {
            const float4 g4 = *reinterpret_cast<const float4*>(ga + 32 * i);
            S[2 * i] = mul2(S[2 * i], make_float2(g4.x, g4.y));
            S[2 * i + 1] = mul2(S[2 * i + 1], make_float2(g4.z, g4.w));
        }
        if constexpr (RULE == LM_DELTA) {
            pk0 = fma2(S[2 * i], kk[2 * i], pk0);
            pk1 = fma2(S[2 * i + 1], kk[2 * i + 1], pk1);
        }
        pq0 = fma2(S[2 * i], make_float2(q4.x, q4.y), pq0);
        pq1 = fma2(S[2 * i + 1], make_float2(q4.z, q4.w), pq1);
    }
    float u = v, o;
    if constexpr (RULE == LM_DELTA) {
        const float p = sum8((pk0.x + pk0.y) + (pk1.x + pk1.y));
        u = beta * (DECAY == LM_CHANNEL ? v - p : fmaf(-a, p, v));
    }
#pragma unroll
    for (int i = 0; i < R / 2; ++i) S[i] = fma2(kk[i], two(u), DECAY == LM_CHANNEL ? S[i] : mul2(two(a), S[i]));
    o = sum8((pq0.x + pq0.y) + (pq1.x + pq1.y));
    return fmaf(kq, u, DECAY == LM_CHANNEL ? o : a * o);
}

// A warp stages one token's k and q (silu, rotation, unit length, q_scale), k . q and the decay per channel. A lane holds
// the elements lane + 32 j.
template <typename T, int DPL>
__device__ __forceinline__ void lm_fetch(const LinMem& m, int row, int h, int lane, float (&kv)[DPL], float (&qv)[DPL]) {
    const T* src = (const T*)m.qkv + (size_t)row * m.stride;
    const int kh = h / (m.H / m.K);
#pragma unroll
    for (int j = 0; j < DPL; ++j) {
        const int d = lane + 32 * j;
        kv[j] = d < m.D ? to_f<T>(src[m.k_off + kh * m.D + d]) : 0.f;
        qv[j] = d < m.D ? to_f<T>(src[m.q_off + kh * m.D + d]) : 0.f;
    }
}
// The same elements' partners in the rotation (which may be another lane's elements), asked for with them; and the rotation,
// cs holding cos and sin of the token's angles.
template <typename T, int DPL>
__device__ __forceinline__ void lm_fetch_partners(const LinMem& m, int row, int h, int lane, float (&kp)[DPL], float (&qp)[DPL]) {
    const T* src = (const T*)m.qkv + (size_t)row * m.stride + (size_t)(h / (m.H / m.K)) * m.D;
#pragma unroll
    for (int j = 0; j < DPL; ++j) {
        const int d = lane + 32 * j, other = d < m.half ? d + m.half : d - m.half;
        kp[j] = d < 2 * m.half ? to_f<T>(src[m.k_off + other]) : 0.f;
        qp[j] = d < 2 * m.half ? to_f<T>(src[m.q_off + other]) : 0.f;
    }
}
template <int DPL>
__device__ __forceinline__ void lm_rotate(const LinMem& m, int lane, const float2* cs, float (&kv)[DPL], float (&qv)[DPL],
                                          float (&kp)[DPL], float (&qp)[DPL]) {
#pragma unroll
    for (int j = 0; j < DPL; ++j) {
        const int d = lane + 32 * j;
        if (m.act) {
            kv[j] = lm_silu(kv[j]), kp[j] = lm_silu(kp[j]);
            qv[j] = lm_silu(qv[j]), qp[j] = lm_silu(qp[j]);
        }
        if (d < 2 * m.half) {
            const float2 c = cs[d < m.half ? d : d - m.half];
            const float s = d < m.half ? -c.y : c.y;
            kv[j] = kv[j] * c.x + kp[j] * s;
            qv[j] = qv[j] * c.x + qp[j] * s;
        }
    }
}
template <int DPL>
__device__ __forceinline__ void lm_shape(const LinMem& m, int lane, float (&kv)[DPL], float (&qv)[DPL], float* ks, float* qs,
                                         float* kq) {
    if (m.act && m.freq == nullptr) {
#pragma unroll
        for (int j = 0; j < DPL; ++j) {
            kv[j] = lm_silu(kv[j]);
            qv[j] = lm_silu(qv[j]);
        }
    }
    float sk = 0.f, sq = 0.f, s = 0.f;
#pragma unroll
    for (int j = 0; j < DPL; ++j) {
        sk = fmaf(kv[j], kv[j], sk);
        sq = fmaf(qv[j], qv[j], sq);
        s = fmaf(kv[j], qv[j], s);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        s += __shfl_xor_sync(0xffffffffu, s, o);
    }
    const float mk = m.unit ? 1.0f / sqrtf(sk + 1e-6f) : 1.0f;
    const float mq = (m.unit ? 1.0f / sqrtf(sq + 1e-6f) : 1.0f) * m.q_scale;
#pragma unroll
    for (int j = 0; j < DPL; ++j) {
        ks[lane + 32 * j] = kv[j] * mk;
        qs[lane + 32 * j] = qv[j] * mq;
    }
    if (lane == 0) *kq = s * mk * mq;
}
}  // namespace

// Portions, first kernel: everything a token brings to the walk that does not depend on the state, formed once and laid
// out as the walk reads it (32-bit, zeros past D and V): kq [K][T'][k | q][DP], decays [H][T'][DP] (per channel),
// values [H][T'][VP], and per head and token (a, beta, k . q, -). T' = T + LM_TOK rows, so that a stage may read past the
// last token. One block per token.
struct LinMemPrep {
    float *kq, *g, *v;
    float4* sc;
    int rows, VP;            // T', the values' padded size
    float* seg;              // [slots][H][V][D]: what each segment adds to the state, or null: no segments
    int n_seqs;
};

// The segment a block works on: sequence s's segments have the slots cu_seqlens[s] / LM_SEG + s and up (as many as it can
// need), so that the slots of all sequences together are at most tokens / LM_SEG + n_seqs.
struct LmSegment {
    int s, j, n;             // sequence, which of its n segments (j >= n: none)
    int slot0;               // its first segment's slot
};
__device__ __forceinline__ LmSegment lm_segment(const LinMem& m, int n_seqs, int slot) {
    // the last sequence whose first slot is not past this one (every warp looks for itself, 32 sequences at a time)
    int lo = -1;
    for (int s0 = 0; s0 < n_seqs; s0 += 32) {
        const int s = s0 + (threadIdx.x & 31);
        const unsigned before = __ballot_sync(0xffffffffu, s < n_seqs && m.cu_seqlens[s] / LM_SEG + s <= slot);
        lo += __popc(before);
        if (before != 0xffffffffu) break;
    }
    LmSegment g;
    g.s = lo;
    const int first = m.cu_seqlens[lo];
    g.slot0 = first / LM_SEG + lo;
    g.j = slot - g.slot0;
    g.n = (m.cu_seqlens[lo + 1] - first + LM_SEG - 1) / LM_SEG;
    return g;
}

template <typename T, int DPL, int RULE, int DECAY>
__global__ void __launch_bounds__(256)
linmem_prepare_kernel(const LinMem m, const LinMemPrep p) {
    constexpr int DP = 32 * DPL;
    extern __shared__ __align__(8) float prep_s[];       // cos and sin [half][2], k . q [K]
    float2* cs = reinterpret_cast<float2*>(prep_s);
    float* kq_s = prep_s + 2 * m.half;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (m.freq != nullptr) {
        const float pos = (float)m.positions[t];
        for (int i = threadIdx.x; i < m.half; i += 256) sincosf(pos * m.freq[i], &cs[i].y, &cs[i].x);
        __syncthreads();
    }
    for (int kh = warp; kh < m.K; kh += 8) {
        float kv[DPL], qv[DPL];
        float* dst = p.kq + ((size_t)kh * p.rows + t) * 2 * DP;
        lm_fetch<T, DPL>(m, t, kh * (m.H / m.K), lane, kv, qv);
        if (m.freq != nullptr) {
            float kp[DPL], qp[DPL];
            lm_fetch_partners<T, DPL>(m, t, kh * (m.H / m.K), lane, kp, qp);
            lm_rotate<DPL>(m, lane, cs, kv, qv, kp, qp);
        }
        lm_shape<DPL>(m, lane, kv, qv, dst, dst + DP, kq_s + kh);
    }
    const T* v = (const T*)m.qkv + (size_t)t * m.stride + m.v_off;
    for (int i = threadIdx.x; i < m.H * p.VP; i += 256) {
        const int h = i / p.VP, c = i % p.VP;
        float x = c < m.V ? to_f<T>(v[h * m.V + c]) : 0.f;
        p.v[((size_t)h * p.rows + t) * p.VP + c] = m.act ? lm_silu(x) : x;
    }
    if constexpr (DECAY == LM_CHANNEL) {
        for (int i = threadIdx.x; i < m.H * DP; i += 256) {
            const int h = i / DP, d = i % DP;
            p.g[((size_t)h * p.rows + t) * DP + d] =
                d < m.D ? lm_decay(m.za[(size_t)t * m.za_stride + h * m.D + d] + m.bias[h * m.D + d], m.A[h]) : 1.f;
        }
    }
    __syncthreads();
    for (int h = threadIdx.x; h < m.H; h += 256) {
        float4 s = make_float4(m.A[h], 0.f, kq_s[h / (m.H / m.K)], 0.f);
        if constexpr (RULE == LM_DELTA) s.y = 1.0f / (1.0f + expf(-m.zb[(size_t)t * m.zb_stride + h]));
        if constexpr (DECAY == LM_HEAD) s.x = lm_decay(m.za[(size_t)t * m.za_stride + h] + m.bias[h], m.A[h]);
        p.sc[(size_t)h * p.rows + t] = s;
    }
}

__device__ __forceinline__ void lm_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// Segments, first pass: what a segment adds to the state (the sequence's first one: on top of the stored state, of which it
// leaves a copy in the last segment's slot, since the last segment's block will overwrite the stored one).
template <int R, int CPT>
__global__ void __launch_bounds__(256)
linmem_segment_kernel(const LinMem m, const LinMemPrep p) {
    constexpr int DP = 8 * R;
    extern __shared__ __align__(16) float smem[];        // [stage][k per token, values]
    pdl_launch_dependents();
    pdl_wait();
    const LmSegment g = lm_segment(m, p.n_seqs, blockIdx.z);
    if (g.j >= g.n - 1) return;                          // the last segment is nobody's past
    const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y, cols = LM_COLS * CPT * warps, c0 = blockIdx.x * cols;
    const int first = m.cu_seqlens[g.s] + g.j * LM_SEG;
    const int r = lane & 7, wc = warp * LM_COLS * CPT + (lane >> 3);
    const int stage_floats = LM_TOK * (DP + cols);
    const float* k = p.kq + ((size_t)(h / (m.H / m.K)) * p.rows + first) * 2 * DP;
    const float* v = p.v + ((size_t)h * p.rows + first) * p.VP + c0;
    const int v_cols = min(cols, p.VP - c0);
    auto issue = [&](int t0, int b) {
        if (t0 < LM_SEG) {
            float* dst = smem + (size_t)b * stage_floats;
            for (int i = threadIdx.x; i < LM_TOK * DP / 4; i += blockDim.x) {
                const int t = i / (DP / 4), d = (i % (DP / 4)) * 4;
                lm_copy16(dst + t * DP + d, k + (size_t)(t0 + t) * 2 * DP + d);
            }
            dst += LM_TOK * DP;
            for (int i = threadIdx.x; i < LM_TOK * cols / 4; i += blockDim.x) {
                const int t = i / (cols / 4), c = (i % (cols / 4)) * 4;
                if (c < v_cols) lm_copy16(dst + t * cols + c, v + (size_t)(t0 + t) * p.VP + c);
            }
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
#pragma unroll
    for (int i = 0; i < LM_STAGES - 1; ++i) issue(i * LM_TOK, i);

    const size_t head = (size_t)m.V * m.D;
    const float* st = m.state + ((size_t)TK_SLOT(TK_K_LINMEM, m.seq_slot[g.s]) * m.H + h) * head;
    float* mine = p.seg + ((size_t)blockIdx.z * m.H + h) * head;
    float* last = p.seg + ((size_t)(g.slot0 + g.n - 1) * m.H + h) * head;
    const bool carried = m.seq_ctx[g.s] > 0 && g.j == 0;
    float2 S[CPT][R / 2];
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const int col = c0 + wc + LM_COLS * c;
        lm_load<R>(S[c], st + (size_t)col * m.D, r, m.D, carried && col < m.V);
        if (g.j == 0) lm_store<R>(S[c], last + (size_t)col * m.D, r, m.D, col < m.V);
    }
    const float2 a = two(m.A[h]);
    int b = 0;
    for (int t0 = 0; t0 < LM_SEG; t0 += LM_TOK) {
        asm volatile("cp.async.wait_group %0;\n" ::"n"(LM_STAGES - 2));
        __syncthreads();                                 // the stage is there, and the one before it is read
        issue(t0 + (LM_STAGES - 1) * LM_TOK, (b + LM_STAGES - 1) % LM_STAGES);
        const float* ks = smem + (size_t)b * stage_floats + 4 * r;
        const float* vt = smem + (size_t)b * stage_floats + LM_TOK * DP + wc;
        b = (b + 1) % LM_STAGES;
#pragma unroll 4
        for (int t = 0; t < LM_TOK; ++t) {
            float2 kk[R / 2];
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const float4 k4 = *reinterpret_cast<const float4*>(ks + t * DP + 32 * i);
                kk[2 * i] = make_float2(k4.x, k4.y);
                kk[2 * i + 1] = make_float2(k4.z, k4.w);
            }
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                const float2 u = two(vt[t * cols + LM_COLS * c]);
#pragma unroll
                for (int i = 0; i < R / 2; ++i) S[c][i] = fma2(kk[i], u, mul2(a, S[c][i]));
            }
        }
    }
    asm volatile("cp.async.wait_group 0;\n" ::);
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const int col = c0 + wc + LM_COLS * c;
        lm_store<R>(S[c], mine + (size_t)col * m.D, r, m.D, col < m.V);
    }
}

// Portions, second kernel: a block owns LM_COLS * CPT columns a warp of a head of a sequence and walks the sequence's
// tokens; stages of LM_TOK tokens are copied LM_STAGES - 1 ahead. SEG: it walks one segment of the sequence.
template <int R, int RULE, int DECAY, int CPT, bool SEG>
__global__ void __launch_bounds__(256)
linmem_scan_kernel(const LinMem m, const LinMemPrep p) {
    constexpr int DP = 8 * R;                            // the key size, padded
    constexpr int VEC = DECAY == LM_CHANNEL ? 3 : 2;     // staged vectors per token
    extern __shared__ __align__(16) float smem[];        // [stage][k | q per token, decays, values, scalars]
    pdl_launch_dependents();
    pdl_wait();
    const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    LmSegment sg{(int)blockIdx.z, 0, 1, 0};
    if constexpr (SEG) {
        sg = lm_segment(m, p.n_seqs, blockIdx.z);
        if (sg.j >= sg.n) return;
    }
    const int s = sg.s, h = blockIdx.y, cols = LM_COLS * CPT * warps, c0 = blockIdx.x * cols;
    const int first = m.cu_seqlens[s] + sg.j * LM_SEG, rest = m.cu_seqlens[s + 1] - first;
    const int len = SEG ? min(rest, LM_SEG) : rest;
    if (len <= 0) return;
    const int r = lane & 7, wc = warp * LM_COLS * CPT + (lane >> 3);        // this thread's first column of the block
    const int stage_floats = LM_TOK * (VEC * DP + cols + 4);
    const float* kq = p.kq + ((size_t)(h / (m.H / m.K)) * p.rows + first) * 2 * DP;
    const float* g = DECAY == LM_CHANNEL ? p.g + ((size_t)h * p.rows + first) * DP : nullptr;
    const float* v = p.v + ((size_t)h * p.rows + first) * p.VP + c0;
    const float* sc = reinterpret_cast<const float*>(p.sc + (size_t)h * p.rows + first);
    const int v_cols = min(cols, p.VP - c0);             // (VP and cols are whole 16-byte chunks)
    auto issue = [&](int t0, int b) {
        if (t0 < len) {
            float* dst = smem + (size_t)b * stage_floats;
            for (int i = threadIdx.x; i < LM_TOK * 2 * DP / 4; i += blockDim.x) lm_copy16(dst + 4 * i, kq + (size_t)t0 * 2 * DP + 4 * i);
            dst += LM_TOK * 2 * DP;
            if constexpr (DECAY == LM_CHANNEL) {
                for (int i = threadIdx.x; i < LM_TOK * DP / 4; i += blockDim.x) lm_copy16(dst + 4 * i, g + (size_t)t0 * DP + 4 * i);
                dst += LM_TOK * DP;
            }
            for (int i = threadIdx.x; i < LM_TOK * cols / 4; i += blockDim.x) {
                const int t = i / (cols / 4), c = (i % (cols / 4)) * 4;
                if (c < v_cols) lm_copy16(dst + t * cols + c, v + (size_t)(t0 + t) * p.VP + c);
            }
            dst += LM_TOK * cols;
            for (int i = threadIdx.x; i < LM_TOK; i += blockDim.x) lm_copy16(dst + 4 * i, sc + 4 * (size_t)(t0 + i));
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
#pragma unroll
    for (int i = 0; i < LM_STAGES - 1; ++i) issue(i * LM_TOK, i);

    float* st = m.state + ((size_t)TK_SLOT(TK_K_LINMEM, m.seq_slot[s]) * m.H + h) * m.V * m.D;
    float2 S[CPT][R / 2];
    const bool carried = m.seq_ctx[s] > 0;
    if (SEG && sg.n > 1) {
        const size_t head = (size_t)m.V * m.D, slot = m.H * head;
        const float* seg = p.seg + (size_t)sg.slot0 * slot + h * head;
        const float* from = seg + (size_t)(sg.j == 0 ? sg.n - 1 : 0) * slot;     // the stored state's copy, or the first segment's
        const float2 a = two(powf(m.A[h], (float)LM_SEG));
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            const int col = c0 + wc + LM_COLS * c;
            lm_load<R>(S[c], from + (size_t)col * m.D, r, m.D, col < m.V);
        }
        for (int i = 1; i < sg.j; ++i) {
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                float2 more[R / 2];
                const int col = c0 + wc + LM_COLS * c;
                lm_load<R>(more, seg + (size_t)i * slot + (size_t)col * m.D, r, m.D, col < m.V);
#pragma unroll
                for (int e = 0; e < R / 2; ++e) S[c][e] = fma2(a, S[c][e], more[e]);
            }
        }
    } else {
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            const int col = c0 + wc + LM_COLS * c;
            lm_load<R>(S[c], st + (size_t)col * m.D, r, m.D, carried && col < m.V);
        }
    }
    const int HV = m.H * m.V;
    float* y = m.y + (size_t)first * HV + h * m.V + c0 + wc;
    int b = 0;
    for (int t0 = 0; t0 < len; t0 += LM_TOK) {
        asm volatile("cp.async.wait_group %0;\n" ::"n"(LM_STAGES - 2));
        __syncthreads();                                 // the stage is there, and the one before it is read
        issue(t0 + (LM_STAGES - 1) * LM_TOK, (b + LM_STAGES - 1) % LM_STAGES);
        const float* base = smem + (size_t)b * stage_floats;
        b = (b + 1) % LM_STAGES;
        const float* ks = base + 4 * r;
        const float* gs = base + LM_TOK * 2 * DP + 4 * r;
        const float* vt = base + LM_TOK * VEC * DP + wc;
        const float4* scs = reinterpret_cast<const float4*>(base + LM_TOK * (VEC * DP + cols));
        auto walk = [&](int t, float (&o)[CPT]) {
            const float4 c4 = scs[t];
#pragma unroll
            for (int c = 0; c < CPT; ++c)
                o[c] = lm_step<R, RULE, DECAY>(S[c], ks + t * 2 * DP, ks + t * 2 * DP + DP, gs + t * DP, c4.x,
                                               vt[t * cols + LM_COLS * c], c4.y, c4.z);
        };
        const int nt = min(LM_TOK, len - t0);
        if (nt == LM_TOK) {
            float keep[CPT];
#pragma unroll 8
            for (int t = 0; t < LM_TOK; ++t) {
                float o[CPT];
                walk(t, o);
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    if (r == (t & 7)) keep[c] = o[c];
                    if ((t & 7) == 7 && c0 + wc + LM_COLS * c < m.V) y[(size_t)(t0 + t - 7 + r) * HV + LM_COLS * c] = keep[c];
                }
            }
        } else {
            for (int t = 0; t < nt; ++t) {
                float o[CPT];
                walk(t, o);
#pragma unroll
                for (int c = 0; c < CPT; ++c)
                    if (r == 0 && c0 + wc + LM_COLS * c < m.V) y[(size_t)(t0 + t) * HV + LM_COLS * c] = o[c];
            }
        }
    }
    asm volatile("cp.async.wait_group 0;\n" ::);
    if (SEG && sg.j + 1 < sg.n) return;                  // the sequence's last segment leaves the new state
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const int col = c0 + wc + LM_COLS * c;
        lm_store<R>(S[c], st + (size_t)col * m.D, r, m.D, col < m.V);
    }
}

// Steps of single tokens (a few a sequence at most): the state streams through, CPT columns a thread, so that many
// bytes are in flight; the block's warps stage a token's vectors together.
// (ROT: the angles' code would take registers that the state's loads in flight want: three blocks an SM)
template <typename T, int R, int RULE, int DECAY, int CPT, bool ROT>
__global__ void __launch_bounds__(256, ROT && R <= 16 ? 3 : 0)
linmem_token_kernel(const LinMem m) {
    constexpr int DPL = R / 4, DP = 8 * R;
    __shared__ __align__(16) float ks[DP], qs[DP], gs[DECAY == LM_CHANNEL ? DP : 4];
    __shared__ float kq_s;
    __shared__ float2 cs[ROT ? DP / 2 : 1];
    pdl_launch_dependents();
    pdl_wait();
    const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int s = blockIdx.z, h = blockIdx.y, c0 = (blockIdx.x * warps + warp) * LM_COLS * CPT + (lane >> 3);
    const int first = m.cu_seqlens[s], len = m.cu_seqlens[s + 1] - first;
    if (len <= 0) return;
    const int r = lane & 7;
    const float A = m.A[h];
    const int ctx = m.seq_ctx[s];
    const bool carried = ctx > 0;
    float* st = m.state + ((size_t)TK_SLOT(TK_K_LINMEM, m.seq_slot[s]) * m.H + h) * m.V * m.D;
    float2 S[CPT][R / 2];
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const int col = c0 + LM_COLS * c;
        lm_load<R>(S[c], st + (size_t)col * m.D, r, m.D, carried && col < m.V);
    }
    for (int t = 0; t < len; ++t) {
        const int row = first + t;
        float v[CPT], beta = 0.f, a = A;
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            const int col = c0 + LM_COLS * c;
            v[c] = col < m.V ? to_f<T>(((const T*)m.qkv)[(size_t)row * m.stride + m.v_off + h * m.V + col]) : 0.f;
            if (m.act) v[c] = lm_silu(v[c]);
        }
        if constexpr (RULE == LM_DELTA) beta = 1.0f / (1.0f + expf(-m.zb[(size_t)row * m.zb_stride + h]));
        if constexpr (DECAY == LM_HEAD) a = lm_decay(m.za[(size_t)row * m.za_stride + h] + m.bias[h], A);
        if (t > 0) __syncthreads();
        if (warp == 0) {
            float kv[DPL], qv[DPL];
            lm_fetch<T, DPL>(m, row, h, lane, kv, qv);
            if constexpr (ROT) {
                float kp[DPL], qp[DPL];
                lm_fetch_partners<T, DPL>(m, row, h, lane, kp, qp);
                const float pos = (float)(ctx + t);          // (the angles are formed while the loads are in flight)
                for (int i = lane; i < m.half; i += 32) sincosf(pos * m.freq[i], &cs[i].y, &cs[i].x);
                __syncwarp();
                lm_rotate<DPL>(m, lane, cs, kv, qv, kp, qp);
            }
            lm_shape<DPL>(m, lane, kv, qv, ks, qs, &kq_s);
        }
        if constexpr (DECAY == LM_CHANNEL) {
            for (int d = threadIdx.x; d < DP; d += blockDim.x) {
                float g = 1.f;
                if (d < m.D) g = lm_decay(m.za[(size_t)row * m.za_stride + h * m.D + d] + m.bias[h * m.D + d], A);
                gs[d] = g;
            }
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
            const float o = lm_step<R, RULE, DECAY>(S[c], ks + 4 * r, qs + 4 * r, gs + (DECAY == LM_CHANNEL ? 4 * r : 0), a,
                                                    v[c], beta, kq_s);
            const int col = c0 + LM_COLS * c;
            if (r == 0 && col < m.V) m.y[(size_t)row * m.H * m.V + h * m.V + col] = o;
        }
    }
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const int col = c0 + LM_COLS * c;
        lm_store<R>(S[c], st + (size_t)col * m.D, r, m.D, col < m.V);
    }
}

namespace {
// Slots of the segments of a step (0: no segments): where the additive rule would otherwise leave most of the GPU idle, or
// might, for all that a recorded step knows of its sequences' lengths.
int lm_slots(int tokens, int n_seqs, int H, int D, int V, int decay, int sm_count) {
    if (decay != LM_FIXED || tokens < 2 * LM_SEG || n_seqs <= 0) return 0;
    const int64_t cols = LM_COLS * (D > 128 ? 1 : 2) * 4, blocks = (V + cols - 1) / cols * H * n_seqs;
    const int64_t slots = tokens / LM_SEG + n_seqs;
    if (blocks >= 2 * sm_count && tokens > 4096) return 0;
    return slots * H * V * D * 4 <= (int64_t)256 << 20 && slots <= 65535 ? (int)slots : 0;
}

template <typename T, int R, int RULE, int DECAY>
void lm_launch(const LinMem& m, int n_seqs, int tokens, float* scratch, int sm_count, cudaStream_t stream) {
    if (scratch == nullptr) {
        constexpr int CPT = R >= 32 ? 1 : 2;
        const int per_warp = LM_COLS * CPT;
        int warps = (m.V + per_warp - 1) / per_warp;
        const int blocks = (warps + 7) / 8;
        warps = (warps + blocks - 1) / blocks;
        const dim3 grid(blocks, m.H, n_seqs), block(32 * warps);
        if (DECAY == LM_FIXED && m.freq != nullptr)
            tk_launch(linmem_token_kernel<T, R, RULE, DECAY, CPT, DECAY == LM_FIXED>, grid, block, 0, stream, m);
        else
            tk_launch(linmem_token_kernel<T, R, RULE, DECAY, CPT, false>, grid, block, 0, stream, m);
        return;
    }
    constexpr int DP = 8 * R, VEC = DECAY == LM_CHANNEL ? 3 : 2;
    LinMemPrep p;
    p.rows = tokens + LM_TOK;
    p.VP = (m.V + 3) / 4 * 4;
    p.kq = scratch;
    p.v = p.kq + (size_t)m.K * p.rows * 2 * DP;
    p.sc = reinterpret_cast<float4*>(p.v + (size_t)m.H * p.rows * p.VP);
    p.g = reinterpret_cast<float*>(p.sc + (size_t)m.H * p.rows);
    p.seg = nullptr;
    p.n_seqs = n_seqs;
    tk_launch(linmem_prepare_kernel<T, R / 4, RULE, DECAY>, dim3(tokens), dim3(256),
              (m.K + 2 * m.half) * sizeof(float), stream, m, p);
    // Two columns a thread (one where a column alone is 32 registers) in blocks of four warps; eight warps, which share
    // a stage's copies among more columns, only where even a quarter of the sequences (the least a recorded step of
    // this shape was recorded for) would fill the GPU with them
    constexpr int CPT = R >= 32 ? 1 : 2;
    int warps = (m.V + LM_COLS * CPT * 8 - 1) / (LM_COLS * CPT * 8) * m.H * (n_seqs / 4) >= sm_count ? 8 : 4;
    while (warps > 1 && m.V <= LM_COLS * CPT * warps / 2) warps /= 2;
    const int cols = LM_COLS * CPT * warps;
    const size_t smem = (size_t)LM_STAGES * LM_TOK * (VEC * DP + cols + 4) * sizeof(float);
    if constexpr (DECAY == LM_FIXED) {
        const int slots = lm_slots(tokens, n_seqs, m.H, m.D, m.V, DECAY, sm_count);
        if (slots > 0) {
            // (four columns of 16 registers a thread: half the reads of shared memory per multiply-add, and segments enough)
            constexpr int SC = R >= 32 ? 1 : R == 16 ? 4 : 2;
            int sw = 4;
            while (sw > 1 && m.V <= LM_COLS * SC * sw / 2) sw /= 2;
            const int sc = LM_COLS * SC * sw;
            const size_t sm = (size_t)LM_STAGES * LM_TOK * (VEC * DP + sc + 4) * sizeof(float);
            p.seg = p.g;                                     // (a fixed decay stages none per channel)
            const dim3 grid((m.V + sc - 1) / sc, m.H, slots);
            static size_t raised_seg = 48 * 1024;
            if (sm > raised_seg) {
                cudaFuncSetAttribute(linmem_segment_kernel<R, SC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
                cudaFuncSetAttribute(linmem_scan_kernel<R, RULE, DECAY, SC, true>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                     (int)sm);
                raised_seg = sm;
            }
            tk_launch_after(linmem_segment_kernel<R, SC>, grid, dim3(32 * sw),
                            (size_t)LM_STAGES * LM_TOK * (DP + sc) * sizeof(float), stream, m, p);
            tk_launch_after(linmem_scan_kernel<R, RULE, DECAY, SC, true>, grid, dim3(32 * sw), sm, stream, m, p);
            return;
        }
    }
    static size_t raised = 48 * 1024;
    if (smem > raised) {
        cudaFuncSetAttribute(linmem_scan_kernel<R, RULE, DECAY, CPT, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        raised = smem;
    }
    tk_launch_after(linmem_scan_kernel<R, RULE, DECAY, CPT, false>, dim3((m.V + cols - 1) / cols, m.H, n_seqs), dim3(32 * warps), smem,
                    stream, m, p);
}

template <typename T, int RULE, int DECAY>
void lm_rows(const LinMem& m, int n_seqs, int tokens, float* scratch, int sm_count, cudaStream_t stream) {
    if (m.D <= 32) lm_launch<T, 4, RULE, DECAY>(m, n_seqs, tokens, scratch, sm_count, stream);
    else if (m.D <= 64) lm_launch<T, 8, RULE, DECAY>(m, n_seqs, tokens, scratch, sm_count, stream);
    else if (m.D <= 128) lm_launch<T, 16, RULE, DECAY>(m, n_seqs, tokens, scratch, sm_count, stream);
    else lm_launch<T, 32, RULE, DECAY>(m, n_seqs, tokens, scratch, sm_count, stream);
}
}  // namespace

TK_API int tk_linmem_max_dim() { return 256; }

// Scratch memory of a step, in units of 32 floats: none for single tokens (a few a sequence at most), else what the
// walk's vectors (and the segments' states) take.
TK_API int tk_linmem_scratch(int tokens, int n_seqs, int H, int K, int D, int V, int decay, int sm_count) {
    if (tokens < 4 * n_seqs || n_seqs == 0) return 0;
    const int64_t DP = D <= 32 ? 32 : D <= 64 ? 64 : D <= 128 ? 128 : 256, VP = (V + 3) / 4 * 4;
    const int64_t floats = (int64_t)(tokens + LM_TOK) * (2 * K * DP + H * (VP + 4) + (decay == LM_CHANNEL ? H * DP : 0)) +
                           (int64_t)lm_slots(tokens, n_seqs, H, D, V, decay, sm_count) * H * V * D;
    return (int)((floats + 31) / 32);
}

// qkv: [T, >= ...] rows `stride` apart holding q (K x D) at column q_off, k at k_off, v (H x V) at v_off; rule 0
// additive, 1 delta (zb: float32 [T, >= H] rows zb_stride apart, beta's logits); decay 0 fixed (A: float32 [H], the
// decays), 1 per head, 2 per channel (za: float32 [T, >= H] or [T, >= H D] rows za_stride apart, bias likewise one
// row, A: float32 [H]). freq (float32 [half], null: none): the rotation's frequencies, with positions [T]. scratch: what tk_linmem_scratch says (16-byte aligned), null for 0. state: float32 [slots, H, V, D]; y: float32 [T, H V].
TK_API int tk_linmem_scan(const void* qkv, int64_t stride, int q_off, int k_off, int v_off, int rule, const float* zb,
                          int64_t zb_stride, int decay, const float* za, int64_t za_stride, const float* bias,
                          const float* A, float* state, const int* cu_seqlens, const int* seq_ctx, const int* seq_slot,
                          int n_seqs, int tokens, float* y, float* scratch, int H, int K, int D, int V, float q_scale, int unit, int act,
                          const float* freq, int half, const int* positions, int sm_count, int dtype, cudaStream_t stream) {
    TK_CHECK_ARG(H > 0 && K > 0 && H % K == 0 && D > 0 && V > 0, "linear memory: %d heads over %d q/k heads", H, K);
    TK_CHECK_ARG(D <= tk_linmem_max_dim(), "linear memory: a key size of %d; up to %d are built", D, tk_linmem_max_dim());
    TK_CHECK_ARG((rule == LM_ADD && decay == LM_FIXED) || (rule == LM_DELTA && (decay == LM_HEAD || decay == LM_CHANNEL)),
                 "linear memory: rule %d with decay %d is not built", rule, decay);
    TK_CHECK_ARG(rule == LM_ADD || (zb != nullptr && za != nullptr && bias != nullptr), "linear memory: missing gates");
    TK_CHECK_ARG(n_seqs >= 0 && tokens >= 0 && A != nullptr, "linear memory: bad sizes");
    if (freq == nullptr) half = 0;
    TK_CHECK_ARG(half >= 0 && 2 * half <= D && (half == 0 || positions != nullptr), "linear memory: %d rotated columns of %d",
                 2 * half, D);
    if (half == 0) freq = nullptr;
    TK_CHECK_ARG(freq == nullptr || decay == LM_FIXED, "linear memory: a rotation is built for a fixed decay");
    if (n_seqs == 0) return 0;
    const LinMem m{qkv, stride, q_off, k_off, v_off, zb, zb_stride, za, za_stride, bias, A, state, cu_seqlens, seq_ctx,
                   seq_slot, y, H, K, D, V, q_scale, unit, act, freq, half, positions};
    TK_CHECK_ARG((scratch != nullptr) == (tk_linmem_scratch(tokens, n_seqs, H, K, D, V, decay, sm_count) > 0),
                 "linear memory: a step of %d tokens in %d sequences without its scratch memory", tokens, n_seqs);
#define TK_LM(TT)                                                                       \
    do {                                                                                \
        if (rule == LM_ADD) lm_rows<TT, LM_ADD, LM_FIXED>(m, n_seqs, tokens, scratch, sm_count, stream);          \
        else if (decay == LM_HEAD) lm_rows<TT, LM_DELTA, LM_HEAD>(m, n_seqs, tokens, scratch, sm_count, stream);  \
        else lm_rows<TT, LM_DELTA, LM_CHANNEL>(m, n_seqs, tokens, scratch, sm_count, stream);                     \
    } while (0)
    if (dtype == TK_F32) TK_LM(float);
    else if (dtype == TK_BF16) TK_LM(__nv_bfloat16);
    else TK_CHECK_ARG(false, "linear memory: unknown dtype %d", dtype);
#undef TK_LM
    TK_CHECK_LAUNCH("linmem_scan");
    return 0;
}

// ---------------------------------------------------------------------------------------------
// out = group_norm(y) * w * gate(z) (w optional): y's row in `groups` equal parts, each divided by its own
// sqrt(mean + eps); gate silu or sigmoid. One warp per (row, group), or, for parts longer than
// LM_WARP_PART, one block.
// ---------------------------------------------------------------------------------------------
namespace {
constexpr int LM_WARP_PART = 512;
enum : int { LM_GATE_SILU = 0, LM_GATE_SIGMOID = 1 };

// 16-bit storage takes the special-function unit's exponential and reciprocal (a few ulp of a float, far below the
// one rounding that follows), 32-bit storage the accurate functions
template <typename T>
__device__ __forceinline__ float lm_gate(float z, int kind) {
    float s;
    if constexpr (sizeof(T) == 2) s = rcp_approx(1.0f + ex2_approx(z * TK_NEG_LOG2E));
    else s = 1.0f / (1.0f + expf(-z));
    return kind == LM_GATE_SILU ? z * s : s;
}
}  // namespace

template <typename T, int ITEMS, bool BLOCK>
__global__ void __launch_bounds__(256)
norm_gate_kernel(const float* y, const T* z, int64_t z_stride, const float* __restrict__ w, float eps, T* out, int rows,
                 int width, int groups, int kind) {
    __shared__ float red[33];
    pdl_launch_dependents();
    pdl_wait();
    const int unit = BLOCK ? blockIdx.x : blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = BLOCK ? threadIdx.x : (threadIdx.x & 31), step = BLOCK ? 256 : 32;
    if (!BLOCK && unit >= rows * groups) return;
    const int r = unit / groups, gw = width / groups, c0 = (unit % groups) * gw;
    const float* src = y + (size_t)r * width + c0;
    const T* gate = z + (size_t)r * z_stride + c0;
    T* dst = out + (size_t)r * width + c0;
    float keep[ITEMS], zv[ITEMS], ss = 0.f;
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
        const int i = lane + step * k;
        keep[k] = i < gw ? src[i] : 0.f;
        zv[k] = i < gw ? to_f<T>(gate[i]) : 0.f;
        ss = fmaf(keep[k], keep[k], ss);
    }
    for (int i = lane + step * ITEMS; i < gw; i += step) ss = fmaf(src[i], src[i], ss);
    ss = BLOCK ? block_sum(ss, red) : warp_sum(ss);
    const float rstd = 1.0f / sqrtf(ss / (float)gw + eps);
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
        const int i = lane + step * k;
        if (i < gw) dst[i] = from_f<T>(keep[k] * rstd * (w != nullptr ? w[c0 + i] : 1.0f) * lm_gate<T>(zv[k], kind));
    }
    for (int i = lane + step * ITEMS; i < gw; i += step)
        dst[i] = from_f<T>(src[i] * rstd * (w != nullptr ? w[c0 + i] : 1.0f) * lm_gate<T>(to_f<T>(gate[i]), kind));
}

// y: float32 [rows, width]; z: [rows, width] (type dtype) rows `z_stride` apart; w: float32 [width] or null; out: [rows, width].
TK_API int tk_norm_gate(const float* y, const void* z, int64_t z_stride, const float* w, float eps, void* out, int rows,
                        int width, int groups, int kind, int dtype, cudaStream_t stream) {
    TK_CHECK_ARG(rows >= 0 && width > 0 && groups > 0 && width % groups == 0, "norm and gate: a row of %d in %d groups",
                 width, groups);
    TK_CHECK_ARG(kind == LM_GATE_SILU || kind == LM_GATE_SIGMOID, "norm and gate: unknown gate %d", kind);
    if (rows == 0) return 0;
    const int gw = width / groups;
#define TK_NG(TT, ITEMS, BLOCK)                                                                                      \
    tk_launch(norm_gate_kernel<TT, ITEMS, BLOCK>, dim3(BLOCK ? rows * groups : (rows * groups + 7) / 8), dim3(256), 0, \
              stream, y, (const TT*)z, z_stride, w, eps, (TT*)out, rows, width, groups, kind)
#define TK_NG_T(TT)                                       \
    do {                                                  \
        if (gw > LM_WARP_PART) TK_NG(TT, 8, true);        \
        else if (gw > 128) TK_NG(TT, 16, false);          \
        else TK_NG(TT, 4, false);                         \
    } while (0)
    if (dtype == TK_F32) TK_NG_T(float);
    else if (dtype == TK_BF16) TK_NG_T(__nv_bfloat16);
    else TK_CHECK_ARG(false, "norm and gate: unknown dtype %d", dtype);
#undef TK_NG_T
#undef TK_NG
    TK_CHECK_LAUNCH("norm_gate");
    return 0;
}

// ---------------------------------------------------------------------------------------------
// Two mixers' outputs joined: out = coef * (a / rms(a) * wa + b / rms(b) * wb), rms over the row with
// eps inside the root, in 32-bit with one rounding. One block per row.
// ---------------------------------------------------------------------------------------------
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
pair_norm_mean_kernel(const T* a, int64_t a_stride, const T* b, int64_t b_stride, const float* __restrict__ wa,
                      const float* __restrict__ wb, float eps, float coef, T* out, int width) {
    constexpr int ITEMS = 2;                              // steps of four elements that stay in registers
    __shared__ float red[66];
    pdl_launch_dependents();
    pdl_wait();
    const size_t r = blockIdx.x;
    const T* pa = a + r * a_stride;
    const T* pb = b + r * b_stride;
    float2 ss = make_float2(0.f, 0.f);
    if constexpr (VEC) {
        auto square = [](float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
        float4 va[ITEMS], vb[ITEMS];
#pragma unroll
        for (int k = 0; k < ITEMS; ++k) {
            const int i = (threadIdx.x + k * blockDim.x) * 4;
            va[k] = i < width ? Quad<T>::load(pa + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            vb[k] = i < width ? Quad<T>::load(pb + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int k = 0; k < ITEMS; ++k) {
            ss.x += square(va[k]);
            ss.y += square(vb[k]);
        }
        for (int i = (threadIdx.x + ITEMS * blockDim.x) * 4; i < width; i += blockDim.x * 4) {
            ss.x += square(Quad<T>::load(pa + i));
            ss.y += square(Quad<T>::load(pb + i));
        }
        ss = block_sum2(ss, red);
        const float ra = coef / sqrtf(ss.x / (float)width + eps), rb = coef / sqrtf(ss.y / (float)width + eps);
        auto join = [&](float4 x, float4 y, int i) {
            const float4 p = *reinterpret_cast<const float4*>(wa + i), q = *reinterpret_cast<const float4*>(wb + i);
            Quad<T>::store(out + r * width + i,
                           make_float4(x.x * ra * p.x + y.x * rb * q.x, x.y * ra * p.y + y.y * rb * q.y,
                                       x.z * ra * p.z + y.z * rb * q.z, x.w * ra * p.w + y.w * rb * q.w));
        };
#pragma unroll
        for (int k = 0; k < ITEMS; ++k) {
            const int i = (threadIdx.x + k * blockDim.x) * 4;
            if (i < width) join(va[k], vb[k], i);
        }
        for (int i = (threadIdx.x + ITEMS * blockDim.x) * 4; i < width; i += blockDim.x * 4)
            join(Quad<T>::load(pa + i), Quad<T>::load(pb + i), i);
    } else {
        for (int i = threadIdx.x; i < width; i += blockDim.x) {
            const float x = to_f<T>(pa[i]), y = to_f<T>(pb[i]);
            ss.x = fmaf(x, x, ss.x);
            ss.y = fmaf(y, y, ss.y);
        }
        ss = block_sum2(ss, red);
        const float ra = coef / sqrtf(ss.x / (float)width + eps), rb = coef / sqrtf(ss.y / (float)width + eps);
        for (int i = threadIdx.x; i < width; i += blockDim.x)
            out[r * width + i] = from_f<T>(to_f<T>(pa[i]) * ra * wa[i] + to_f<T>(pb[i]) * rb * wb[i]);
    }
}

// a, b: [rows, width] (type dtype) rows `a_stride` / `b_stride` apart; wa, wb: float32 [width]; out: [rows, width].
TK_API int tk_pair_norm_mean(const void* a, int64_t a_stride, const void* b, int64_t b_stride, const float* wa,
                             const float* wb, float eps, float coef, void* out, int rows, int width, int dtype,
                             cudaStream_t stream) {
    TK_CHECK_ARG(rows >= 0 && width > 0, "pair_norm_mean: bad sizes rows=%d width=%d", rows, width);
    if (rows == 0) return 0;
    const int threads = width >= 1024 ? 256 : 128, es = dtype == TK_BF16 ? 2 : 4;
    const bool vec = width % 4 == 0 && a_stride % 4 == 0 && b_stride % 4 == 0 && (((uintptr_t)wa | (uintptr_t)wb) & 15) == 0 &&
                     (((uintptr_t)a | (uintptr_t)b | (uintptr_t)out) & (4 * es - 1)) == 0;
#define TK_PM(TT, VEC)                                                                                              \
    tk_launch(pair_norm_mean_kernel<TT, VEC>, dim3(rows), dim3(threads), 0, stream, (const TT*)a, a_stride, (const TT*)b, \
              b_stride, wa, wb, eps, coef, (TT*)out, width)
    if (dtype == TK_F32) {
        if (vec) TK_PM(float, true);
        else TK_PM(float, false);
    } else if (dtype == TK_BF16) {
        if (vec) TK_PM(__nv_bfloat16, true);
        else TK_PM(__nv_bfloat16, false);
    } else
        TK_CHECK_ARG(false, "pair_norm_mean: unknown dtype %d", dtype);
#undef TK_PM
    TK_CHECK_LAUNCH("pair_norm_mean");
    return 0;
}
