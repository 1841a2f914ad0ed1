// Linear recurrences with a state matrix S [d key rows, e value columns] per head, 32-bit throughout:
//
// * the gated delta rule with a decay per key channel (DELTA):
//     S <- diag(g_t) S,   u_t = b_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t
//   with unit keys and queries and g_t = exp(-exp(A) softplus(z_t + bias)) made here;
// * linear attention with a constant decay per head: S <- decay S + k_t v_t^T, o_t = S^T q_t.
//
// Prompt portions go in chunks of 16 tokens (RC).  With G_t = g_1 .. g_t (row-wise products from the chunk's
// start) and S_0 the state before the chunk, the u_t of a chunk solve a lower triangular system,
//     u_t + b_t sum_{s<t} A_ts u_s = b_t (v_t - (G_t k_t)^T S_0),   A_ts = sum_c k_t[c] k_s[c] (g_{s+1} .. g_t)[c],
// so that with M = (I + diag(b) A)^-1 diag(b)
//     U = M (V - (G k) S_0),   o_t = (G_t q_t)^T S_0 + sum_{s<=t} B_ts u_s,   B_ts as A_ts with q_t for k_t,
//     S_end = diag(G_end) S_0 + sum_s (g_{s+1} .. g_end k_s) u_s^T.
// All decays appear as products of factors from 0 to 1 (no quotients), so nothing overflows however strong
// they are.  Without the delta rule U = V.  A first kernel makes, for every chunk and head at once, the rows
// G k, G q, g_{s+1..end} k, the row G_end and the matrices M and B; a second kernel walks over a sequence's
// chunks with a piece of S (all d rows of COLS columns) in registers.  A chunk that is not full has zero
// rows for the tokens it lacks.
//
// Few tokens a sequence (decode steps) run token by token in a kernel of their own.
#define CHIBI_UNIT linear_recurrence
#define CHIBI_UNIT_ID 14
#include "common.cuh"

namespace chibi {

constexpr int RC = 16;                                  // tokens of a chunk

// Threads that share the inner products of the chunk kernel's first phase, and the pitch of a row of d
// padded to DP: rows that a quarter of a warp reads together start on other banks.
__host__ __device__ constexpr int rc_split(int DP, bool delta) { return delta ? DP / 32 : DP / 16; }
__host__ __device__ constexpr int rc_pitch(int DP, bool delta)
{
    return DP + (rc_split(DP, delta) < 8 ? 4 * rc_split(DP, delta) : 4);
}
// A chunk's block in the scratch array, in floats: KE [RC][pitch] | QT [RC][pitch] | GE [DP] | B [RC][RC] and,
// with the delta rule, | KT [RC][pitch] | M [RC][RC].
__host__ __device__ constexpr int rc_block(int DP, bool delta)
{
    return (delta ? 3 : 2) * RC * rc_pitch(DP, delta) + DP + (delta ? 2 : 1) * RC * RC;
}

__device__ __forceinline__ float lr_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float lr_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

struct RecurrenceParams {
    const void* q;             // [T, stride]: q of qk_heads * d columns
    const void* k;
    const void* v;             // heads * e columns
    long long stride;          // of q, k and v
    int activate;              // q, k and v are raw: silu comes first
    // delta rule
    const float* logits;       // [T, logit_stride]: z, heads * d columns
    long long logit_stride;
    const void* beta;          // [T, beta_stride]: heads columns
    long long beta_stride;
    const float* a_log;        // [heads]
    const float* dt_bias;      // [heads * d]
    float key_eps, q_scale;
    // linear attention
    const float* decay;        // [heads]
    float* state;              // [slots, heads, d, e]
    float* o;                  // [T, heads * e]
    float* scratch;
    const int* q_start;
    const int* slots;
    int heads, qk_heads, d, e;
};

// ---------------------------------------------------------------- per chunk and head: what the chunk kernel needs
// grid (chunks, heads, sequences), eight warps.  For a source token s a lane holds, for its channels, the
// key times the decays since then, and walks over the later tokens t: its parts of A_ts and B_ts for all t
// are folded over the lanes at once.
template <int DP, bool DELTA, typename TX>
__global__ void __launch_bounds__(256)
recurrence_prepare_kernel(const RecurrenceParams p)
{
    pdl_enter();
    constexpr int P = rc_pitch(DP, DELTA), R = DP / 32;
    extern __shared__ __align__(16) float sm[];
    float* ks = sm;                                     // [RC][DP]
    float* qs = ks + RC * DP;
    float* gs = qs + RC * DP;                           // [RC][DP] (delta rule)
    __shared__ float As[RC][RC + 1];
    __shared__ float Bs[RC][RC + 1];
    __shared__ float bs[RC];
    const int h = blockIdx.y, seq = blockIdx.z;
    const int row0 = p.q_start[seq];
    const int base = blockIdx.x * RC;
    const int n = min(RC, p.q_start[seq + 1] - row0 - base);
    if (n <= 0)
        return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int d = p.d, kh = h / (p.heads / p.qk_heads);
    const TX* q = static_cast<const TX*>(p.q) + (size_t)(row0 + base) * p.stride + kh * d;
    const TX* k = static_cast<const TX*>(p.k) + (size_t)(row0 + base) * p.stride + kh * d;
    float* out = p.scratch + ((size_t)((row0 / RC) + seq + blockIdx.x) * p.heads + h) * rc_block(DP, DELTA);
    float* KE = out;
    float* QT = KE + RC * P;
    float* GE = QT + RC * P;
    float* Bo = GE + DP;
    float* KT = Bo + RC * RC;
    float* Mo = KT + RC * P;
    const float rate = DELTA ? -expf(p.a_log[h]) : 0.f;
    const float decay = DELTA ? 1.f : p.decay[h];

    for (int i = tid; i < RC * DP; i += 256) {
        const int t = i / DP, c = i - t * DP;
        float kv = 0.f, qv = 0.f, g = 1.f;
        if (t < n && c < d) {
            kv = to_f32(k[(size_t)t * p.stride + c]);
            qv = to_f32(q[(size_t)t * p.stride + c]);
            if (p.activate)
                kv = lr_silu(kv), qv = lr_silu(qv);
            if (DELTA)
                g = expf(rate * lr_softplus(p.logits[(size_t)(row0 + base + t) * p.logit_stride + h * d + c]
                                            + p.dt_bias[h * d + c]));
        }
        ks[i] = kv;
        qs[i] = qv;
        if (DELTA)
            gs[i] = g;
    }
    if (DELTA && tid < RC)
        bs[tid] = tid < n ? 1.f / (1.f + expf(-to_f32(static_cast<const TX*>(p.beta)[(size_t)(row0 + base + tid)
                                                                                    * p.beta_stride + h]))) : 0.f;
    __syncthreads();
    if (DELTA) {                                        // unit keys and queries: two tokens to a warp
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int t = warp + 8 * u;
            float sk = 0.f, sq = 0.f;
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const float a = ks[t * DP + lane + 32 * i], b = qs[t * DP + lane + 32 * i];
                sk = fmaf(a, a, sk);
                sq = fmaf(b, b, sq);
            }
            const float ik = 1.f / sqrtf(warp_sum(sk) + p.key_eps);
            const float iq = p.q_scale / sqrtf(warp_sum(sq) + p.key_eps);
#pragma unroll
            for (int i = 0; i < R; ++i) {
                ks[t * DP + lane + 32 * i] *= ik;
                qs[t * DP + lane + 32 * i] *= iq;
            }
        }
        __syncthreads();
    }
    // decays from the chunk's start, a thread to a channel
    for (int c = tid; c < DP; c += 256) {
        float g = 1.f;
#pragma unroll
        for (int t = 0; t < RC; ++t) {
            g *= DELTA ? gs[t * DP + c] : (t < n ? decay : 1.f);
            QT[t * P + c] = qs[t * DP + c] * g;
            if (DELTA)
                KT[t * P + c] = ks[t * DP + c] * g;
        }
        GE[c] = g;
    }
    // a warp takes the source tokens `warp` and 15 - `warp`
#pragma unroll 1
    for (int u = 0; u < 2; ++u) {
        const int s = u ? RC - 1 - warp : warp;
        float w[R], acc[2 * RC];                        // [t]: B_ts, A_ts
#pragma unroll
        for (int i = 0; i < R; ++i)
            w[i] = ks[s * DP + lane + 32 * i];
#pragma unroll
        for (int t = 0; t < RC; ++t) {
            float b = 0.f, a = 0.f;
            if (t >= s) {
#pragma unroll
                for (int i = 0; i < R; ++i) {
                    const int c = t * DP + lane + 32 * i;
                    if (t > s)
                        w[i] *= DELTA ? gs[c] : (t < n ? decay : 1.f);
                    b = fmaf(qs[c], w[i], b);
                    if (DELTA)
                        a = fmaf(ks[c], w[i], a);
                }
            }
            acc[t] = b;
            acc[RC + t] = a;
        }
#pragma unroll
        for (int i = 0; i < R; ++i)
            KE[s * P + lane + 32 * i] = w[i];
        // fold: after the steps 16, 8, 4, 2, 1 lane l holds the sum over all lanes of value l
#pragma unroll
        for (int half = RC, o = 16; half >= 1; half >>= 1, o >>= 1) {
            const bool upper = (lane & o) != 0;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float send = upper ? acc[i] : acc[i + half];
                const float keep = upper ? acc[i + half] : acc[i];
                acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        }
        if (lane < RC)
            Bs[lane][s] = acc[0];
        else
            As[lane - RC][s] = acc[0];
    }
    __syncthreads();
    Bo[tid] = Bs[tid / RC][tid % RC];                   // (256 threads, 16 x 16 values)
    if (DELTA && tid < RC) {
        // column tid of M: forward substitution
        float m[RC];
#pragma unroll
        for (int t = 0; t < RC; ++t) {
            float v = t == tid ? 1.f : 0.f;
#pragma unroll
            for (int s = 0; s < t; ++s)
                v = fmaf(-As[t][s], m[s], v);
            m[t] = bs[t] * v;
            Mo[t * RC + tid] = m[t];
        }
    }
}

// ---------------------------------------------------------------- over a sequence's chunks
__device__ __forceinline__ void rc_copy16(float* dst, const float* src)
{
    const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(src) : "memory");
}

// grid (blocks of COLS value columns, heads, sequences), DP * COLS / 16 threads.  A thread owns 4 x 4 elements
// of S (rows r0 .., columns c0 ..) in registers; a copy lies in shared memory, column by column, for the
// first phase, in which KS neighbouring threads share a tile of 4 tokens x 4 columns of (G k) S_0 or (G q) S_0
// (each its part of the d rows) and fold their sums.
template <int DP, int COLS, bool DELTA, typename TX>
__global__ void __launch_bounds__(DP * COLS / 16)
chunk_recurrence_kernel(const RecurrenceParams p)
{
    constexpr int NT = DP * COLS / 16, P = rc_pitch(DP, DELTA), KS = rc_split(DP, DELTA), BLOCK = rc_block(DP, DELTA);
    constexpr int CP = COLS + 4;                        // pitch of the chunk's small arrays
    constexpr int CG = COLS / 4;                        // groups of four columns
    constexpr int OWN = 16 / KS;                        // sums a thread is left with after the fold
    static_assert(NT % 32 == 0 && KS >= 1 && KS <= 16 && DP % (4 * KS) == 0, "sizes");
#ifdef CHIBI_TIMELINE
    pdl_enter();
#endif
    extern __shared__ __align__(16) float sm[];
    float* bufs = sm;                                   // two chunks
    float* Sc = bufs + 2 * BLOCK;                       // [COLS][P]
    float* Us = Sc + COLS * P;                          // [RC][CP]
    float* Os = Us + RC * CP;                           // [RC][CP]
    float* Rs = Os + RC * CP;                           // [RC][CP] (delta rule)
    const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
    const int d = p.d, e = p.e;
    const int col0 = blockIdx.x * COLS;
    const int row0 = p.q_start[seq];
    const int len = p.q_start[seq + 1] - row0;
    if (len <= 0)
        return;
    const int r0 = 4 * (tid % (DP / 4)), c0 = 4 * (tid / (DP / 4));
    float* st = p.state + ((size_t)p.slots[seq] * p.heads + h) * d * e;
    float S[4][4];                                      // [column][row]
    // (the state is what an earlier step left: fetched before the kernel ahead is through)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            S[j][i] = (r0 + i < d && col0 + c0 + j < e) ? st[(size_t)(r0 + i) * e + col0 + c0 + j] : 0.f;
#ifndef CHIBI_TIMELINE
    pdl_wait();
#endif
    // the tile of the first phase, and the sums of it that this thread is left with
    const int ks = tid % KS, tile = tid / KS;
    const int tg = tile & 3, cg = (tile >> 2) % CG;
    const bool keys = DELTA && tile >= 4 * CG;          // this thread works on (G k) S_0, else on (G q) S_0
    const int first = ks * OWN;                         // values first .. first + OWN - 1 of the tile's 16 (token-major)
    const TX* v = static_cast<const TX*>(p.v) + (size_t)row0 * p.stride + (size_t)h * e + col0;
    const bool takes_v = !DELTA || keys;
    float vn[OWN];
    auto fetch_v = [&](int base) {
#pragma unroll
        for (int m = 0; m < OWN; ++m) {
            const int t = tg + 4 * ((first + m) >> 2), c = cg + CG * ((first + m) & 3);
            vn[m] = 0.f;
            if (takes_v && base + t < len && col0 + c < e) {
                vn[m] = to_f32(v[(size_t)(base + t) * p.stride + c]);
                if (p.activate)
                    vn[m] = lr_silu(vn[m]);
            }
        }
    };
    const float* chunk_src = p.scratch + ((size_t)(row0 / RC + seq) * p.heads + h) * BLOCK;
    auto fetch = [&](int c, float* dst) {
        const float* src = chunk_src + (size_t)c * p.heads * BLOCK;
        for (int i = 4 * tid; i < BLOCK; i += 4 * NT)
            rc_copy16(dst + i, src + i);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, bufs);
    fetch_v(0);
#pragma unroll
    for (int j = 0; j < 4; ++j)
        *reinterpret_cast<float4*>(Sc + (c0 + j) * P + r0) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);

    const int chunks = (len + RC - 1) / RC;
    for (int c = 0; c < chunks; ++c) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                // the chunk is there; everyone is through with the last one
        if (c + 1 < chunks)
            fetch(c + 1, bufs + ((c + 1) & 1) * BLOCK);
        const float* KE = bufs + (c & 1) * BLOCK;
        const float* QT = KE + RC * P;
        const float* GE = QT + RC * P;
        const float* B = GE + DP;
        const float* KT = B + RC * RC;
        const float* M = KT + RC * P;
        const int base = c * RC;
        float v_now[OWN];
#pragma unroll
        for (int m = 0; m < OWN; ++m)
            v_now[m] = vn[m];
        if (c + 1 < chunks)
            fetch_v(base + RC);
        // ---- (G q) S_0 and (G k) S_0
        {
            float acc[16];
#pragma unroll
            for (int i = 0; i < 16; ++i)
                acc[i] = 0.f;
            const float* a_rows = (keys ? KT : QT) + tg * P + 4 * ks;
            const float* b_rows = Sc + cg * P + 4 * ks;
#pragma unroll 4
            for (int k4 = 0; k4 < DP / (4 * KS); ++k4) {
                float4 a[4], b[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    a[i] = *reinterpret_cast<const float4*>(a_rows + 4 * i * P + 4 * KS * k4);
                    b[i] = *reinterpret_cast<const float4*>(b_rows + CG * i * P + 4 * KS * k4);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        float s = acc[4 * i + j];
                        s = fmaf(a[i].x, b[j].x, s);
                        s = fmaf(a[i].y, b[j].y, s);
                        s = fmaf(a[i].z, b[j].z, s);
                        acc[4 * i + j] = fmaf(a[i].w, b[j].w, s);
                    }
            }
#pragma unroll
            for (int o = KS / 2, half = 8; o >= 1; o >>= 1, half >>= 1) {
                const bool upper = (ks & o) != 0;
#pragma unroll
                for (int i = 0; i < half; ++i) {
                    const float send = upper ? acc[i] : acc[i + half];
                    const float keep = upper ? acc[i + half] : acc[i];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
#pragma unroll
            for (int m = 0; m < OWN; ++m) {
                const int t = tg + 4 * ((first + m) >> 2), cc = cg + CG * ((first + m) & 3);
                if (keys) {
                    Rs[t * CP + cc] = v_now[m] - acc[m];
                } else {
                    Os[t * CP + cc] = acc[m];
                    if (!DELTA)
                        Us[t * CP + cc] = v_now[m];
                }
            }
        }
        __syncthreads();
        // ---- U = M R, four columns of a token to a thread
        if (DELTA) {
            for (int i = tid; i < RC * CG; i += NT) {
                const int t = i / CG, cc = 4 * (i - t * CG);
                float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int s = 0; s < RC; ++s) {
                    const float m = M[t * RC + s];
                    const float4 r = *reinterpret_cast<const float4*>(Rs + s * CP + cc);
                    u.x = fmaf(m, r.x, u.x), u.y = fmaf(m, r.y, u.y), u.z = fmaf(m, r.z, u.z), u.w = fmaf(m, r.w, u.w);
                }
                *reinterpret_cast<float4*>(Us + t * CP + cc) = u;
            }
            __syncthreads();
        }
        // ---- o = (G q) S_0 + B U
        for (int i = NT - 1 - tid; i < RC * CG; i += NT) {
            const int t = i / CG, cc = 4 * (i - t * CG);
            if (base + t >= len)
                continue;
            float4 u = *reinterpret_cast<const float4*>(Os + t * CP + cc);
#pragma unroll
            for (int s = 0; s < RC; ++s) {
                const float m = B[t * RC + s];
                const float4 r = *reinterpret_cast<const float4*>(Us + s * CP + cc);
                u.x = fmaf(m, r.x, u.x), u.y = fmaf(m, r.y, u.y), u.z = fmaf(m, r.z, u.z), u.w = fmaf(m, r.w, u.w);
            }
            float* dst = p.o + (size_t)(row0 + base + t) * p.heads * e + (size_t)h * e + col0 + cc;
            const float out[4] = { u.x, u.y, u.z, u.w };
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (col0 + cc + j < e)
                    dst[j] = out[j];
        }
        // ---- S = diag(G_end) S_0 + KE^T U
        {
            const float4 g = *reinterpret_cast<const float4*>(GE + r0);
#pragma unroll
            for (int j = 0; j < 4; ++j)
                S[j][0] *= g.x, S[j][1] *= g.y, S[j][2] *= g.z, S[j][3] *= g.w;
#pragma unroll
            for (int s = 0; s < RC; ++s) {
                const float4 k = *reinterpret_cast<const float4*>(KE + s * P + r0);
                const float4 u4 = *reinterpret_cast<const float4*>(Us + s * CP + c0);
                const float u[4] = { u4.x, u4.y, u4.z, u4.w };
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    S[j][0] = fmaf(k.x, u[j], S[j][0]);
                    S[j][1] = fmaf(k.y, u[j], S[j][1]);
                    S[j][2] = fmaf(k.z, u[j], S[j][2]);
                    S[j][3] = fmaf(k.w, u[j], S[j][3]);
                }
            }
            // (nobody reads the copy between the first phase's barrier and the next chunk's)
#pragma unroll
            for (int j = 0; j < 4; ++j)
                *reinterpret_cast<float4*>(Sc + (c0 + j) * P + r0) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (r0 + i < d && col0 + c0 + j < e)
                st[(size_t)(r0 + i) * e + col0 + c0 + j] = S[j][i];
}

// ---------------------------------------------------------------- few tokens a sequence
// grid (blocks of 32 value columns, heads, sequences), W warps: lane = column, a warp owns R key rows in
// registers.  Per token a warp makes its rows' key, query and decay, the block adds up what the warps find in
// the old state, and one barrier later everyone knows u: with S' = diag(g) S,
// o = S'^T q + (k . q) u, so the read-out needs no second barrier.
template <int W, int R, bool DELTA, typename TX>
__global__ void __launch_bounds__(32 * W)
recurrence_tokens_kernel(const RecurrenceParams p)
{
#ifdef CHIBI_TIMELINE
    pdl_enter();
#else
    pdl_trigger();
#endif
    __shared__ float part[2][3][W][32];                 // [turn]: S'^T k, S'^T q, and k . q of the warp's rows
    __shared__ float vec[W][3][R];                      // the warp's k, q, g
    const int h = blockIdx.y, seq = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int d = p.d, e = p.e, kh = h / (p.heads / p.qk_heads);
    const int row0 = p.q_start[seq];
    const int len = p.q_start[seq + 1] - row0;
    if (len <= 0)
        return;
    const int col = blockIdx.x * 32 + lane, r0 = warp * R;
    float* st = p.state + ((size_t)p.slots[seq] * p.heads + h) * d * e;
    float S[R];
    // (the state is what an earlier step left: fetched before the kernel ahead is through)
#pragma unroll
    for (int i = 0; i < R; ++i)
        S[i] = (col < e && r0 + i < d) ? st[(size_t)(r0 + i) * e + col] : 0.f;
    const float rate = DELTA ? -expf(p.a_log[h]) : 0.f;
    const float decay = DELTA ? 1.f : p.decay[h];
#ifndef CHIBI_TIMELINE
    pdl_wait();
#endif
    for (int t = 0; t < len; ++t) {
        const size_t row = (size_t)(row0 + t);
        const TX* q = static_cast<const TX*>(p.q) + row * p.stride + kh * d;
        const TX* k = static_cast<const TX*>(p.k) + row * p.stride + kh * d;
        float v = col < e ? to_f32(static_cast<const TX*>(p.v)[row * p.stride + (size_t)h * e + col]) : 0.f;
        if (p.activate)
            v = lr_silu(v);
        float beta = 1.f, ik = 1.f, iq = 1.f;
        if (DELTA) {
            beta = 1.f / (1.f + expf(-to_f32(static_cast<const TX*>(p.beta)[row * p.beta_stride + h])));
            float sk = 0.f, sq = 0.f;
            for (int c = lane; c < d; c += 32) {
                const float a = to_f32(k[c]), b = to_f32(q[c]);
                sk = fmaf(a, a, sk);
                sq = fmaf(b, b, sq);
            }
            ik = 1.f / sqrtf(warp_sum(sk) + p.key_eps);
            iq = p.q_scale / sqrtf(warp_sum(sq) + p.key_eps);
        }
        __syncwarp();
        for (int i = lane; i < R; i += 32) {
            const int c = r0 + i;
            float kv = 0.f, qv = 0.f, g = 0.f;
            if (c < d) {
                kv = to_f32(k[c]);
                qv = to_f32(q[c]);
                if (p.activate)
                    kv = lr_silu(kv), qv = lr_silu(qv);
                kv *= ik;
                qv *= iq;
                g = DELTA ? expf(rate * lr_softplus(p.logits[row * p.logit_stride + h * d + c] + p.dt_bias[h * d + c])) : decay;
            }
            vec[warp][0][i] = kv;
            vec[warp][1][i] = qv;
            vec[warp][2][i] = g;
        }
        __syncwarp();
        float sk = 0.f, sq = 0.f, kq = 0.f;
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const float kv = vec[warp][0][i], qv = vec[warp][1][i];
            S[i] *= vec[warp][2][i];
            if (DELTA)
                sk = fmaf(S[i], kv, sk);
            sq = fmaf(S[i], qv, sq);
            kq = fmaf(kv, qv, kq);
        }
        const int turn = t & 1;
        if (DELTA)
            part[turn][0][warp][lane] = sk;
        part[turn][1][warp][lane] = sq;
        part[turn][2][warp][lane] = kq;
        __syncthreads();
        sk = sq = kq = 0.f;
#pragma unroll
        for (int w = 0; w < W; ++w) {
            if (DELTA)
                sk += part[turn][0][w][lane];
            sq += part[turn][1][w][lane];
            kq += part[turn][2][w][lane];
        }
        const float u = DELTA ? beta * (v - sk) : v;
#pragma unroll
        for (int i = 0; i < R; ++i)
            S[i] = fmaf(vec[warp][0][i], u, S[i]);
        if (warp == 0 && col < e)
            p.o[row * p.heads * e + (size_t)h * e + col] = fmaf(kq, u, sq);
    }
#pragma unroll
    for (int i = 0; i < R; ++i)
        if (col < e && r0 + i < d)
            st[(size_t)(r0 + i) * e + col] = S[i];
}

// ---------------------------------------------------------------- launches
static inline int padded_rows(int d) { return d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : d <= 256 ? 256 : 0; }

static inline int recurrence_sm_count()
{
    static int sms = 0;
    if (sms == 0) {
        int dev = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    }
    return sms;
}

template <int DP, int COLS, bool DELTA, typename TX>
static void launch_chunks(const RecurrenceParams& p, int seqs, cudaStream_t stream)
{
    const size_t smem = (size_t)(2 * rc_block(DP, DELTA) + COLS * rc_pitch(DP, DELTA) + 3 * RC * (COLS + 4)) * sizeof(float);
    auto kernel = chunk_recurrence_kernel<DP, COLS, DELTA, TX>;
    if (smem > 48 * 1024)
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch(kernel, dim3((unsigned)((p.e + COLS - 1) / COLS), (unsigned)p.heads, (unsigned)seqs), dim3(DP * COLS / 16), smem,
           stream, p);
}

template <int DP, bool DELTA, typename TX>
static void launch_prompt(const RecurrenceParams& p, int seqs, int max_q_len, cudaStream_t stream)
{
    const size_t smem = (size_t)(DELTA ? 3 : 2) * RC * DP * sizeof(float);
    auto prepare = recurrence_prepare_kernel<DP, DELTA, TX>;
    if (smem > 44 * 1024)
        cudaFuncSetAttribute(prepare, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch(prepare, dim3((unsigned)((max_q_len + RC - 1) / RC), (unsigned)p.heads, (unsigned)seqs), dim3(256), smem, stream, p);
    // blocks of 32 columns where they give two SMs of three one, else of 16 (the work of a thread is the same)
    if ((long long)((p.e + 31) / 32) * p.heads * seqs * 3 >= 2 * recurrence_sm_count())
        launch_chunks<DP, 32, DELTA, TX>(p, seqs, stream);
    else
        launch_chunks<DP, 16, DELTA, TX>(p, seqs, stream);
}

template <bool DELTA, typename TX>
static void launch_tokens(const RecurrenceParams& p, int seqs, cudaStream_t stream)
{
    const dim3 grid((unsigned)((p.e + 31) / 32), (unsigned)p.heads, (unsigned)seqs);
    if (p.d <= 32)
        launch(recurrence_tokens_kernel<8, 4, DELTA, TX>, grid, dim3(256), 0, stream, p);
    else if (p.d <= 64)
        launch(recurrence_tokens_kernel<8, 8, DELTA, TX>, grid, dim3(256), 0, stream, p);
    else if (p.d <= 128)
        launch(recurrence_tokens_kernel<8, 16, DELTA, TX>, grid, dim3(256), 0, stream, p);
    else if (p.d <= 256)
        launch(recurrence_tokens_kernel<16, 16, DELTA, TX>, grid, dim3(512), 0, stream, p);
    else
        launch(recurrence_tokens_kernel<16, 32, DELTA, TX>, grid, dim3(512), 0, stream, p);
}

template <bool DELTA>
static int launch_recurrence(const RecurrenceParams& p, int x_type, long long scratch_floats, long long tokens, int seqs,
                             int max_q_len, int few, cudaStream_t stream)
{
    if (p.d > 512 || p.heads > 65535 || seqs > 65535)
        return CHIBI_ERR_UNSUPPORTED;
    const int DP = padded_rows(p.d);
    if (max_q_len <= few || DP == 0) {
        CHIBI_DISPATCH_TYPE(x_type, TX, { launch_tokens<DELTA, TX>(p, seqs, stream); });
        return launch_status();
    }
    if (!p.scratch || (reinterpret_cast<uintptr_t>(p.scratch) & 15)
        || scratch_floats < (tokens / RC + seqs) * (long long)p.heads * rc_block(DP, DELTA))
        return CHIBI_ERR_ARGUMENT;
    CHIBI_DISPATCH_TYPE(x_type, TX, {
        if (DP == 32)
            launch_prompt<32, DELTA, TX>(p, seqs, max_q_len, stream);
        else if (DP == 64)
            launch_prompt<64, DELTA, TX>(p, seqs, max_q_len, stream);
        else if (DP == 128)
            launch_prompt<128, DELTA, TX>(p, seqs, max_q_len, stream);
        else
            launch_prompt<256, DELTA, TX>(p, seqs, max_q_len, stream);
    });
    return launch_status();
}

} // namespace chibi

using namespace chibi;

// Floats of scratch that a step of so many tokens and sequences needs where a sequence brings more tokens
// than the token-by-token kernel is used for; a sequence's chunks start at slot q_start / 16 + sequence.
CHIBI_API int chibi_recurrence_scratch(long long tokens, int seqs, int heads, int d, int delta, long long* floats)
{
    const int DP = padded_rows(d);
    if (!floats || tokens < 0 || seqs < 0 || heads <= 0 || d <= 0)
        return CHIBI_ERR_ARGUMENT;
    *floats = DP == 0 ? 0 : (tokens / RC + seqs) * (long long)heads * rc_block(DP, delta != 0);
    return CHIBI_OK;
}

// q | k | v of a row lie side by side: qk_heads * d, qk_heads * d, heads * e columns.  `few`: steps whose
// sequences bring at most so many tokens run token by token.
CHIBI_API int chibi_channel_delta(const void* qkv, int x_type, long long stride, const float* logits,
                                  long long logit_stride, const void* beta, long long beta_stride, const float* a_log,
                                  const float* dt_bias, float* state, float* o, float* scratch, long long scratch_floats,
                                  const int* q_start, const int* slots, long long tokens, int seqs, int max_q_len,
                                  int heads, int qk_heads, int d, int e, float key_eps, float q_scale, int few,
                                  cudaStream_t stream)
{
    if (seqs <= 0 || tokens <= 0 || max_q_len <= 0)
        return CHIBI_OK;
    if (!qkv || !logits || !beta || !a_log || !dt_bias || !state || !o || heads <= 0 || qk_heads <= 0
        || heads % qk_heads != 0 || d <= 0 || e <= 0)
        return CHIBI_ERR_ARGUMENT;
    const int size = x_type == CHIBI_BF16 ? 2 : 4;
    RecurrenceParams p = {};
    p.q = qkv;
    p.k = static_cast<const char*>(qkv) + (size_t)qk_heads * d * size;
    p.v = static_cast<const char*>(qkv) + (size_t)2 * qk_heads * d * size;
    p.stride = stride;
    p.logits = logits;
    p.logit_stride = logit_stride;
    p.beta = beta;
    p.beta_stride = beta_stride;
    p.a_log = a_log;
    p.dt_bias = dt_bias;
    p.key_eps = key_eps;
    p.q_scale = q_scale;
    p.state = state;
    p.o = o;
    p.scratch = scratch;
    p.q_start = q_start;
    p.slots = slots;
    p.heads = heads;
    p.qk_heads = qk_heads;
    p.d = d;
    p.e = e;
    return launch_recurrence<true>(p, x_type, scratch_floats, tokens, seqs, max_q_len, few, stream);
}

CHIBI_API int chibi_decayed_attention(const void* qkv, int x_type, long long stride, int activate, const float* decay,
                                      float* state, float* o, float* scratch, long long scratch_floats,
                                      const int* q_start, const int* slots, long long tokens, int seqs, int max_q_len,
                                      int heads, int d, int e, int few, cudaStream_t stream)
{
    if (seqs <= 0 || tokens <= 0 || max_q_len <= 0)
        return CHIBI_OK;
    if (!qkv || !decay || !state || !o || heads <= 0 || d <= 0 || e <= 0)
        return CHIBI_ERR_ARGUMENT;
    const int size = x_type == CHIBI_BF16 ? 2 : 4;
    RecurrenceParams p = {};
    p.q = qkv;
    p.k = static_cast<const char*>(qkv) + (size_t)heads * d * size;
    p.v = static_cast<const char*>(qkv) + (size_t)2 * heads * d * size;
    p.stride = stride;
    p.activate = activate;
    p.decay = decay;
    p.state = state;
    p.o = o;
    p.scratch = scratch;
    p.q_start = q_start;
    p.slots = slots;
    p.heads = heads;
    p.qk_heads = heads;
    p.d = d;
    p.e = e;
    return launch_recurrence<false>(p, x_type, scratch_floats, tokens, seqs, max_q_len, few, stream);
}
