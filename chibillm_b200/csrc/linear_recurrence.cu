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
// so that with M = (I + diag(b) A)^-1 diag(b) and B_ts as A_ts with q_t for k_t (s <= t)
//     U = M V - W S_0,               W = M (G k),
//     O = (G q) S_0 + B U = B M V + Q S_0,   Q = (G q) - B W,
//     S_end = diag(G_end) S_0 + sum_s (g_{s+1} .. g_end k_s) u_s^T.
// All decays appear as products of factors from 0 to 1 (no quotients), so nothing overflows however strong
// they are.  Without the delta rule U = V, Q = G q and O = B V + Q S_0.  A first kernel makes, for every chunk
// and head at once, the rows W, Q, g_{s+1..end} k, the row G_end and the matrices M, B M; a second kernel walks
// over a sequence's chunks with a piece of S (all d rows of some columns) in registers: two small products
// with S_0 and V, then one into S.  A chunk that is not full has zero rows for the tokens it lacks.
//
// Few tokens a sequence (decode steps) run token by token in a kernel of their own.
#define CHIBI_UNIT linear_recurrence
#define CHIBI_UNIT_ID 14
#include "common.cuh"

namespace chibi {

constexpr int RC = 16;                                  // tokens of a chunk

// A chunk's block in the scratch array, in floats (d padded to DP): KE [RC][DP] | GE [DP] | Q [RC][DP] |
// B M or B [RC][RC] and, with the delta rule, | -W [RC][DP] | M [RC][RC].
__host__ __device__ constexpr int rc_block(int DP, bool delta)
{
    return (delta ? 3 : 2) * RC * DP + DP + (delta ? 2 : 1) * RC * RC;
}

// silu, and the decay exp(rate * softplus(z)).  Beside bfloat16 activations CUDA's faster exponential and logarithm
// (32-bit too, good to a few units of the last place of their results and to 2^-21 near one) are enough: an
// input's own rounding is ten thousand times larger.
template <typename TX> __device__ __forceinline__ float lr_silu(float z)
{
    if constexpr (sizeof(TX) == 2)
        return __fdividef(z, 1.f + __expf(-z));
    return z / (1.f + expf(-z));
}
template <typename TX> __device__ __forceinline__ float lr_decay(float rate, float z)
{
    if constexpr (sizeof(TX) == 2)
        return __expf(rate * (z > 20.f ? z : __logf(1.f + __expf(z))));
    return expf(rate * (z > 20.f ? z : log1pf(expf(z))));
}

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
// grid (chunks, heads, sequences), eight warps.  The inner products of a chunk's tokens come in tiles of four
// sources s and four targets t, lanes along the channels.  Off the diagonal the sources are decayed to the
// targets' first token and the targets from there, so that a tile is a plain product; on it the sources are
// decayed token by token.  A tile's 32 sums over the lanes are folded together.
template <int DP, bool DELTA, typename TX>
__global__ void __launch_bounds__(256)
recurrence_prepare_kernel(const RecurrenceParams p)
{
    // No trigger here: the chunk kernel's few blocks are to be dealt out to empty SMs, one to each.  Let in while
    // this kernel's last blocks run, they crowd on the SMs that have room (2,048 tokens of 16 heads of 64: 0.18 ms
    // became 0.47).
#ifdef CHIBI_TIMELINE
    pdl_enter();
#else
    pdl_wait();
#endif
    constexpr int R = DP / 32;
    extern __shared__ __align__(16) float sm[];
    float* ks = sm;                                     // [RC][DP]
    float* qs = ks + RC * DP;
    float* gs = qs + RC * DP;                           // [RC][DP] (delta rule)
    float* gg = gs + RC * DP;                           // [4][DP]: the decays' products over four tokens each
    __shared__ __align__(16) float As[RC][RC];
    __shared__ __align__(16) float Bs[RC][RC];
    __shared__ __align__(16) float Ms[RC][RC];
    __shared__ float bs[RC], power[RC + 1];
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
    float* KE = p.scratch + ((size_t)((row0 / RC) + seq + blockIdx.x) * p.heads + h) * rc_block(DP, DELTA);
    float* GE = KE + RC * DP;
    float* Qo = GE + DP;
    float* No = Qo + RC * DP;                           // B M, or B
    float* Wo = No + RC * RC;
    float* Mo = Wo + RC * DP;
    const float rate = DELTA ? -expf(p.a_log[h]) : 0.f;

    // ---- the chunk's keys, queries and decays
    {
        constexpr int PER = RC * DP / 256;              // a thread's values: the channel is the same for all (or two)
        TX kr[PER], qr[PER];
        float zr[PER];
#pragma unroll
        for (int u = 0; u < PER; ++u) {
            const int i = tid + 256 * u, t = i / DP, c = i - t * DP;
            kr[u] = qr[u] = from_f32<TX>(0.f);
            zr[u] = 0.f;
            if (t < n && c < d) {
                kr[u] = k[(size_t)t * p.stride + c];
                qr[u] = q[(size_t)t * p.stride + c];
                if (DELTA)
                    zr[u] = p.logits[(size_t)(row0 + base + t) * p.logit_stride + h * d + c] + p.dt_bias[h * d + c];
            }
        }
#pragma unroll
        for (int u = 0; u < PER; ++u) {
            const int i = tid + 256 * u, t = i / DP, c = i - t * DP;
            float kv = to_f32(kr[u]), qv = to_f32(qr[u]);
            if (p.activate)
                kv = lr_silu<TX>(kv), qv = lr_silu<TX>(qv);     // (silu(0) is 0)
            ks[i] = kv;
            qs[i] = qv;
            if (DELTA)
                gs[i] = t < n && c < d ? lr_decay<TX>(rate, zr[u]) : 1.f;
        }
    }
    if (tid < RC) {
        if (DELTA) {
            bs[tid] = tid < n ? 1.f / (1.f + expf(-to_f32(static_cast<const TX*>(p.beta)[(size_t)(row0 + base + tid)
                                                                                        * p.beta_stride + h]))) : 0.f;
        } else {
            float v = 1.f;
            for (int i = 0; i < tid; ++i)
                v *= p.decay[h];
            power[tid] = v;
            if (tid == RC - 1)
                power[RC] = v * p.decay[h];
        }
    }
    if (tid < RC * RC / 4) {                            // (what lies above the diagonal)
        reinterpret_cast<float4*>(&As[0][0])[tid] = make_float4(0.f, 0.f, 0.f, 0.f);
        reinterpret_cast<float4*>(&Bs[0][0])[tid] = make_float4(0.f, 0.f, 0.f, 0.f);
        reinterpret_cast<float4*>(&Ms[0][0])[tid] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    __syncthreads();
    if (DELTA) {
        // unit keys and queries: two tokens to a warp
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
        for (int i = tid; i < 4 * DP; i += 256) {
            const int b = i / DP, c = i - b * DP;
            const float* g = gs + 4 * b * DP + c;
            gg[i] = g[0] * g[DP] * (g[2 * DP] * g[3 * DP]);
        }
        __syncthreads();
    }
    // ---- tiles of inner products: (block of targets, block of sources); warps 6 and 7 take two on the diagonal
#pragma unroll 1
    for (int item = warp; item < 10; item = item < 6 ? 10 : item + 2) {
        const int I = item < 6 ? (item == 0 ? 1 : item < 3 ? 2 : 3) : item - 6;
        const int J = item < 6 ? (item == 0 ? 0 : item < 3 ? item - 1 : item - 3) : item - 6;
        float acc[32];                                  // [4 t + s]: A, then B
#pragma unroll
        for (int i = 0; i < 32; ++i)
            acc[i] = 0.f;
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int c = lane + 32 * r;
            float w[4];
#pragma unroll
            for (int s = 0; s < 4; ++s)
                w[s] = ks[(4 * J + s) * DP + c];
            if (!DELTA) {
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    const float qv = qs[(4 * I + t) * DP + c];
#pragma unroll
                    for (int s = 0; s < 4; ++s)
                        acc[16 + 4 * t + s] = fmaf(qv, w[s], acc[16 + 4 * t + s]);
                }
            } else if (item < 6) {
                float f = 1.f;                          // from the end of the sources' block to the targets' first token
                for (int b = J + 1; b < I; ++b)
                    f *= gg[b * DP + c];
#pragma unroll
                for (int s = 3; s >= 0; --s) {
                    w[s] *= f;
                    if (s > 0)
                        f *= gs[(4 * J + s) * DP + c];
                }
                f = 1.f;
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    const int at = (4 * I + t) * DP + c;
                    f *= gs[at];
                    const float kv = ks[at] * f, qv = qs[at] * f;
#pragma unroll
                    for (int s = 0; s < 4; ++s) {
                        acc[4 * t + s] = fmaf(kv, w[s], acc[4 * t + s]);
                        acc[16 + 4 * t + s] = fmaf(qv, w[s], acc[16 + 4 * t + s]);
                    }
                }
            } else {
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    const int at = (4 * I + t) * DP + c;
                    const float kv = ks[at], qv = qs[at], g = gs[at];
#pragma unroll
                    for (int s = 0; s < t; ++s) {
                        w[s] *= g;
                        acc[4 * t + s] = fmaf(kv, w[s], acc[4 * t + s]);
                        acc[16 + 4 * t + s] = fmaf(qv, w[s], acc[16 + 4 * t + s]);
                    }
                    acc[16 + 4 * t + t] = fmaf(qv, w[t], acc[16 + 4 * t + t]);
                }
            }
        }
        // fold: after the steps 16, 8, 4, 2, 1 lane l holds the sum over all lanes of value l
#pragma unroll
        for (int half = 16, o = 16; half >= 1; half >>= 1, o >>= 1) {
            const bool upper = (lane & o) != 0;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float send = upper ? acc[i] : acc[i + half];
                const float keep = upper ? acc[i + half] : acc[i];
                acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        }
        const int t = 4 * I + ((lane >> 2) & 3), s = 4 * J + (lane & 3);
        if (lane < 16) {
            if (DELTA)
                As[t][s] = acc[0];
        } else if (t >= s) {
            Bs[t][s] = DELTA ? acc[0] : acc[0] * power[t - s];
        }
    }
    __syncthreads();
    if (!DELTA) {
        No[tid] = Bs[tid / RC][tid % RC];               // (256 threads, 16 x 16 values)
        for (int c = tid; c < DP; c += 256) {
#pragma unroll
            for (int t = 0; t < RC; ++t) {
                Qo[t * DP + c] = qs[t * DP + c] * power[t + 1];
                KE[t * DP + c] = t < n ? ks[t * DP + c] * power[n - 1 - t] : 0.f;
            }
            GE[c] = power[n];
        }
        return;
    }
    // ---- M: a column to a thread, forward substitution; meanwhile the other warps decay the keys to the chunk's end
    if (tid < RC) {
        float m[RC];
#pragma unroll
        for (int t = 0; t < RC; ++t) {
            float v0 = t == tid ? 1.f : 0.f, v1 = 0.f;
#pragma unroll
            for (int s = 0; s < t; ++s) {
                if (s & 1)
                    v1 = fmaf(-As[t][s], m[s], v1);
                else
                    v0 = fmaf(-As[t][s], m[s], v0);
            }
            m[t] = bs[t] * (v0 + v1);
            Ms[t][tid] = m[t];
        }
    } else if (tid >= 32) {
        for (int c = tid - 32; c < DP; c += 224) {
            float f = 1.f;
#pragma unroll
            for (int t = RC - 1; t >= 0; --t) {
                KE[t * DP + c] = ks[t * DP + c] * f;
                f *= gs[t * DP + c];
            }
            GE[c] = f;
        }
    }
    __syncthreads();
    {
        const int t = tid / RC, j = tid % RC;
        float v = 0.f;
#pragma unroll
        for (int s = 0; s < RC; ++s)
            v = fmaf(Bs[t][s], Ms[s][j], v);
        No[tid] = v;
        Mo[tid] = Ms[t][j];
    }
    // ---- W and Q, a channel to a thread
    for (int c = tid; c < DP; c += 256) {
        float w[RC], g[RC];
        float f = 1.f;
#pragma unroll
        for (int t = 0; t < RC; ++t) {
            f *= gs[t * DP + c];
            g[t] = f;
        }
        {
            float kt[RC];
#pragma unroll
            for (int t = 0; t < RC; ++t) {
                kt[t] = ks[t * DP + c] * g[t];
                float v = 0.f;
#pragma unroll
                for (int s4 = 0; s4 <= t; s4 += 4) {
                    const float4 m = *reinterpret_cast<const float4*>(&Ms[t][s4]);
                    v = fmaf(m.x, kt[s4], v);
                    if (s4 + 1 <= t) v = fmaf(m.y, kt[s4 + 1], v);
                    if (s4 + 2 <= t) v = fmaf(m.z, kt[s4 + 2], v);
                    if (s4 + 3 <= t) v = fmaf(m.w, kt[s4 + 3], v);
                }
                w[t] = v;
                Wo[t * DP + c] = -v;
            }
        }
#pragma unroll
        for (int t = 0; t < RC; ++t) {
            float v = qs[t * DP + c] * g[t];
#pragma unroll
            for (int s4 = 0; s4 <= t; s4 += 4) {
                const float4 m = *reinterpret_cast<const float4*>(&Bs[t][s4]);
                v = fmaf(-m.x, w[s4], v);
                if (s4 + 1 <= t) v = fmaf(-m.y, w[s4 + 1], v);
                if (s4 + 2 <= t) v = fmaf(-m.z, w[s4 + 2], v);
                if (s4 + 3 <= t) v = fmaf(-m.w, w[s4 + 3], v);
            }
            Qo[t * DP + c] = v;
        }
    }
}

// ---------------------------------------------------------------- over a sequence's chunks
__device__ __forceinline__ void rc_copy16(float* dst, const float* src)
{
    const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(src) : "memory");
}

// Two 32-bit values in one 64-bit register, and the multiply-add that takes two such pairs (each half rounded
// like fmaf).
__device__ __forceinline__ uint64_t rc_pair(float a, float b)
{
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 rc_halves(uint64_t v)
{
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ uint64_t rc_fma2(uint64_t a, uint64_t b, uint64_t c)
{
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ uint64_t rc_mul2(uint64_t a, uint64_t b)
{
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// grid (blocks of COLS value columns, heads, sequences).  A thread owns RT rows (runs of four) of CT columns of S
// in registers, two neighbouring rows to a pair, DP / RT threads of a warp lie side by side along the rows, and the
// chunk's rows come from shared memory.  The sums over the rows are spread over those threads and folded at the end of a product, all of its
// values together.  Small pieces of S and many threads: a sequence's chunks come one after the other, so the
// time of a chunk counts, and with a few columns a block every SM has one.
template <int DP, int RT, int CT, int COLS, bool DELTA, typename TX>
__global__ void __launch_bounds__((DP / RT) * (COLS / CT))
chunk_recurrence_kernel(const RecurrenceParams p)
{
    constexpr int L = DP / RT;                          // threads along the rows
    constexpr int NT = L * (COLS / CT), BLOCK = rc_block(DP, DELTA), CP = COLS + 4;
    constexpr int VR = L >= RC ? 1 : RC / L;            // rows of V (tokens) that a thread owns for the products
    constexpr int SUMS = RC * CT, OWN = SUMS / L;       // a product's values, and those that a thread is left with
    constexpr int RUNS = RT / 4, RUN_STEP = DP / RUNS;  // its rows: runs r0 + RUN_STEP i .. + 3
    static_assert(L <= 32 && 32 % L == 0 && NT % 32 == 0 && RT % 4 == 0 && OWN >= 1, "sizes");
#ifdef CHIBI_TIMELINE
    pdl_enter();
#endif
    extern __shared__ __align__(16) float sm[];
    float* bufs = sm;                                   // two chunks
    float* Us = bufs + 2 * BLOCK;                       // [RC][CP]
    const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
    const int d = p.d, e = p.e;
    const int row0 = p.q_start[seq];
    const int len = p.q_start[seq + 1] - row0;
    if (len <= 0)
        return;
    const int lr = tid % L, c0 = CT * (tid / L), r0 = 4 * lr;
    const int col = blockIdx.x * COLS + c0;             // the thread's first column
    float* st = p.state + ((size_t)p.slots[seq] * p.heads + h) * d * e;
    uint64_t S[RT / 2][CT];
    // (the state is what an earlier step left: fetched before the kernel ahead is through)
#pragma unroll
    for (int i = 0; i < RT / 2; ++i) {
        const int r = r0 + RUN_STEP * (i / 2) + 2 * (i % 2);
#pragma unroll
        for (int j = 0; j < CT; ++j)
            S[i][j] = rc_pair((r < d && col + j < e) ? st[(size_t)r * e + col + j] : 0.f,
                              (r + 1 < d && col + j < e) ? st[(size_t)(r + 1) * e + col + j] : 0.f);
    }
#ifndef CHIBI_TIMELINE
    pdl_wait();
#endif
    const TX* v = static_cast<const TX*>(p.v) + (size_t)row0 * p.stride + (size_t)h * e + col;
    TX vn[VR][CT];                                      // on their way: nothing is done with them before their chunk
    auto fetch_v = [&](int base) {
#pragma unroll
        for (int i = 0; i < VR; ++i) {
            const int t = lr + L * i;
#pragma unroll
            for (int j = 0; j < CT; ++j)
                vn[i][j] = (t < RC && base + t < len && col + j < e) ? v[(size_t)(base + t) * p.stride + j]
                                                                    : from_f32<TX>(0.f);
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

    const int chunks = (len + RC - 1) / RC;
    for (int c = 0; c < chunks; ++c) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                // the chunk is there; everyone is through with the last one
        if (c + 1 < chunks)
            fetch(c + 1, bufs + ((c + 1) & 1) * BLOCK);
        const float* KE = bufs + (c & 1) * BLOCK;
        const float* GE = KE + RC * DP;
        const float* Q = GE + DP;
        const float* NO = Q + RC * DP;
        const float* W = NO + RC * RC;
        const float* M = W + RC * DP;
        const int base = c * RC;
        float vt[VR][CT];
#pragma unroll
        for (int i = 0; i < VR; ++i)
#pragma unroll
            for (int j = 0; j < CT; ++j) {
                vt[i][j] = to_f32(vn[i][j]);
                if (p.activate)
                    vt[i][j] = lr_silu<TX>(vt[i][j]);
            }
        if (c + 1 < chunks)
            fetch_v(base + RC);
        // A S_0 + N V, folded: thread lr ends with values lr OWN .. of the [token][column] tile
        auto product = [&](const float* A, const float* N, float (&acc)[SUMS]) {
#pragma unroll
            for (int t = 0; t < RC; ++t) {
                uint64_t pair[CT];
#pragma unroll
                for (int u = 0; u < RUNS; ++u) {
                    const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(A + t * DP + r0 + RUN_STEP * u);
#pragma unroll
                    for (int j = 0; j < CT; ++j) {
                        pair[j] = u == 0 ? rc_mul2(a.x, S[0][j]) : rc_fma2(a.x, S[2 * u][j], pair[j]);
                        pair[j] = rc_fma2(a.y, S[2 * u + 1][j], pair[j]);
                    }
                }
                float s[CT];
#pragma unroll
                for (int j = 0; j < CT; ++j) {
                    const float2 halves = rc_halves(pair[j]);
                    s[j] = halves.x + halves.y;
                }
#pragma unroll
                for (int i = 0; i < VR; ++i) {
                    const float m = L <= RC || lr < RC ? N[t * RC + lr + L * i] : 0.f;
#pragma unroll
                    for (int j = 0; j < CT; ++j)
                        s[j] = fmaf(m, vt[i][j], s[j]);
                }
#pragma unroll
                for (int j = 0; j < CT; ++j)
                    acc[CT * t + j] = s[j];
            }
#pragma unroll
            for (int o = L / 2, half = SUMS / 2; o >= 1; o >>= 1, half >>= 1) {
                const bool upper = (lr & o) != 0;
#pragma unroll
                for (int i = 0; i < half; ++i) {
                    const float send = upper ? acc[i] : acc[i + half];
                    const float keep = upper ? acc[i + half] : acc[i];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
        };
        if (DELTA) {
            float acc[SUMS];
            product(W, M, acc);
#pragma unroll
            for (int i = 0; i < OWN; ++i)
                Us[((lr * OWN + i) / CT) * CP + c0 + (lr * OWN + i) % CT] = acc[i];
        } else {
#pragma unroll
            for (int i = 0; i < VR; ++i)
#pragma unroll
                for (int j = 0; j < CT; ++j)
                    if (lr + L * i < RC)
                        Us[(lr + L * i) * CP + c0 + j] = vt[i][j];
        }
        __syncthreads();
        {
            float acc[SUMS];
            product(Q, NO, acc);
#pragma unroll
            for (int i = 0; i < OWN; ++i) {
                const int t = (lr * OWN + i) / CT, j = (lr * OWN + i) % CT;
                if (base + t < len && col + j < e)
                    p.o[(size_t)(row0 + base + t) * p.heads * e + (size_t)h * e + col + j] = acc[i];
            }
        }
        // S = diag(G_end) S_0 + KE^T U
#pragma unroll
        for (int u = 0; u < RUNS; ++u) {
            const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(GE + r0 + RUN_STEP * u);
#pragma unroll
            for (int j = 0; j < CT; ++j) {
                S[2 * u][j] = rc_mul2(S[2 * u][j], g.x);
                S[2 * u + 1][j] = rc_mul2(S[2 * u + 1][j], g.y);
            }
        }
#pragma unroll
        for (int s = 0; s < RC; ++s) {
            float uv[CT];
            if constexpr (CT == 4) {
                const float4 u4 = *reinterpret_cast<const float4*>(Us + s * CP + c0);
                uv[0] = u4.x, uv[1] = u4.y, uv[2] = u4.z, uv[3] = u4.w;
            } else if constexpr (CT == 2) {
                const float2 u2 = *reinterpret_cast<const float2*>(Us + s * CP + c0);
                uv[0] = u2.x, uv[1] = u2.y;
            } else {
                uv[0] = Us[s * CP + c0];
            }
#pragma unroll
            for (int u = 0; u < RUNS; ++u) {
                const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(KE + s * DP + r0 + RUN_STEP * u);
#pragma unroll
                for (int j = 0; j < CT; ++j) {
                    const uint64_t both = rc_pair(uv[j], uv[j]);
                    S[2 * u][j] = rc_fma2(k.x, both, S[2 * u][j]);
                    S[2 * u + 1][j] = rc_fma2(k.y, both, S[2 * u + 1][j]);
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < RT / 2; ++i) {
        const int r = r0 + RUN_STEP * (i / 2) + 2 * (i % 2);
#pragma unroll
        for (int j = 0; j < CT; ++j) {
            const float2 halves = rc_halves(S[i][j]);
            if (r < d && col + j < e)
                st[(size_t)r * e + col + j] = halves.x;
            if (r + 1 < d && col + j < e)
                st[(size_t)(r + 1) * e + col + j] = halves.y;
        }
    }
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
            v = lr_silu<TX>(v);
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
                    kv = lr_silu<TX>(kv), qv = lr_silu<TX>(qv);
                kv *= ik;
                qv *= iq;
                g = DELTA ? lr_decay<TX>(rate, p.logits[row * p.logit_stride + h * d + c] + p.dt_bias[h * d + c]) : decay;
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

template <int DP, int RT, int CT, int COLS, bool DELTA, typename TX>
static void launch_chunks(const RecurrenceParams& p, int seqs, cudaStream_t stream)
{
    const size_t smem = (size_t)(2 * rc_block(DP, DELTA) + RC * (COLS + 4)) * sizeof(float);
    auto kernel = chunk_recurrence_kernel<DP, RT, CT, COLS, DELTA, TX>;
    if (smem > 48 * 1024)
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch(kernel, dim3((unsigned)((p.e + COLS - 1) / COLS), (unsigned)p.heads, (unsigned)seqs),
           dim3((DP / RT) * (COLS / CT)), smem, stream, p);
}

template <int DP, bool DELTA, typename TX>
static void launch_prompt(const RecurrenceParams& p, int seqs, int max_q_len, cudaStream_t stream)
{
    const size_t smem = (size_t)(DELTA ? 3 * RC + 4 : 2 * RC) * DP * sizeof(float);
    auto prepare = recurrence_prepare_kernel<DP, DELTA, TX>;
    if (smem > 44 * 1024)
        cudaFuncSetAttribute(prepare, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch(prepare, dim3((unsigned)((max_q_len + RC - 1) / RC), (unsigned)p.heads, (unsigned)seqs), dim3(256), smem, stream, p);
    // as few columns a block as give every SM one block and no more, and the fewer the smaller a thread's piece
    constexpr int RT = DP >= 128 ? 8 : 4;
    const long long per_head = (long long)p.heads * seqs, sms = recurrence_sm_count();
    if (((p.e + 7) / 8) * per_head <= sms)
        launch_chunks<DP, RT, DP >= 256 ? 2 : 1, 8, DELTA, TX>(p, seqs, stream);
    else if (((p.e + 15) / 16) * per_head <= sms)
        launch_chunks<DP, DP >= 256 ? 8 : 4, DP >= 128 ? 4 : 2, 16, DELTA, TX>(p, seqs, stream);
    else
        launch_chunks<DP, RT, 4, 32, DELTA, TX>(p, seqs, stream);
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
