// Kernels of attention over cached latents whose queries come straight from the layer's input, and of learned
// absolute positions:
//
// * position_rows: x = factor * x + table[position], then, with a weight, x / rms(x) * weight.
// * latent_heads_append: from a row q | c | k_rot | gates of a product (an array or partial sums): every head's
//   first features rotated, the rest of it copied -> array; RMS norm of c and the rotation of k_rot -> one
//   cache row k_rot | c; sigmoid of the heads' gates -> array.
// * head_gate: every head of a row times one number.
//
// Sums, norms, angles and gates are 32-bit whatever the activations' type is.
#define CHIBI_UNIT latent_ops
#define CHIBI_UNIT_ID 15
#include "common.cuh"
#include "row_access.cuh"

namespace chibi {

// ---------------------------------------------------------------- learned positions
// One block per token; the row stays in shared memory between the sum of squares and the output.
template <typename TW, int V>
__global__ void __launch_bounds__(256)
position_rows_kernel(float* __restrict__ x, float factor, const TW* __restrict__ table, int rows,
                     const int* __restrict__ positions, const float* __restrict__ w, float eps, int n,
                     int* __restrict__ error)
{
    pdl_enter();
    extern __shared__ float held[];
    __shared__ float red[33];
    const long long t = blockIdx.x;
    const int pos = positions[t];
    const bool ok = pos >= 0 && pos < rows;
    if (!ok && threadIdx.x == 0 && error)
        atomicExch(error, 6);
    const TW* add = table + (size_t)(ok ? pos : 0) * n;
    float* row = x + t * n;
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < n; c += 256 * V) {
        float a[V], b[V];
        load_values<float, V>(a, row + c);
        load_values<TW, V>(b, add + c);
#pragma unroll
        for (int i = 0; i < V; ++i) {
            a[i] = fmaf(a[i], factor, ok ? b[i] : 0.f);
            ss = fmaf(a[i], a[i], ss);
        }
        store_values<float, V>(w ? held + c : row + c, a);
    }
    if (!w)
        return;
    ss = block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)n + eps);
    for (int c = threadIdx.x * V; c < n; c += 256 * V) {
        float a[V], b[V];
        load_values<float, V>(a, held + c);          // (this thread's own values)
        load_values<float, V>(b, w + c);
#pragma unroll
        for (int i = 0; i < V; ++i)
            a[i] = a[i] * inv * b[i];
        store_values<float, V>(row + c, a);
    }
}

// ---------------------------------------------------------------- queries, cache row and gates
struct LatentHeads {
    const float* kv_norm;            // [kv_rank]
    float eps;
    const float* inv_freq;           // [rot / 2]
    int heads, kv_rank, rot;
    const int* positions;
    const int* seq_of_token;
    const int* seq_rows;             // row of the block table per sequence, or null
    const int* table;
    long long table_stride;
    int page_size, num_pages;
    long long tokens;
    float* gates;                    // [tokens, heads] or null
    int* error;
};

// A warp per job; the jobs of a token are its query heads, its cache row (with a cache) and its gates (with an
// array for them).  Shared memory: kv_rank floats per warp, with a cache.
template <typename TX, typename TC, int V>
__global__ void __launch_bounds__(128)
latent_heads_append_kernel(const LatentHeads p, const ProductRows<TX> rows, TC* __restrict__ q_out,
                           TC* __restrict__ k_cache)
{
    pdl_enter();
    extern __shared__ float smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int own = k_cache ? 1 : 0;
    const unsigned jobs = (unsigned)(p.heads + own + (p.gates ? 1 : 0));
    const unsigned job = blockIdx.x * 4u + (unsigned)warp;
    if (job >= (unsigned)p.tokens * jobs)
        return;
    const long long t = job / jobs;
    const int j = (int)(job % jobs);
    const int kd = p.rot + p.kv_rank, half = p.rot >> 1;
    const int after = p.heads * kd;                       // where c starts
    if (j >= p.heads + own) {
        const int col0 = after + (own ? kd : 0);
        for (int h = lane; h < p.heads; h += 32)
            p.gates[t * p.heads + h] = 1.f / (1.f + expf(-rows.at(t, col0 + h)));
        return;
    }
    TC* dst;
    float inv = 1.f;
    const int turned_at = j < p.heads ? j * kd : after + p.kv_rank;
    float first[2] = {};                                  // the lane's first pair of the rotated part
    if (lane < half)
        first[0] = rows.at(t, turned_at + lane), first[1] = rows.at(t, turned_at + half + lane);
    const int pos = p.positions[t];
    if (j < p.heads) {
        dst = q_out + (t * p.heads + j) * kd;
        for (int c = lane * V; c < p.kv_rank; c += 32 * V) {
            float v[V];
            rows.template load<V>(v, t, turned_at + p.rot + c);
            store_values<TC, V>(dst + p.rot + c, v);
        }
    } else {
        const int seq = p.seq_of_token[t];
        const int page = p.table[(p.seq_rows ? p.seq_rows[seq] : seq) * p.table_stride + pos / p.page_size];
        if (page < 0 || page >= p.num_pages) {
            if (p.error && lane == 0)
                atomicExch(p.error, 2);
            return;
        }
        dst = k_cache + ((long long)page * p.page_size + pos % p.page_size) * kd;
        float* held = smem + (size_t)warp * p.kv_rank;
        float ss = 0.f;
        for (int c = lane * V; c < p.kv_rank; c += 32 * V) {
            float v[V];
            rows.template load<V>(v, t, after + c);
#pragma unroll
            for (int i = 0; i < V; ++i) {
                ss = fmaf(v[i], v[i], ss);
                held[c + i] = v[i];
            }
        }
        inv = 1.f / sqrtf(warp_sum(ss) / (float)p.kv_rank + p.eps);
        for (int c = lane * V; c < p.kv_rank; c += 32 * V) {      // (the lane's own values)
            float v[V];
#pragma unroll
            for (int i = 0; i < V; ++i)
                v[i] = held[c + i] * inv * p.kv_norm[c + i];
            store_values<TC, V>(dst + p.rot + c, v);
        }
    }
    for (int i = lane; i < half; i += 32) {
        float sn, cs;
        sincosf((float)pos * p.inv_freq[i], &sn, &cs);
        const float u = i < 32 ? first[0] : rows.at(t, turned_at + i);
        const float v = i < 32 ? first[1] : rows.at(t, turned_at + half + i);
        dst[i] = from_f32<TC>(u * cs - v * sn);
        dst[half + i] = from_f32<TC>(v * cs + u * sn);
    }
}

// ---------------------------------------------------------------- a gate per head
template <typename T, int V>
__global__ void __launch_bounds__(256)
head_gate_kernel(T* __restrict__ x, const float* __restrict__ gates, long long rows, int heads, int size)
{
    pdl_enter();
    const int n = heads * size;
    const int c = (blockIdx.x * 256 + threadIdx.x) * V;
    if (c >= n)
        return;
    const int h = c / size;
    for (long long t = blockIdx.y; t < rows; t += gridDim.y) {
        const float g = gates[t * heads + h];
        float a[V];
        load_values<T, V>(a, x + t * n + c);
#pragma unroll
        for (int i = 0; i < V; ++i)
            a[i] *= g;
        store_values<T, V>(x + t * n + c, a);
    }
}

} // namespace chibi

using namespace chibi;

CHIBI_API int chibi_position_rows(float* x, float factor, const void* table, int table_type, int table_rows,
                                  const int* positions, const float* w, float eps, long long rows, int n, int* error,
                                  cudaStream_t stream)
{
    if (rows <= 0)
        return CHIBI_OK;
    if (!x || !table || !positions || table_rows <= 0 || n <= 0 || rows > 2147483647LL)
        return CHIBI_ERR_ARGUMENT;
    const size_t smem = w ? (size_t)n * sizeof(float) : 0;
    if (smem > 200 * 1024)
        return CHIBI_ERR_UNSUPPORTED;
    const bool fours = n % 4 == 0 && reinterpret_cast<uintptr_t>(x) % 16 == 0
                       && (!w || reinterpret_cast<uintptr_t>(w) % 16 == 0) && rows_in_fours(table, table_type, n, 0);
    CHIBI_DISPATCH_TYPE(table_type, TW, {
        auto kernel = fours ? position_rows_kernel<TW, 4> : position_rows_kernel<TW, 1>;
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch(kernel, dim3((unsigned)rows), dim3(256), smem, stream, x, factor, (const TW*)table, table_rows, positions,
               w, eps, n, error);
    });
    return launch_status();
}

// `rows`: [tokens] rows of heads * (rot + kv_rank) query columns | (with a cache) kv_rank + rot | (with gates)
// heads; splits > 1: 32-bit partial sums, split_stride apart.  q_out and k_cache have type `out_type`.
CHIBI_API int chibi_latent_heads_append(const void* rows, int x_type, long long stride, int splits,
                                        long long split_stride, void* q_out, void* k_cache, int out_type,
                                        const float* kv_norm, float eps, const float* inv_freq, int heads, int kv_rank,
                                        int rot, float* gates, const int* positions, const int* seq_of_token,
                                        const int* seq_rows, const int* table, long long table_stride, int page_size,
                                        int num_pages, long long tokens, int* error, cudaStream_t stream)
{
    if (tokens <= 0)
        return CHIBI_OK;
    if (!rows || !q_out || !inv_freq || !positions || heads <= 0 || kv_rank <= 0 || rot <= 0 || rot % 2 || splits < 1
        || (splits > 1 && x_type != CHIBI_F32)
        || (k_cache && (!kv_norm || !seq_of_token || !table || page_size <= 0)))
        return CHIBI_ERR_ARGUMENT;
    const long long jobs = tokens * (heads + (k_cache ? 1 : 0) + (gates ? 1 : 0));
    const size_t smem = k_cache ? (size_t)4 * kv_rank * sizeof(float) : 0;
    if (jobs > 2147483647LL || smem > 200 * 1024)
        return CHIBI_ERR_UNSUPPORTED;
    const LatentHeads p { kv_norm, eps, inv_freq, heads, kv_rank, rot, positions, seq_of_token, seq_rows, table,
                          table_stride, page_size, num_pages, tokens, gates, error };
    const uintptr_t unit = out_type == CHIBI_F32 ? 16 : 8;
    const bool fours = kv_rank % 4 == 0 && rot % 4 == 0 && rows_in_fours(rows, x_type, stride, split_stride)
                       && reinterpret_cast<uintptr_t>(q_out) % unit == 0 && reinterpret_cast<uintptr_t>(k_cache) % unit == 0;
    CHIBI_DISPATCH_TYPE(x_type, TX, CHIBI_DISPATCH_TYPE(out_type, TC, {
        auto kernel = fours ? latent_heads_append_kernel<TX, TC, 4> : latent_heads_append_kernel<TX, TC, 1>;
        const ProductRows<TX> source { (const TX*)rows, stride, splits, split_stride };
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch(kernel, dim3((unsigned)((jobs + 3) / 4)), dim3(128), smem, stream, p, source, (TC*)q_out, (TC*)k_cache);
    }));
    return launch_status();
}

CHIBI_API int chibi_head_gate(void* x, int x_type, const float* gates, long long rows, int heads, int size,
                              cudaStream_t stream)
{
    if (rows <= 0)
        return CHIBI_OK;
    if (!x || !gates || heads <= 0 || size <= 0 || (long long)heads * size > 2147483647LL)
        return CHIBI_ERR_ARGUMENT;
    const int n = heads * size;
    const unsigned row_blocks = (unsigned)(rows < 16384 ? rows : 16384);
    const bool wide = size % 8 == 0 && reinterpret_cast<uintptr_t>(x) % 16 == 0;
    CHIBI_DISPATCH_TYPE(x_type, T, {
        if (wide)
            launch(head_gate_kernel<T, 8>, dim3((unsigned)((n / 8 + 255) / 256), row_blocks), dim3(256), 0, stream, (T*)x,
                   gates, rows, heads, size);
        else
            launch(head_gate_kernel<T, 1>, dim3((unsigned)((n + 255) / 256), row_blocks), dim3(256), 0, stream, (T*)x,
                   gates, rows, heads, size);
    });
    return launch_status();
}
