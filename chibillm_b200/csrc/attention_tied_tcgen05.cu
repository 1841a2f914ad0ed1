// Causal attention for prompt portions on the 5th-generation tensor cores where the values are the keys (one array,
// as attention over cached latents has it) and a cache row is wider than 128 numbers: -DCHIBI_HEAD_DIM=d, d a
// multiple of 16 above 128 and up to 256.
//
// One CTA owns 128 query rows of one key head, (token, head of the group) pairs, and walks over the keys in tiles of
// 96.  A tile is fetched once: it is the K-major operand of S = Q K^T and the MN-major operand of O += P K.
//
//   warp 0      loads key tiles with TMA, three tiles deep: one box brings eight keys with all whole 64-wide
//               slices of their rows (one more the rest of a row, zeros past its end).  A tile lies in shared memory
//               as [8 keys][slice], a swizzle atom each: with a box per page and slice, 2 KB each, the loader took
//               2,200 cycles a tile of 48 KB, and everything waited for it;
//   warp 1      issues the MMAs:  S(j + 1) into one of two TMEM buffers before  O += P(j) K(j);
//   warps 2..9  softmax: two threads, of warps w and w + 4, share query row r, half of a tile's keys each (one warp
//               to a scheduler would wait for its own results most of the time).  They exchange their halves' maxima
//               through shared memory; P = exp2(S * scale - max) goes back into the first columns of its S buffer
//               as packed bfloat16 and is the A operand from there, so it never leaves TMEM.
//
// With one key head the query rows of a CTA are neighbours in memory: they come by TMA, and a full tile of output rows
// leaves by TMA from where they were (with loads and stores by the threads a CTA's start and end took as long as
// eleven tiles).  The output accumulates in TMEM over all tiles and is rescaled there only when a row's maximum has grown by more
// than 2^8.  TMEM: S at columns 0 and 128, O from 256 on.  All waits are bounded.
#define CHIBI_UNIT attention_tied_tcgen05
#define CHIBI_UNIT_ID 16
#include "common.cuh"
#include "sm100.cuh"
#include "attention_tc.cuh"
#include "tensor_map.cuh"

#ifndef CHIBI_HEAD_DIM
#define CHIBI_HEAD_DIM 256
#endif

namespace chibi {

using namespace sm100;

constexpr int D = CHIBI_HEAD_DIM;
static_assert(D % 16 == 0 && D > 128 && D <= 256, "rows of 144 to 256 numbers, a multiple of 16");
constexpr int ROWS = 128;                      // query rows per CTA = UMMA M
constexpr int KEYS = 96;                       // keys per tile
constexpr int STAGES = 3;
constexpr int SLICES = (D + 63) / 64;          // 64-wide (128-byte) slices of a row
constexpr int WHOLE = D / 64;                  // of which are whole
constexpr int GROUPS = KEYS / 8;               // keys of a tile, eight by eight
constexpr int GROUP_BYTES = SLICES * 1024;
constexpr int THREADS = 320;
constexpr int HALF = KEYS / 2;                 // keys of a tile per softmax thread
constexpr int Q_BYTES = SLICES * ROWS * 128;
constexpr int TILE_BYTES = SLICES * KEYS * 128;
constexpr int SMEM_TILES = Q_BYTES + STAGES * TILE_BYTES;
constexpr int NUM_BARS = 2 * STAGES + 7;
constexpr int EXCHANGE_BYTES = 2 * 2 * ROWS * 4;
constexpr size_t SMEM = SMEM_TILES + EXCHANGE_BYTES + NUM_BARS * 8 + 16 + 1024;
static_assert(SMEM <= 227 * 1024, "shared memory of one CTA");
constexpr uint32_t TMEM_O = 256;

// A 128-byte-swizzled operand: leading and stride byte offsets as the layout above has them (a key group of eight
// is the stride of both products; the slices of a row are the leading offset where the row is the N dimension).
__device__ __forceinline__ uint64_t sw128_desc(uint32_t smem_byte_addr, uint32_t lbo_bytes, uint32_t sbo_bytes)
{
    uint64_t d = 0;
    d |= static_cast<uint64_t>((smem_byte_addr & 0x3ffff) >> 4);
    d |= static_cast<uint64_t>(lbo_bytes == 1 ? 1 : (lbo_bytes >> 4) & 0x3fff) << 16;
    d |= static_cast<uint64_t>(sbo_bytes >> 4) << 32;
    d |= static_cast<uint64_t>(1) << 46;
    d |= static_cast<uint64_t>(2) << 61;
    return d;
}

// O[row, columns] *= f for this thread's half of its row's runs of 16 columns (a rare event: out of line so that its
// registers do not count against the loop).
__device__ __noinline__ void rescale_row(uint32_t o_addr, int half, float f)
{
#pragma unroll 1
    for (int c0 = 16 * half; c0 < D; c0 += 32) {
        uint32_t v[16];
        tmem_load_32x16(o_addr + c0, v);
        tmem_load_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i)
            v[i] = __float_as_uint(__uint_as_float(v[i]) * f);
        tmem_store_32x16(o_addr + c0, v);
    }
    tmem_store_wait();
}

// Maps of the rows of the cache (boxes of 8 rows), of q and of the output (boxes of 128): all whole slices, the rest.
struct TiedMaps {
    CUtensorMap cache, cache_rest, q, q_rest, out, out_rest;
};

__global__ void __launch_bounds__(THREADS, 1)
attn_prefill_tied_kernel(const __grid_constant__ TiedMaps maps, const AttnTcParams p)
{
    pdl_enter();
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* q_s = smem;
    uint8_t* k_s = q_s + Q_BYTES;                  // STAGES tiles
    float* exchange = reinterpret_cast<float*>(smem + SMEM_TILES);           // [2][half][row]
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + SMEM_TILES + EXCHANGE_BYTES);
    uint64_t* k_full = bars;                       // [STAGES] TMA
    uint64_t* k_empty = bars + STAGES;             // [STAGES] MMA commit: both products of the tile are done
    uint64_t* s_full = bars + 2 * STAGES;          // [2] MMA commit
    uint64_t* p_full = s_full + 2;                 // [2] 256 threads
    uint64_t* o_done = p_full + 2;                 // [2] MMA commit: O holds tile j
    uint64_t* q_full = o_done + 2;                 // TMA (one key head)
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + NUM_BARS);

    // the row tiles with the most keys start first, for all key heads
    const int seq = blockIdx.z / p.kv_splits, split = blockIdx.z - seq * p.kv_splits;
    const int linear = blockIdx.x + gridDim.x * blockIdx.y;
    const int kv_head = linear % gridDim.y, tile_rank = linear / gridDim.y;
    const int t0 = p.q_start[seq];
    const int q_len = p.q_start[seq + 1] - t0;
    const int rows_total = q_len * p.group;
    const int row0 = (gridDim.x - 1 - tile_rank) * ROWS;
    if (q_len <= 0 || (q_len == 1 && p.skip_single) || row0 >= rows_total)
        return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos0 = p.ctx_len[seq] - q_len;
    const int* table = p.block_table + (size_t)(p.seq_rows ? p.seq_rows[seq] : seq) * p.table_stride;

    const int last_row = min(rows_total, row0 + ROWS) - 1;
    const int min_pos = pos0 + row0 / p.group, max_pos = pos0 + last_row / p.group;
    int key_begin = first_visible_key(min_pos, p.window, p.chunk);
    key_begin = key_begin / p.page_size * p.page_size;           // tiles start on a page
    const int key_end = max_pos + 1;
    int n_tiles = (key_end - key_begin + KEYS - 1) / KEYS;
    if (p.kv_splits > 1) {
        // this CTA's range of the row tile's key tiles (it may be empty)
        const int per = (n_tiles + p.kv_splits - 1) / p.kv_splits;
        const int lo = split * per;
        n_tiles = max(0, min(per, n_tiles - lo));
        key_begin += lo * KEYS;
    }

    if (threadIdx.x == 0) {
        for (int i = 0; i < STAGES; ++i) {
            mbar_init(&k_full[i], 1);
            mbar_init(&k_empty[i], 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&s_full[i], 1);
            mbar_init(&p_full[i], 256);
            mbar_init(&o_done[i], 1);
        }
        mbar_init(q_full, 1);
        fence_barrier_init();
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, 512);
        tmem_relinquish();
    }
    // query rows -> shared memory in the swizzled K-major layout: by TMA below, or all threads help, eight loads of a
    // thread at a time
    const bool neighbours = p.nkv == 1;
    for (int c0 = threadIdx.x; !neighbours && c0 < ROWS * (D / 8); c0 += 8 * THREADS) {
        uint4 v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = c0 + i * THREADS;
            const int row = c / (D / 8), chunk = c - row * (D / 8);
            const int r = row0 + row;
            v[i] = make_uint4(0, 0, 0, 0);
            if (c < ROWS * (D / 8) && r < rows_total) {
                const int tok = r / p.group, h = r - tok * p.group;
                v[i] = *reinterpret_cast<const uint4*>(p.q + ((size_t)(t0 + tok) * p.nq + kv_head * p.group + h) * D + chunk * 8);
            }
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = c0 + i * THREADS;
            const int row = c / (D / 8), chunk = c - row * (D / 8);
            if (c < ROWS * (D / 8))
                *reinterpret_cast<uint4*>(q_s + (chunk >> 3) * (ROWS * 128) + swizzled_chunk(row, chunk & 7)) = v[i];
        }
    }
    fence_proxy_async();               // the tensor core reads what these threads wrote
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        // Lane i brings keys 8 i .. 8 i + 7 of every tile (of one page: pages are multiples of eight keys), their
        // page looked up one tile ahead.
        if (lane == 0) {
            tma_prefetch_descriptor(&maps.cache);
            if (neighbours) {
                // (rows past the sequence's end are somebody else's or zeros; their results go nowhere)
                mbar_arrive_expect_tx(q_full, Q_BYTES);
                tma_load_3d(q_s, &maps.q, q_full, 0, t0 * p.nq + row0, 0);
                if (WHOLE < SLICES)
                    tma_load_2d(q_s + WHOLE * (ROWS * 128), &maps.q_rest, q_full, WHOLE * 64, t0 * p.nq + row0);
            }
        }
        __syncwarp();
        auto first_row_of = [&](int j) -> long long {
            const int key = key_begin + j * KEYS + lane * 8;
            if (lane >= GROUPS || key >= key_end)
                return p.cache_rows;      // past the context: read outside the array, zeros
            const int page = table[key / p.page_size];
            if (page < 0 || page >= p.num_pages) {
                if (p.error)
                    atomicExch(p.error, 3);
                return p.cache_rows;
            }
            return ((long long)page * p.nkv + kv_head) * p.page_size + key % p.page_size;
        };
        long long row = n_tiles > 0 ? first_row_of(0) : 0;
        for (int j = 0; j < n_tiles; ++j) {
            const long long row_next = j + 1 < n_tiles ? first_row_of(j + 1) : 0;
            const int st = j % STAGES, round = j / STAGES;
            uint8_t* dst = k_s + st * TILE_BYTES;
            if (lane == 0) {
                if (round > 0)
                    mbar_wait(&k_empty[st], (round - 1) & 1, p.error, 21);
                mbar_arrive_expect_tx(&k_full[st], TILE_BYTES);
            }
            __syncwarp();
            if (lane < GROUPS) {
                tma_load_3d(dst + lane * GROUP_BYTES, &maps.cache, &k_full[st], 0, (int)row, 0);
                if (WHOLE < SLICES)
                    tma_load_2d(dst + lane * GROUP_BYTES + WHOLE * 1024, &maps.cache_rest, &k_full[st], WHOLE * 64, (int)row);
            }
            row = row_next;
        }
    } else if (warp == 1) {
        if (elect_one()) {
            constexpr uint32_t idesc_qk = make_idesc_bf16_f32(ROWS, KEYS);
            constexpr uint32_t idesc_pv = make_idesc_bf16_f32(ROWS, D) | (1u << 16);    // B is MN-major
            const uint32_t q_addr = smem_addr(q_s);
            auto issue_qk = [&](int j) {
                const int st = j % STAGES;
                mbar_wait(&k_full[st], (j / STAGES) & 1, p.error, 22);
                tcgen05_fence_after();
                const uint32_t k_addr = smem_addr(k_s + st * TILE_BYTES);
#pragma unroll
                for (int ks = 0; ks < D / 16; ++ks)
                    tcgen05_mma_bf16(tmem_base + (j & 1) * 128,
                                     make_kmajor_sw128_desc(q_addr + (ks >> 2) * (ROWS * 128) + (ks & 3) * 32),
                                     sw128_desc(k_addr + (ks >> 2) * 1024 + (ks & 3) * 32, 1, GROUP_BYTES), idesc_qk,
                                     ks > 0 ? 1u : 0u);
                tcgen05_commit(&s_full[j & 1]);
            };
            if (neighbours)
                mbar_wait(q_full, 0, p.error, 23);       // (also with no tile: nothing may be on its way at the end)
            if (n_tiles > 0)
                issue_qk(0);
            for (int j = 0; j < n_tiles; ++j) {
                // S(j + 1) may be overwritten: its buffer's last reader, the product with P(j - 1), was issued before
                if (j + 1 < n_tiles)
                    issue_qk(j + 1);                                  // runs while the softmax threads work on tile j
                const int st = j % STAGES;
                mbar_wait(&p_full[j & 1], (j >> 1) & 1, p.error, 24);    // P(j) is in TMEM
                tcgen05_fence_after();
                const uint32_t k_addr = smem_addr(k_s + st * TILE_BYTES);
#pragma unroll
                for (int ks = 0; ks < KEYS / 16; ++ks)
                    tcgen05_mma_bf16_a_tmem(tmem_base + TMEM_O, tmem_base + (j & 1) * 128 + ks * 8,
                                            sw128_desc(k_addr + ks * 2 * GROUP_BYTES, 1024, GROUP_BYTES), idesc_pv,
                                            (j > 0 || ks > 0) ? 1u : 0u);
                tcgen05_commit(&o_done[j & 1]);
                tcgen05_commit(&k_empty[st]);
            }
        }
    } else {
        const int quarter = warp & 3, half = warp >= 6 ? 1 : 0;
        const int row = quarter * 32 + lane;                 // this thread's query row = its TMEM lane
        const int r = row0 + row;
        const bool live = r < rows_total;
        const int tok = live ? r / p.group : 0;
        const int pos = live ? pos0 + tok : -1;
        const int first = first_visible_key(pos, p.window, p.chunk);
        const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quarter * 32) << 16);
        const uint32_t o_addr = lane_addr + TMEM_O;
        const float sl2 = p.scale_log2;
        // `m`: the maximum that the exponents are taken against; it follows the true maximum only when that has
        // grown by more than 2^8, so the probabilities stay below 2^8
        float m = -INFINITY, l = 0.f;
        for (int j = 0; j < n_tiles; ++j) {
            const int key0 = key_begin + j * KEYS;
            mbar_wait(&s_full[j & 1], (j >> 1) & 1, p.error, 26);
            tcgen05_fence_after();
            const uint32_t s_addr = lane_addr + (j & 1) * 128;
            uint32_t sv[HALF];
#pragma unroll
            for (int c0 = 0; c0 < HALF; c0 += 16)
                tmem_load_32x16(s_addr + half * HALF + c0, *reinterpret_cast<uint32_t(*)[16]>(&sv[c0]));
            tmem_load_wait();
            // masks only where a row's visible range ends inside the tile; the warp takes one path
            if (__any_sync(0xffffffffu, key0 + KEYS - 1 > pos || key0 < first)) {
#pragma unroll
                for (int i = 0; i < HALF; ++i) {
                    const int key = key0 + half * HALF + i;
                    if (!(key <= pos && key >= first))
                        sv[i] = 0xff800000u;                 // -inf
                }
            }
            float mx4[4] = { -INFINITY, -INFINITY, -INFINITY, -INFINITY };
#pragma unroll
            for (int i = 0; i < HALF; ++i)
                mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sv[i]));
            float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * sl2;      // the scale is positive
            // the other half's maximum; behind this barrier both halves of S are in registers, so P may overwrite it
            float* slots = exchange + (j & 1) * 2 * ROWS;
            slots[half * ROWS + row] = mx;
            tcgen05_fence_before();
            asm volatile("bar.sync %0, 64;" ::"r"(quarter + 1) : "memory");
            tcgen05_fence_after();
            mx = fmaxf(mx, slots[(half ^ 1) * ROWS + row]);
            const bool grow = mx > m + 8.f;                  // also true for the first visible key (m = -inf)
            if (__any_sync(0xffffffffu, grow && m != -INFINITY && j > 0)) {
                // rescale what has accumulated: the product of tile j-1 must have landed first
                mbar_wait(&o_done[(j - 1) & 1], ((j - 1) >> 1) & 1, p.error, 27);
                tcgen05_fence_after();
                rescale_row(o_addr, half, (grow && m != -INFINITY) ? fast_exp2(m - mx) : 1.f);
            }
            if (grow) {
                l *= (m == -INFINITY) ? 0.f : fast_exp2(m - mx);
                m = mx;
            }
            const float base = m == -INFINITY ? 0.f : m;
            float sum4[4] = { 0.f, 0.f, 0.f, 0.f };
#pragma unroll
            for (int c0 = 0; c0 < HALF; c0 += 16) {
                uint32_t packed[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const float p0 = fast_exp2(fmaf(__uint_as_float(sv[c0 + 2 * i]), sl2, -base));
                    const float p1 = fast_exp2(fmaf(__uint_as_float(sv[c0 + 2 * i + 1]), sl2, -base));
                    sum4[i & 3] += p0 + p1;
                    const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
                    packed[i] = *reinterpret_cast<const uint32_t*>(&h);
                }
                tmem_store_32x8(s_addr + ((half * HALF + c0) >> 1), packed);
            }
            l += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
            // rows past the context may hold anything (a page is loaded whole): make them zero, so that
            // 0 * value stays 0.  Only the last tile can hold such keys, and its S has been made.
            if (key0 + KEYS > key_end) {
                mbar_wait(&k_full[j % STAGES], (j / STAGES) & 1, p.error, 29);
                uint8_t* tile = k_s + (j % STAGES) * TILE_BYTES;
                for (int c = half * 128 + row; c < (key0 + KEYS - key_end) * (SLICES * 8); c += 256) {
                    const int krow = key_end - key0 + c / (SLICES * 8), chunk = c % (SLICES * 8);
                    *reinterpret_cast<uint4*>(tile + (krow >> 3) * GROUP_BYTES + (chunk >> 3) * 1024 + swizzled_chunk(krow & 7, chunk & 7)) =
                        make_uint4(0, 0, 0, 0);
                }
                fence_proxy_async();
            }
            tmem_store_wait();
            tcgen05_fence_before();
            mbar_arrive(&p_full[j & 1]);
        }
        // the two halves' sums (the exponents' base is the same)
        float* slots = exchange + (n_tiles & 1) * 2 * ROWS;
        slots[half * ROWS + row] = l;
        asm volatile("bar.sync %0, 64;" ::"r"(quarter + 1) : "memory");
        l += slots[(half ^ 1) * ROWS + row];
        // the last product has landed: normalise and write the rows out, every other run of 16 columns
        if (n_tiles > 0)
            mbar_wait(&o_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1, p.error, 28);
        tcgen05_fence_after();
        const int head = kv_head * p.group + (live ? r - tok * p.group : 0);      // (rows past the end have none)
        const bool ranged = p.kv_splits > 1;
        const size_t slot = ((size_t)(t0 + tok) * p.nq + head) * p.kv_splits + split;
        float inv = 1.f;
        if (!ranged) {
            l += sink_weight(p.sink, head, m);
            inv = l > 0.f ? 1.f / l : 0.f;
        } else if (live && half == 0) {
            // one of several key ranges: the row as it stands, with its maximum and sum
            p.part_ml[slot * 2] = m;
            p.part_ml[slot * 2 + 1] = l;
        }
        __nv_bfloat16* dst_row = p.out + ((size_t)(t0 + tok) * p.nq + head) * D;
        // a full tile of neighbouring rows: through shared memory, where the queries were (the last product that reads
        // them, S of the last tile, is long done)
        const bool staged = neighbours && !ranged && row0 + ROWS <= rows_total && n_tiles > 0;
#pragma unroll 1
        for (int c0 = 16 * half; c0 < D; c0 += 32) {
            uint32_t ov[16];
            if (n_tiles > 0) {
                tmem_load_32x16(o_addr + c0, ov);
                tmem_load_wait();
            } else {
#pragma unroll
                for (int i = 0; i < 16; ++i)
                    ov[i] = 0;
            }
            if (!live)
                continue;
            if (ranged) {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    reinterpret_cast<uint4*>(p.part_o + slot * D + c0)[c] = make_uint4(ov[4 * c], ov[4 * c + 1], ov[4 * c + 2], ov[4 * c + 3]);
                continue;
            }
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                __nv_bfloat162 h[4];
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    h[u] = __floats2bfloat162_rn(__uint_as_float(ov[8 * c + 2 * u]) * inv, __uint_as_float(ov[8 * c + 2 * u + 1]) * inv);
                const int chunk = (c0 >> 3) + c;
                uint4* dst = staged ? reinterpret_cast<uint4*>(q_s + (chunk >> 3) * (ROWS * 128) + swizzled_chunk(row, chunk & 7))
                                    : reinterpret_cast<uint4*>(dst_row + c0) + c;
                *dst = *reinterpret_cast<uint4*>(h);
            }
        }
        if (staged) {
            fence_proxy_async();
            asm volatile("bar.sync 5, 256;" ::: "memory");
            if (threadIdx.x == 64) {
                tma_store_3d(&maps.out, q_s, 0, t0 * p.nq + row0, 0);
                if (WHOLE < SLICES)
                    tma_store_2d(&maps.out_rest, q_s + WHOLE * (ROWS * 128), WHOLE * 64, t0 * p.nq + row0);
                tma_store_done();
            }
        }
    }
    tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) {
        tcgen05_fence_after();
        tmem_dealloc(tmem_base, 512);
    }
}

} // namespace chibi

using namespace chibi;

CHIBI_API int chibi_attention_tied_head_dim() { return D; }

// Attention of the sequences that bring more than one token (all sequences when skip_single is 0); `cache`
// [pages][nkv][page_size][D] holds the keys, which are the values.  CHIBI_ERR_UNSUPPORTED for page sizes it does not
// take (multiples of eight are taken).
CHIBI_API int chibi_attention_prefill_tied(const void* q, const void* cache, void* out, const int* block_table,
                                           int table_stride, const int* seq_rows, const int* q_start, const int* ctx_len,
                                           int seqs, int nq, int nkv, int page_size, int num_pages, float scale, int window,
                                           int chunk, int skip_single, int max_q_len, int kv_splits, float* scratch,
                                           long long scratch_floats, long long tokens, const float* sink, int* error,
                                           cudaStream_t stream)
{
    if (seqs <= 0)
        return CHIBI_OK;
    if (nkv <= 0 || nq % nkv != 0 || window < 0 || chunk < 0 || !(scale > 0.f) || max_q_len <= 0 || kv_splits < 1)
        return CHIBI_ERR_ARGUMENT;
    if (page_size < 8 || page_size % 8 != 0 || (reinterpret_cast<uintptr_t>(cache) & 15)
        || (reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(out) & 15))
        return CHIBI_ERR_UNSUPPORTED;
    AttnTcParams p {};
    p.q = static_cast<const __nv_bfloat16*>(q);
    p.out = static_cast<__nv_bfloat16*>(out);
    p.block_table = block_table;
    p.table_stride = table_stride;
    p.seq_rows = seq_rows;
    p.q_start = q_start;
    p.ctx_len = ctx_len;
    p.nq = nq;
    p.nkv = nkv;
    p.group = nq / nkv;
    p.page_size = page_size;
    p.num_pages = num_pages;
    p.cache_rows = (long long)num_pages * nkv * page_size;
    p.scale_log2 = scale * 1.4426950408889634f;
    p.window = window;
    p.chunk = chunk;
    p.skip_single = skip_single;
    p.error = error;
    p.kv_splits = kv_splits;
    p.sink = sink;
    if (kv_splits > 1) {
        if (kv_splits > 64 || !scratch || tokens <= 0 || scratch_floats < tokens * nq * kv_splits * (long long)(D + 2)
            || (long long)seqs * kv_splits > 65535)
            return CHIBI_ERR_ARGUMENT;
        p.part_o = scratch;
        p.part_ml = scratch + (size_t)tokens * nq * kv_splits * D;
    }
    TiedMaps maps;
    const long long q_rows = tokens * nq;
    if (p.cache_rows > 2147483647LL || q_rows <= 0 || q_rows > 2147483647LL
        || !tensor_map_of_rows(cache, p.cache_rows, D, D, 8, WHOLE, &maps.cache)
        || !tensor_map_2d(cache, p.cache_rows, D, D, 8, &maps.cache_rest)
        || !tensor_map_of_rows(q, q_rows, D, D, ROWS, WHOLE, &maps.q) || !tensor_map_2d(q, q_rows, D, D, ROWS, &maps.q_rest)
        || !tensor_map_of_rows(out, q_rows, D, D, ROWS, WHOLE, &maps.out)
        || !tensor_map_2d(out, q_rows, D, D, ROWS, &maps.out_rest))
        return CHIBI_ERR_UNSUPPORTED;
    static bool configured = false;
    if (!configured) {
        const cudaError_t e = cudaFuncSetAttribute(attn_prefill_tied_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                   (int)SMEM);
        if (e != cudaSuccess)
            return (int)e;
        configured = true;
    }
    const long long rows = (long long)max_q_len * p.group;
    launch(attn_prefill_tied_kernel, dim3((unsigned)((rows + ROWS - 1) / ROWS), nkv, seqs * kv_splits), dim3(THREADS), SMEM,
           stream, maps, p);
    int st = launch_status();
    if (st == CHIBI_OK && kv_splits > 1) {
        launch(attn_prefill_merge_kernel<D>, dim3(nq, max_q_len, seqs), dim3(D), 0, stream, p);
        st = launch_status();
    }
    return st;
}
