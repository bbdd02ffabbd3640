// Differential attention for long prompt portions on the tensor-memory path (tcgen05), bfloat16: both
// softmax maps of a head, their difference, its norm and the gate in one kernel.
//
// One CTA owns 128 consecutive query rows of one sequence and one head and walks the key tiles of 64
// positions its rows can see.  A head's two maps are two attentions over the same values: each has its
// own queries and keys (D = 32 or 64 channels), scores, statistics and accumulator, and they share every value tile
// that is brought in.  The maps also take the place of the two query tiles that ping-pong on the tensor
// core elsewhere: four warps run one map's softmax while the other map's products run.
//
//   S_m = Q_m K_m^T   tcgen05.mma (M 128, N 64, K D) into 64 float columns of tensor memory; read once by
//                     the map's four warps, a thread per row, after which the next tile's scores may be
//                     formed there while this tile's exponentials are taken;
//   P_m               back to tensor memory as bfloat16, in one of two buffers;
//   O_m += P_m V      tcgen05.mma with P as the A operand from tensor memory and V as it lies in the cache
//                     (positions x channels), 64 channels an instruction, into VH * 64 float columns.
//
// The running maximum is raised only by a tile that exceeds it by more than 2^8 (see the single-map
// kernel in attention_prefill_tc.cu, whose softmax this is).  At the end both maps' warps know each row's
// sums: each map's warps form the difference a_1 - second * a_2 of one half of the row's channels, the two
// halves' sums of squares meet in shared memory, and the normed, gated rows are written once, head by head.
//
// Key and value tiles come from the paged cache by TMA, one box per page and 64 channels, four stages
// ahead.  The cache's rows of a key head are [map 1 | map 2]: two boxes where D = 64, one where D = 32.
// Pages outside the rows' range are fetched past the end of the cache (zeros); rows outside it are
// masked in the scores and zeroed in the value tile.  512 tensor-memory columns, one CTA an SM.  Every
// mbarrier wait is bounded and reports through the status word.
#include "tcgen05.cuh"

namespace {

using namespace tc;

constexpr int BQ = 128, BKEY = 64, ROW = 128;
constexpr int TILE_BYTES = BKEY * ROW;  // 64 positions x 64 channels
constexpr int Q_BYTES = BQ * ROW;       // a map's queries
constexpr int STAGES = 4;
constexpr int SOFTMAX_THREADS = 256;    // warps 0-3: map 1, 4-7: map 2
constexpr int THREADS = SOFTMAX_THREADS + 64;  // 8 producer, 9 MMA
constexpr int TMEM_COLS = 512;
constexpr float RAISE_STEP = 8.0f;

struct DiffArgs {
    const int *block_table, *q_start, *start_pos;
    const __nv_bfloat16* gate;  // [T, heads * V], rows gate_ld apart
    __nv_bfloat16* out;         // [T, heads * V], rows out_ld apart
    long long gate_ld, out_ld;
    int* status;
    int width, num_seqs, heads, kv_heads, page_size, window, cache_rows;
    float scale_log2, second, factor, eps;
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float max3(float a, float b, float c) {
    float d;
    asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
    return d;
}
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint32_t bf16x2(float lo, float hi) {
    uint32_t r;
    asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r) : "f"(hi), "f"(lo));
    return r;
}
__device__ __forceinline__ void ld32(uint32_t addr, uint32_t* r) {
    tmem_ld32_issue(addr, r);
    tmem_ld_wait();
    tmem_ld_pin(r);
    tmem_ld_pin(r + 16);
}
__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, %0;" ::"n"(SOFTMAX_THREADS) : "memory"); }

// D: channels of a map; VH: value channels / 64.
template <int D, int VH>
struct Layout {
    static constexpr int KB = 2 * D / 64;  // key boxes a page
    static constexpr int V = 64 * VH;
    static constexpr int K_BYTES = KB * TILE_BYTES, V_BYTES = VH * TILE_BYTES;
    static constexpr int RING = STAGES * (K_BYTES + V_BYTES);
    static constexpr int SMEM = 2 * Q_BYTES + RING + 1024 + 512 + 4 * BQ * 4;
    static constexpr int S_COL = 0;                 // two maps of 64 float columns
    static constexpr int O_COL = 2 * BKEY;          // two maps of V float columns
    static constexpr int P_COL = O_COL + 2 * V;     // two maps of two buffers of 32 columns
};

template <int D, int VH>
__global__ void __launch_bounds__(THREADS, 1)
differential_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                       const __grid_constant__ CUtensorMap map_v, DiffArgs a) {
    using L = Layout<D, VH>;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint8_t* q_s = smem;                           // [2][Q_BYTES]
    uint8_t* k_s = q_s + 2 * Q_BYTES;              // [STAGES][KB][TILE_BYTES]
    uint8_t* v_s = k_s + STAGES * L::K_BYTES;      // [STAGES][VH][TILE_BYTES]
    uint64_t* bars = (uint64_t*)(v_s + STAGES * L::V_BYTES);
    uint64_t* q_full = bars;
    uint64_t* k_full = bars + 1;
    uint64_t* k_empty = k_full + STAGES;
    uint64_t* v_full = k_empty + STAGES;
    uint64_t* v_empty = v_full + STAGES;
    uint64_t* s_full = v_empty + STAGES;           // [map] a tile's scores are complete
    uint64_t* s_free = s_full + 2;                 // [map] they are in registers
    uint64_t* p_full = s_free + 2;                 // [map][2] a tile's P is written
    uint64_t* pv_done = p_full + 4;                // [map][2] its product with the values is complete
    uint32_t* tmem_slot = (uint32_t*)(pv_done + 4);
    int* shared_ints = (int*)(tmem_slot + 1);      // failed, sequence, first row of the tile
    float* row_inv = (float*)((uint8_t*)bars + 512);  // [map][BQ]
    float* row_ss = row_inv + 2 * BQ;                 // [half][BQ]

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int i = 0; i < STAGES; ++i) {
            mbar_init(&k_full[i], 1);
            mbar_init(&k_empty[i], 1);
            mbar_init(&v_full[i], 1);
            mbar_init(&v_empty[i], 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&s_full[i], 1);
            mbar_init(&s_free[i], 4);  // one arrival per softmax warp of the map
        }
        for (int i = 0; i < 4; ++i) {
            mbar_init(&p_full[i], 4);
            mbar_init(&pv_done[i], 1);
        }
        shared_ints[0] = 0;
        // the last tiles of a portion have the most keys: they take the first CTAs of every head
        int left = gridDim.y - 1 - blockIdx.y, found = -1, row0 = 0;
        for (int s = 0; s < a.num_seqs; ++s) {
            const int tiles = (a.q_start[s + 1] - a.q_start[s] + BQ - 1) / BQ;
            if (left < tiles) {
                found = s;
                row0 = left * BQ;
                break;
            }
            left -= tiles;
        }
        shared_ints[1] = found;
        shared_ints[2] = row0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __syncthreads();
    const int seq = shared_ints[1];
    if (seq < 0) return;  // uniform: before any TMEM allocation
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_base = *tmem_slot;

    const int row0 = shared_ints[2];
    const int first_token = a.q_start[seq] + row0;
    const int rows = min(BQ, a.q_start[seq + 1] - first_token);
    const int first_pos = a.start_pos[seq] + row0, last_pos = first_pos + rows - 1;
    const int head = blockIdx.x, per = a.heads / a.kv_heads, kv_head = head / per;
    const int key_lo = a.window > 0 ? max(0, first_pos + 1 - a.window) : 0;  // the smallest key any row sees
    const int tile_first = key_lo / BKEY, num_tiles = last_pos / BKEY - tile_first + 1;
    bool failed = false;

    pdl_wait();  // queries, keys and values were written by the kernels before this one

    if (warp == 8) {
        // ---- producer: lane p brings page p of every tile, looked up a tile ahead
        if (lane == 0) {
            mbar_expect_tx(q_full, 2 * Q_BYTES);
            for (int m = 0; m < 2; ++m)
                tma_load_2d(q_s + m * Q_BYTES, &map_q, ((2 * kv_head + m) * per + head % per) * D, first_token, q_full);
        }
        const int* table = a.block_table + (size_t)seq * a.width;
        const int pages_per_tile = BKEY / a.page_size;
        auto lookup = [&](int it) {
            const int key = (tile_first + it) * BKEY + lane * a.page_size;
            int page = -1;
            if (lane < pages_per_tile && key <= last_pos && key + a.page_size > key_lo) page = table[key / a.page_size];
            return page >= 0 ? page * a.page_size : a.cache_rows;  // a row past the end of the cache: zeros
        };
        int row_next = lookup(0);
        for (int it = 0; it < num_tiles; ++it) {
            const int s = it % STAGES, uses_before = it / STAGES, row = row_next;
            if (it + 1 < num_tiles) row_next = lookup(it + 1);
            if (uses_before > 0 && !mbar_wait(&k_empty[s], (uses_before - 1) & 1)) failed = true;
            if (lane == 0) mbar_expect_tx(&k_full[s], L::K_BYTES);
            __syncwarp();
            if (lane < pages_per_tile)
                for (int b = 0; b < L::KB; ++b)
                    tma_load_3d(k_s + s * L::K_BYTES + b * TILE_BYTES + lane * a.page_size * ROW, &map_k, 0, kv_head * L::KB + b, row, &k_full[s]);
            if (uses_before > 0 && !mbar_wait(&v_empty[s], (uses_before - 1) & 1)) failed = true;
            if (lane == 0) mbar_expect_tx(&v_full[s], L::V_BYTES);
            __syncwarp();
            if (lane < pages_per_tile)
                for (int b = 0; b < VH; ++b)
                    tma_load_3d(v_s + s * L::V_BYTES + b * TILE_BYTES + lane * a.page_size * ROW, &map_v, 0, kv_head * VH + b, row, &v_full[s]);
        }
    } else if (warp == 9) {
        // ---- MMA issuer
        if (lane == 0) {
            const uint32_t idesc_s = umma_idesc(BQ, BKEY);
            const uint32_t idesc_o = umma_idesc(BQ, 64) | (1u << 16);  // B (the value tile) is MN-major
            auto scores = [&](int m, int it) {
                const int s = it % STAGES;
                if (!mbar_wait(&k_full[s], (it / STAGES) & 1)) failed = true;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t q_addr = smem_u32(q_s + m * Q_BYTES);
                const uint32_t k_addr = smem_u32(k_s + s * L::K_BYTES) + (D == 64 ? m * TILE_BYTES : m * D * 2);
#pragma unroll
                for (int ks = 0; ks < D / UMMA_K; ++ks)
                    umma_bf16(tmem_base + L::S_COL + m * BKEY, umma_desc(q_addr + ks * 32), umma_desc(k_addr + ks * 32), idesc_s, ks > 0 ? 1u : 0u);
                umma_commit(&s_full[m]);
                if (m == 1) umma_commit(&k_empty[s]);
            };
            if (!mbar_wait(q_full, 0)) failed = true;
            scores(0, 0);
            scores(1, 0);
            for (int it = 0; it < num_tiles; ++it) {
                const int b = it & 1, s = it % STAGES;
                if (it + 1 < num_tiles)
                    for (int m = 0; m < 2; ++m) {  // the next tile's scores, while this tile's exponentials are taken
                        if (!mbar_wait(&s_free[m], it & 1)) failed = true;
                        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                        scores(m, it + 1);
                    }
                for (int m = 0; m < 2; ++m) {
                    if (!mbar_wait(&p_full[2 * m + b], (it >> 1) & 1)) failed = true;
                    if (!mbar_wait(&v_full[s], (it / STAGES) & 1)) failed = true;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
                    for (int h = 0; h < VH; ++h) {
                        const uint32_t v_addr = smem_u32(v_s + s * L::V_BYTES + h * TILE_BYTES);
#pragma unroll
                        for (int ks = 0; ks < BKEY / UMMA_K; ++ks)
                            umma_bf16_a_tmem(tmem_base + L::O_COL + m * L::V + h * 64, tmem_base + L::P_COL + (2 * m + b) * (BKEY / 2) + ks * (UMMA_K / 2),
                                             umma_desc(v_addr + ks * 16 * ROW), idesc_o, (it > 0 || ks > 0) ? 1u : 0u);
                    }
                    umma_commit(&pv_done[2 * m + b]);
                }
                umma_commit(&v_empty[s]);
            }
        }
    } else {
        // ---- softmax warps: thread = query row = TMEM lane, of map `m`
        const int m = warp >> 2, quad = warp & 3;
        const int r = quad * 32 + lane;
        const int my_pos = first_pos + r;
        const uint32_t lane_base = tmem_base + ((uint32_t)(quad * 32) << 16);
        const uint32_t s_tmem = lane_base + L::S_COL + m * BKEY, o_tmem = lane_base + L::O_COL + m * L::V;
        float row_max = -INFINITY, row_sum = 0.0f;  // the maximum in use (scaled, log2 units) and the sum against it
        for (int it = 0; it < num_tiles; ++it) {
            const int b = it & 1;
            const int key0 = (tile_first + it) * BKEY;
            // every key of the tile is seen by every row of the CTA: no mask, nothing to zero
            const bool open = key0 + BKEY - 1 <= first_pos && (a.window <= 0 || key0 > first_pos + BQ - 1 - a.window);
            if (!mbar_wait(&s_full[m], it & 1)) failed = true;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            uint32_t sv[BKEY];
            tmem_ld32_issue(s_tmem, sv);
            tmem_ld32_issue(s_tmem + 32, sv + 32);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < BKEY; i += 16) tmem_ld_pin(sv + i);
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_free[m]);
            if (!open) {
                // a key this row does not see scores minus infinity: its exponential is zero
#pragma unroll
                for (int i = 0; i < BKEY; ++i) {
                    const int key = key0 + i;
                    if (!(key <= my_pos && (a.window <= 0 || key > my_pos - a.window))) sv[i] = __float_as_uint(-INFINITY);
                }
            }
            float part_max[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) part_max[j] = fmaxf(__uint_as_float(sv[2 * j]), __uint_as_float(sv[2 * j + 1]));
#pragma unroll
            for (int i = 16; i < BKEY; i += 2) part_max[(i >> 1) & 7] = max3(part_max[(i >> 1) & 7], __uint_as_float(sv[i]), __uint_as_float(sv[i + 1]));
            // the scale is positive: the maximum commutes with it
            const float tile_max = fmaxf(max3(part_max[0], part_max[1], part_max[2]), max3(max3(part_max[3], part_max[4], part_max[5]), part_max[6], part_max[7])) * a.scale_log2;
            const float new_max = tile_max - row_max > RAISE_STEP ? tile_max : row_max;
            const float base = new_max == -INFINITY ? 0.0f : new_max;  // a row that has seen nothing yet
            const float alpha = ex2(row_max - base);
            // this tile's P buffer was the A operand of the product two tiles back
            if (it >= 2 && !mbar_wait(&pv_done[2 * m + b], ((it - 2) >> 1) & 1)) failed = true;
            if (it > 0 && __any_sync(0xffffffffu, new_max != row_max)) {
                // some row of this warp raises its maximum: every product of this map issued so far must
                // be complete, then O *= exp2(old - new) in tensor memory
                if (!mbar_wait(&pv_done[2 * m + (b ^ 1)], ((it - 1) >> 1) & 1)) failed = true;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                uint32_t o[32];
#pragma unroll 1
                for (int c = 0; c < L::V; c += 32) {
                    ld32(o_tmem + c, o);
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                    tmem_st32(o_tmem + c, o);
                }
            }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            // exponentials, their sum, and P into tensor memory
            const uint64_t scale2 = pack2(a.scale_log2, a.scale_log2), minus_base2 = pack2(-base, -base);
            uint64_t sum2[2] = {pack2(0.0f, 0.0f), pack2(0.0f, 0.0f)};
#pragma unroll
            for (int c = 0; c < BKEY; c += 32) {
                uint32_t packed[16];
#pragma unroll
                for (int i = 0; i < 32; i += 2) {
                    float p0, p1;
                    unpack2(fma2(pack2(__uint_as_float(sv[c + i]), __uint_as_float(sv[c + i + 1])), scale2, minus_base2), p0, p1);
                    p0 = ex2(p0);
                    p1 = ex2(p1);
                    sum2[(i >> 1) & 1] = add2(sum2[(i >> 1) & 1], pack2(p0, p1));
                    packed[i >> 1] = bf16x2(p0, p1);
                }
                tmem_st16(lane_base + L::P_COL + (2 * m + b) * (BKEY / 2) + (c >> 1), packed);
            }
            float s0, s1, s2, s3;
            unpack2(sum2[0], s0, s1);
            unpack2(sum2[1], s2, s3);
            row_sum = row_sum * alpha + ((s0 + s1) + (s2 + s3));
            row_max = new_max;
            if (!open && m == 0) {
                // map 1's thread r also looks after value row r of the tile (both maps' products wait for
                // map 1's P): outside the range it becomes zero
                const int vs = it % STAGES;
                if (!mbar_wait(&v_full[vs], (it / STAGES) & 1)) failed = true;
                const int key = key0 + r;
                if (r < BKEY && (key < key_lo || key > last_pos)) {
#pragma unroll
                    for (int h = 0; h < VH; ++h) {
                        uint4* row = reinterpret_cast<uint4*>(v_s + vs * L::V_BYTES + h * TILE_BYTES + r * ROW);
#pragma unroll
                        for (int i = 0; i < ROW / 16; ++i) row[i] = make_uint4(0u, 0u, 0u, 0u);
                    }
                }
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // value rows zeroed by threads, read by the MMA
            }
            tmem_st_wait();  // P (and a scaled O) are in tensor memory
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[2 * m + b]);
        }
        pdl_trigger();
        // ---- the difference: this map's warps take the channels [m * V / 2, (m + 1) * V / 2) of their rows
        constexpr int HALF = L::V / 2;
        // (each map's warps wait for their own last product: only they have followed that barrier's phases)
        if (!mbar_wait(&pv_done[2 * m + ((num_tiles - 1) & 1)], ((num_tiles - 1) >> 1) & 1)) failed = true;
        row_inv[m * BQ + r] = row_sum > 0.0f ? 1.0f / row_sum : 0.0f;  // an empty span yields zeros
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        softmax_sync();
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const float inv1 = row_inv[r], inv2 = -a.second * row_inv[BQ + r];
        float d[HALF];
        float ss = 0.0f;
#pragma unroll
        for (int c = 0; c < HALF; c += 32) {
            uint32_t o1[32], o2[32];
            ld32(lane_base + L::O_COL + m * HALF + c, o1);
            ld32(lane_base + L::O_COL + L::V + m * HALF + c, o2);
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                d[c + i] = fmaf(__uint_as_float(o2[i]), inv2, __uint_as_float(o1[i]) * inv1);
                ss = fmaf(d[c + i], d[c + i], ss);
            }
        }
        row_ss[m * BQ + r] = ss;
        softmax_sync();
        const float f = rsqrtf((row_ss[r] + row_ss[BQ + r]) / (float)L::V + a.eps) * a.factor;
        if (r < rows) {
            const size_t col = (size_t)head * L::V + m * HALF;
            const uint4* g = reinterpret_cast<const uint4*>(a.gate + (size_t)(first_token + r) * a.gate_ld + col);
            uint4* dst = reinterpret_cast<uint4*>(a.out + (size_t)(first_token + r) * a.out_ld + col);
#pragma unroll
            for (int i = 0; i < HALF / 8; ++i) {
                const uint4 raw = g[i];
                const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
                uint32_t o[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float g0 = __uint_as_float(w[j] << 16), g1 = __uint_as_float(w[j] & 0xffff0000u);
                    o[j] = bf16x2(d[8 * i + 2 * j] * f * __fdividef(1.0f, 1.0f + __expf(-g0)), d[8 * i + 2 * j + 1] * f * __fdividef(1.0f, 1.0f + __expf(-g1)));
                }
                dst[i] = make_uint4(o[0], o[1], o[2], o[3]);
            }
        }
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    }
    if (failed) shared_ints[0] = 1;
    __syncwarp();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (shared_ints[0] != 0 && threadIdx.x == 0 && a.status) atomicExch(a.status, 1);
    if (warp == 9) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(TMEM_COLS) : "memory");
    }
}

// Query columns of wider rows, as tiles of BQ x 64 with the 128B swizzle (encoded at every call: such views are not kept).
bool query_map(const void* ptr, int rows, int cols, long long ld, CUtensorMap* out) {
    EncodeTiledFn encode = encode_fn();
    if (!encode || ((uintptr_t)ptr & 15)) return false;
    cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    cuuint32_t box[2] = {64u, (cuuint32_t)BQ};
    cuuint32_t elem[2] = {1, 1};
    return encode(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int D, int VH>
int launch_differential(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const DiffArgs& a, int tiles, cudaStream_t stream) {
    // (at least 120 KB, so that an SM never holds two CTAs: each takes all of the tensor memory)
    constexpr int SMEM = Layout<D, VH>::SMEM > 120 * 1024 ? Layout<D, VH>::SMEM : 120 * 1024;
    auto kernel = differential_tc_kernel<D, VH>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    launch_kernel(kernel, dim3(a.heads, tiles), THREADS, SMEM, stream, mq, mk, mv, a);
    return launch_status();
}

}  // namespace

// Whether the kernel takes these sizes (dim: channels of one map).
SHISO_API int shiso_differential_prefill_supported(int dim, int vdim, int page_size) {
    return (dim == 32 || dim == 64) && (vdim == 64 || vdim == 128) && page_size >= 8 && page_size <= BKEY && page_size % 8 == 0 &&
           BKEY % page_size == 0 && tc::encode_fn() != nullptr;
}

// q: columns (key head, map, query head of the group) x dim of rows q_ld apart; k_cache [pages, page, 2 kv_heads, dim];
// v_cache [pages, page, kv_heads, vdim]; gate and out [T, heads * vdim], rows gate_ld / out_ld apart; max_tiles >= the
// number of 128-row tiles over all sequences; window 0: none.  The scale is positive.
SHISO_API int shiso_differential_prefill(const void* q, long long q_ld, const void* k_cache, const void* v_cache, const int* block_table,
                                         int table_width, const int* q_start, const int* start_pos, const void* gate, long long gate_ld,
                                         void* out, long long out_ld, int tokens, int num_seqs, int max_tiles, int heads, int kv_heads,
                                         int dim, int vdim, int page_size, long long num_pages, float scale, int window, float second,
                                         float factor, float eps, cudaStream_t stream) {
    if (num_seqs <= 0 || max_tiles <= 0 || tokens <= 0) return SHISO_OK;
    if (kv_heads <= 0 || heads % kv_heads || !(scale > 0.0f)) return SHISO_ERR_SHAPE;
    if (!shiso_differential_prefill_supported(dim, vdim, page_size) || max_tiles > 65535) return SHISO_ERR_UNSUPPORTED;
    if ((((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)gate | (uintptr_t)out) & 15) || q_ld % 8 || gate_ld % 8 || out_ld % 8)
        return SHISO_ERR_ALIGN;
    const long long cache_rows = num_pages * page_size;
    if (cache_rows + page_size > 0x7fffffffLL) return SHISO_ERR_UNSUPPORTED;
    CUtensorMap mq, mk, mv;
    if (!query_map(q, tokens, 2 * heads * dim, q_ld, &mq) || !tc::tensor_map_paged(k_cache, cache_rows, kv_heads * 2 * dim / 64, page_size, &mk) ||
        !tc::tensor_map_paged(v_cache, cache_rows, kv_heads * vdim / 64, page_size, &mv))
        return SHISO_ERR_UNSUPPORTED;
    DiffArgs a = {block_table, q_start, start_pos, (const __nv_bfloat16*)gate, (__nv_bfloat16*)out, gate_ld, out_ld, shiso_tc_status_word(),
                  table_width, num_seqs, heads, kv_heads, page_size, window, (int)cache_rows, scale * 1.4426950408889634f, second, factor, eps};
    if (dim == 64) return vdim == 128 ? launch_differential<64, 2>(mq, mk, mv, a, max_tiles, stream) : launch_differential<64, 1>(mq, mk, mv, a, max_tiles, stream);
    return vdim == 128 ? launch_differential<32, 2>(mq, mk, mv, a, max_tiles, stream) : launch_differential<32, 1>(mq, mk, mv, a, max_tiles, stream);
}
