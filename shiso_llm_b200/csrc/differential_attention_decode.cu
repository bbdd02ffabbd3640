// Differential attention for steps of single tokens, bfloat16: both softmax maps of a group of heads from one
// read of its keys and values, their difference, its norm and the gate in one kernel.
//
// One CTA per (part of the keys, key head, sequence), as in attention_decode_tma.cu, whose way of moving
// bytes this is: a producer warp brings every page of a 64-key tile with 3-D TMA boxes of 64 channels
// into a ring of six tiles; the parts of a (sequence, key head) are a thread-block cluster and are merged
// through its shared memory.  What differs:
//   * a cached key row holds the keys of both maps, [map 1 | map 2].  The rows of the MMA's A operand are the
//     group's query heads of map 1 and then of map 2, each zero outside its own map's channels, so one
//     product over the whole key row gives both maps' scores;
//   * eight consumer warps, four to a tile and every second tile each: a tile is up to 32 KB here;
//   * whoever merges a head gets both of its maps' rows, and a warp forms the difference, its root mean
//     square over the head and the gated output.
// Sums run in an order that depends on the sequence's length and the launch's shape only.  Every wait is
// bounded and reports through the status word.
#include "tcgen05.cuh"

namespace {

using namespace tc;

constexpr int TILE = 64, ROW = 128;
constexpr int BOX_BYTES = TILE * ROW;  // 64 positions x 64 channels
constexpr int STAGES = 6;
constexpr int CONSUMERS = 8;           // two sets of four warps
constexpr int THREADS = (CONSUMERS + 1) * 32;
constexpr int MAX_PARTS = 8;
constexpr int INBOX_ROWS = 32;         // parts x 2 maps x the heads a CTA merges: at most 28 for 8 heads a group

struct DiffDecodeArgs {
    const __nv_bfloat16 *q, *gate;
    const int *block_table, *positions, *seq_of_token;
    __nv_bfloat16* out;
    int* status;
    long long q_ld, gate_ld, out_ld;
    int width, heads, kv_heads, page_size, splits, window, cache_rows;
    float scale_log2, second, factor, eps;
};

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ void cluster_meet() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t in_cta(uint32_t local, uint32_t rank) {
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(local), "r"(rank));
    return r;
}
__device__ __forceinline__ void store_remote(uint32_t address, float v) { asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(address), "f"(v) : "memory"); }
__device__ __forceinline__ void consumer_sync() { asm volatile("bar.sync 1, %0;" ::"n"(CONSUMERS * 32) : "memory"); }

template <int D, int VH>
struct Layout {
    static constexpr int KB = 2 * D / 64, V = 64 * VH, BOXES = KB + VH;
    static constexpr int STAGE_BYTES = BOXES * BOX_BYTES;
    static constexpr int MERGE_ROW = V + 2;  // sums, running maximum (log2 units), sum of weights
    static constexpr int SMEM = STAGES * STAGE_BYTES + 256 + INBOX_ROWS * MERGE_ROW * 4 + 1024;
};

template <int D, int VH>
__global__ void __launch_bounds__(THREADS, 1)
differential_decode_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, DiffDecodeArgs a) {
    using L = Layout<D, VH>;
    constexpr int KSTEPS = 2 * D / 16, DTILES = L::V / 8;
    static_assert(CONSUMERS * 16 * L::MERGE_ROW * 4 <= STAGES * L::STAGE_BYTES, "the merge area lies over the ring");
    extern __shared__ uint8_t smem_raw[];
    uint8_t* ring = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);  // [STAGES][key boxes | value boxes]
    uint64_t* full = (uint64_t*)(ring + STAGES * L::STAGE_BYTES);
    uint64_t* empty = full + STAGES;
    int* shared_ints = (int*)(empty + STAGES);  // failed
    float* inbox = (float*)(ring + STAGES * L::STAGE_BYTES + 256);
    float* merge = (float*)ring;                // after the loop: [CONSUMERS][16][MERGE_ROW]

    const int split = blockIdx.x, g_head = blockIdx.y, t = blockIdx.z;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int pages_per_tile = TILE / a.page_size;
    // step data was uploaded before the chain of kernels began
    const int pos = a.positions[t], seq = a.seq_of_token[t];
    const int lo = a.window > 0 ? max(0, pos + 1 - a.window) : 0;
    const int first_tile = lo / TILE, n_tiles = pos / TILE - first_tile + 1;
    const int per_part = (n_tiles + a.splits - 1) / a.splits;
    const int parts = (n_tiles + per_part - 1) / per_part;  // parts that have keys
    const int tile0 = split * per_part;
    const int my_tiles = min(per_part, n_tiles - tile0);
    if (my_tiles <= 0) {  // uniform: a part past the sequence's end has nothing to send
        if (parts > 1) cluster_meet();
        return;
    }
    if (tid == 0) {
        for (int s = 0; s < STAGES; ++s) {
            mbar_init(&full[s], L::BOXES * pages_per_tile);  // one arrival (with its bytes) per box
            mbar_init(&empty[s], 4);
        }
        shared_ints[0] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __syncthreads();
    bool failed = false;
    const int per = a.heads / a.kv_heads, group = 2 * per;  // rows of the MMA: map 1's query heads, map 2's
    const int g = lane >> 2, t4 = lane & 3;
    float o_acc[DTILES][4];
    float row_max[2] = {-INFINITY, -INFINITY}, row_sum[2] = {0.0f, 0.0f};

    if (warp == CONSUMERS) {
        // ---- producer: a lane owns one box of one of the tiles of a round
        const int boxes = L::BOXES * pages_per_tile;  // at most 32
        const int tiles_per_round = min(STAGES, 32 / boxes);
        const int sub = lane / boxes, rest = lane % boxes, what = rest % L::BOXES, pg = rest / L::BOXES;
        const int* table = a.block_table + (size_t)seq * a.width;
        const uint32_t box_bytes = a.page_size * ROW;
        for (int base = 0; base < my_tiles && !failed; base += tiles_per_round) {
            const int i = base + sub;
            const bool on = sub < tiles_per_round && i < my_tiles;
            int row = a.cache_rows;  // a page wholly outside the keys this token sees: zeros
            if (on) {
                const int key = (first_tile + tile0 + i) * TILE + pg * a.page_size;
                if (key <= pos && key + a.page_size > lo) row = table[key / a.page_size] * a.page_size;
            }
            if (base == 0) pdl_wait();  // the cache rows of this step were written by the kernel before
            if (on) {
                const int stage = i % STAGES, use = i / STAGES;
                if (use > 0 && !mbar_wait(&empty[stage], (use - 1) & 1)) {
                    failed = true;
                } else {
                    mbar_expect_tx(&full[stage], box_bytes);
                    const bool key_box = what < L::KB;
                    tma_load_3d(ring + stage * L::STAGE_BYTES + what * BOX_BYTES + pg * box_bytes, key_box ? &map_k : &map_v, 0,
                                key_box ? g_head * L::KB + what : g_head * VH + what - L::KB, row, &full[stage]);
                }
            }
            failed = __any_sync(0xffffffffu, failed);
        }
    } else {
        // ---- consumers: warp w takes keys 16 (w % 4) .. + 15 of the tiles of parity w / 4
        pdl_wait();
        const int quarter = warp & 3;
        uint32_t q_frag[KSTEPS][4];
        {
            const __nv_bfloat16* rows = a.q + (size_t)t * a.q_ld + (size_t)g_head * group * D;
#pragma unroll
            for (int half = 0; half < 2; ++half) {  // MMA rows g and g + 8
                const int row = g + 8 * half, m = row / per;
                const uint32_t* src = reinterpret_cast<const uint32_t*>(rows + (size_t)min(row, group - 1) * D);
#pragma unroll
                for (int kk = 0; kk < KSTEPS; ++kk) {
                    const bool mine = row < group && kk / (D / 16) == m;
                    const int word = (kk % (D / 16)) * 8 + t4;
                    q_frag[kk][half] = mine ? src[word] : 0u;
                    q_frag[kk][2 + half] = mine ? src[word + 4] : 0u;
                }
            }
        }
#pragma unroll
        for (int i = 0; i < DTILES; ++i) o_acc[i][0] = o_acc[i][1] = o_acc[i][2] = o_acc[i][3] = 0.0f;
        const uint32_t swz = lane & 7;  // a row's 16-byte pieces are stored at piece ^ (row & 7)
        for (int i = warp >> 2; i < my_tiles; i += 2) {
            const int stage = i % STAGES, use = i / STAGES;
            if (!mbar_wait(&full[stage], use & 1)) {
                failed = true;
                break;
            }
            const uint32_t kt = smem_u32(ring + stage * L::STAGE_BYTES) + quarter * 16 * ROW;
            const uint32_t vt = kt + L::KB * BOX_BYTES;
            const int key0 = (first_tile + tile0 + i) * TILE + quarter * 16;
            if (key0 <= pos && key0 + 16 > lo) {  // warp-uniform: some of this warp's keys are seen
                float s_acc[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
#pragma unroll
                for (int kk = 0; kk < KSTEPS; ++kk) {
                    const uint32_t r = (lane & 7) + (lane >> 4) * 8;
                    const uint32_t piece = (kk & 3) * 2 + ((lane >> 3) & 1);
                    uint32_t b0, b1, b2, b3;
                    ldsm_x4(kt + (kk >> 2) * BOX_BYTES + r * ROW + ((piece ^ swz) << 4), b0, b1, b2, b3);
                    mma16816(s_acc[0], q_frag[kk], b0, b1);
                    mma16816(s_acc[1], q_frag[kk], b2, b3);
                }
                float tile_max[2] = {-INFINITY, -INFINITY};
#pragma unroll
                for (int j = 0; j < 2; ++j) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int key = key0 + j * 8 + t4 * 2 + (e & 1);
                        const float v = key >= lo && key <= pos ? s_acc[j][e] * a.scale_log2 : -INFINITY;
                        s_acc[j][e] = v;
                        tile_max[e >> 1] = fmaxf(tile_max[e >> 1], v);
                    }
                }
                float correction[2], use_max[2];
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    float mx = tile_max[r];
                    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                    const float new_max = fmaxf(row_max[r], mx);  // finite: one of the 16 keys is seen
                    use_max[r] = new_max;
                    correction[r] = exp2f(row_max[r] - new_max);
                    row_max[r] = new_max;
                }
                float tile_sum[2] = {0.0f, 0.0f};
                uint32_t p_frag[4];
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    float p[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        p[e] = exp2f(s_acc[j][e] - use_max[e >> 1]);
                        tile_sum[e >> 1] += p[e];
                    }
                    p_frag[j * 2 + 0] = pack2(p[0], p[1]);
                    p_frag[j * 2 + 1] = pack2(p[2], p[3]);
                }
#pragma unroll
                for (int r = 0; r < 2; ++r) row_sum[r] = row_sum[r] * correction[r] + tile_sum[r];
#pragma unroll
                for (int d = 0; d < DTILES; ++d) {
                    o_acc[d][0] *= correction[0];
                    o_acc[d][1] *= correction[0];
                    o_acc[d][2] *= correction[1];
                    o_acc[d][3] *= correction[1];
                }
#pragma unroll
                for (int dn = 0; dn < DTILES; dn += 2) {
                    const uint32_t r = (lane & 7) + ((lane >> 3) & 1) * 8;
                    const uint32_t piece = (dn & 7) + (lane >> 4);
                    uint32_t b0, b1, b2, b3;
                    ldsm_x4_trans(vt + (dn >> 3) * BOX_BYTES + r * ROW + ((piece ^ swz) << 4), b0, b1, b2, b3);
                    mma16816(o_acc[dn], p_frag, b0, b1);
                    mma16816(o_acc[dn + 1], p_frag, b2, b3);
                }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[stage]);  // the producer may refill the stage
        }
    }
    pdl_trigger();
    if (failed) shared_ints[0] = 1;
    if (warp == CONSUMERS) {
        if (parts > 1) cluster_meet();
        return;
    }

    // ---- the warps' results side by side (over the ring: every tile has been consumed)
    consumer_sync();
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        float sum = row_sum[r];
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        float* dst = merge + ((size_t)warp * 16 + g + r * 8) * L::MERGE_ROW;
#pragma unroll
        for (int d = 0; d < DTILES; ++d) *reinterpret_cast<float2*>(dst + d * 8 + t4 * 2) = make_float2(o_acc[d][r * 2], o_acc[d][r * 2 + 1]);
        if (t4 == 0) {
            dst[L::V] = row_max[r];
            dst[L::V + 1] = sum;
        }
    }
    consumer_sync();
    // head j of the group is merged by part j % parts, which keeps what part p sends it of map m at
    // inbox[((j / parts) * 2 + m) * parts + p]
    const uint32_t inbox_local = smem_u32(inbox);
    for (int i = tid; i < group * L::V; i += CONSUMERS * 32) {
        const int row = i / L::V, col = i % L::V, m = row / per, j = row % per;
        float top = -INFINITY;
#pragma unroll
        for (int w = 0; w < CONSUMERS; ++w) top = fmaxf(top, merge[((size_t)w * 16 + row) * L::MERGE_ROW + L::V]);
        float sum = 0.0f, o = 0.0f;
#pragma unroll
        for (int w = 0; w < CONSUMERS; ++w) {
            const float* src = merge + ((size_t)w * 16 + row) * L::MERGE_ROW;
            const float f = src[L::V] == -INFINITY ? 0.0f : exp2f(src[L::V] - top);
            sum += f * src[L::V + 1];
            o += f * src[col];
        }
        const int place = ((j / parts) * 2 + m) * parts + split;
        if (parts == 1) {
            float* dst = inbox + place * L::MERGE_ROW;
            dst[col] = o;
            if (col == 0) dst[L::V] = top, dst[L::V + 1] = sum;
        } else {
            const uint32_t dst = in_cta(inbox_local, (uint32_t)(j % parts)) + (uint32_t)(place * L::MERGE_ROW) * 4u;
            store_remote(dst + col * 4u, o);
            if (col == 0) {
                store_remote(dst + L::V * 4u, top);
                store_remote(dst + (L::V + 1) * 4u, sum);
            }
        }
    }
    if (parts == 1) consumer_sync();
    else cluster_meet();
    // ---- a warp a head: both maps' parts in part order, the difference, its norm, the gate
    for (int j = split + warp * parts; j < per; j += CONSUMERS * parts) {
        constexpr int C = L::V / 32;
        float d[C];
#pragma unroll
        for (int c = 0; c < C; ++c) d[c] = 0.0f;
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            const float* base = inbox + (size_t)((j / parts) * 2 + m) * parts * L::MERGE_ROW;
            float top = -INFINITY;
            for (int p = 0; p < parts; ++p) top = fmaxf(top, base[p * L::MERGE_ROW + L::V]);
            float sum = 0.0f, acc[C];
#pragma unroll
            for (int c = 0; c < C; ++c) acc[c] = 0.0f;
            for (int p = 0; p < parts; ++p) {
                const float* src = base + p * L::MERGE_ROW;
                const float f = src[L::V] == -INFINITY ? 0.0f : exp2f(src[L::V] - top);
                sum += f * src[L::V + 1];
#pragma unroll
                for (int c = 0; c < C; ++c) acc[c] += f * src[lane + 32 * c];
            }
            const float inv = sum > 0.0f ? (m == 0 ? 1.0f : -a.second) / sum : 0.0f;
#pragma unroll
            for (int c = 0; c < C; ++c) d[c] = fmaf(acc[c], inv, d[c]);
        }
        float ss = 0.0f;
#pragma unroll
        for (int c = 0; c < C; ++c) ss = fmaf(d[c], d[c], ss);
        const float f = rsqrtf(warp_sum(ss) / (float)L::V + a.eps) * a.factor;
        const size_t col = (size_t)(g_head * per + j) * L::V;
        const __nv_bfloat16* gate = a.gate + (size_t)t * a.gate_ld + col;
        __nv_bfloat16* out = a.out + (size_t)t * a.out_ld + col;
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const float z = __bfloat162float(gate[lane + 32 * c]);
            out[lane + 32 * c] = __float2bfloat16_rn(d[c] * f * __fdividef(1.0f, 1.0f + __expf(-z)));
        }
    }
    if (tid == 0 && shared_ints[0] != 0 && a.status) atomicExch(a.status, 1);
}

template <int D, int VH>
int launch_differential_decode(const CUtensorMap& mk, const CUtensorMap& mv, const DiffDecodeArgs& a, int tokens, cudaStream_t stream) {
    constexpr int SMEM = Layout<D, VH>::SMEM;
    auto kernel = differential_decode_kernel<D, VH>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.splits, a.kv_heads, tokens);
    cfg.blockDim = dim3(THREADS);
    cfg.dynamicSmemBytes = SMEM;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = shiso_pdl_enabled() ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;  // the parts of a (sequence, key head)
    attr[1].val.clusterDim.x = a.splits;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    return (int)cudaLaunchKernelEx(&cfg, kernel, mk, mv, a);
}

}  // namespace

// Whether the kernel takes these sizes (dim: channels of one map).
SHISO_API int shiso_differential_decode_supported(int heads, int kv_heads, int dim, int vdim, int page_size) {
    return (dim == 32 || dim == 64) && (vdim == 64 || vdim == 128) && kv_heads > 0 && heads % kv_heads == 0 && heads / kv_heads <= 8 &&
           page_size >= 8 && page_size <= TILE && page_size % 8 == 0 && TILE % page_size == 0 && tc::encode_fn() != nullptr;
}

// As shiso_differential_prefill, for one row per sequence; at most 8 parts.
SHISO_API int shiso_differential_decode(const void* q, long long q_ld, const void* k_cache, const void* v_cache, const int* block_table,
                                        int table_width, const int* positions, const int* seq_of_token, const void* gate, long long gate_ld,
                                        void* out, long long out_ld, int tokens, int heads, int kv_heads, int dim, int vdim, int page_size,
                                        long long num_pages, float scale, int window, int splits, float second, float factor, float eps,
                                        cudaStream_t stream) {
    if (tokens <= 0) return SHISO_OK;
    if (splits < 1 || splits > MAX_PARTS || tokens > 65535 || kv_heads > 65535) return SHISO_ERR_SHAPE;
    if (!shiso_differential_decode_supported(heads, kv_heads, dim, vdim, page_size)) return SHISO_ERR_UNSUPPORTED;
    if ((((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) || ((uintptr_t)q & 3) || q_ld % 2) return SHISO_ERR_ALIGN;
    const long long cache_rows = num_pages * page_size;
    if (cache_rows + page_size > 0x7fffffffLL) return SHISO_ERR_UNSUPPORTED;
    CUtensorMap mk, mv;
    if (!tc::tensor_map_paged(k_cache, cache_rows, kv_heads * 2 * dim / 64, page_size, &mk) ||
        !tc::tensor_map_paged(v_cache, cache_rows, kv_heads * vdim / 64, page_size, &mv))
        return SHISO_ERR_UNSUPPORTED;
    DiffDecodeArgs a = {(const __nv_bfloat16*)q, (const __nv_bfloat16*)gate, block_table, positions, seq_of_token, (__nv_bfloat16*)out,
                        shiso_tc_status_word(), q_ld, gate_ld, out_ld, table_width, heads, kv_heads, page_size, splits, window,
                        (int)cache_rows, scale * 1.4426950408889634f, second, factor, eps};
    if (dim == 64) return vdim == 128 ? launch_differential_decode<64, 2>(mk, mv, a, tokens, stream) : launch_differential_decode<64, 1>(mk, mv, a, tokens, stream);
    return vdim == 128 ? launch_differential_decode<32, 2>(mk, mv, a, tokens, stream) : launch_differential_decode<32, 1>(mk, mv, a, tokens, stream);
}
