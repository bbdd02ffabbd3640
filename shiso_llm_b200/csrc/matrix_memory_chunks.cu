// The matrix memory's recurrence for prompt portions in chunks of 64 rows on the tensor cores (bfloat16 rows).
//
// With S the state before a chunk, l_t <= 0 the base-2 logarithm of row t's factor on the old state, b_t <= 0
// that of its factor on the new write and L_i = l_1 + .. + l_i,
//
//     S^T q read at row i = 2^(L_i) S^T q_i + sum_(j<=i) 2^(L_i - L_j + b_j) (q_i . k_j) v_j
//     S behind the chunk  = 2^(L_64) S + sum_j 2^(L_64 - L_j + b_j) k_j v_j^T,
//
// every exponent at most zero.  The normaliser is one more value column that is always 1.
//
// One CTA walks the chunks of one (head, sequence, slice of value columns); eight warps, m16n8k16 products
// with float accumulators.  Queries, keys and values are bfloat16 as they came; whatever is float - the
// state, the weighted dot products and the weighted values - enters a product as the sum of two bfloat16
// numbers (what the first leaves over is the second), which keeps 16 bits of mantissa and more, so the
// state stays a float state: it lives in the registers of the warps that update it and is
// written to shared memory, split, once a chunk for the read-out.  Warp (r, c) = (warp % 4, warp / 4):
//
//   dot products   rows 16 r .. + 15 against columns 32 c .. + 31 (nothing where all lie behind the rows);
//   read-out       the same rows; c shares out the key channels of S^T q and the columns of the second sum;
//                  the two shares meet in shared memory;
//   update         16 key channels of the state a warp: K^T (weighted values).
//
// Queries, keys, values and factors of the next chunk are on their way (cp.async) while one is worked on;
// two barriers a chunk.  Chunks are counted from a portion's start: another cut of a prompt adds the same
// numbers up in another order; nothing depends on the rest of the batch.
#include "mma_tiles.cuh"

namespace {

using namespace mma_tiles;

constexpr int CH = 64;       // rows a chunk
constexpr int VC = 16;       // value columns a CTA
constexpr int MC_THREADS = 256;
constexpr int MC_MAX_DIM = 128;
constexpr int V_ROW = VC * 2 + 16;  // bytes of a padded row of values, weighted values or state

struct ChunkArgs {
    const __nv_bfloat16 *q, *k, *v;
    long long q_ld, k_ld, v_ld;
    const float *log_keep, *log_add;  // [T, heads], base 2
    float *state, *normaliser;
    long long state_stride, norm_stride;
    const int *q_start, *state_slots;
    float *out, *norm_out;            // [T, heads * vdim], [T, heads]
    int heads, dim, vdim;
};

__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}

// Two floats as two pairs of bfloat16: the nearest ones and what those leave over.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    const float hx = __uint_as_float(hi << 16), hy = __uint_as_float(hi & 0xffff0000u);
    lo = pack_bf16(x - hx, y - hy);
}

__device__ __forceinline__ void ldmatrix_a_trans(uint32_t addr, uint32_t (&r)[4]) { ldmatrix_x4_trans(addr, r[0], r[1], r[2], r[3]); }

// 2^x of a weight (x <= 0): two units in the last place, below 2^-126 zero.
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// DIM: the key size, or 0 where it is a run-time number.
template <int DIM>
__global__ void __launch_bounds__(MC_THREADS, 2) memory_chunks_kernel(const ChunkArgs a) {
    const int h = blockIdx.x, s = blockIdx.y, col0 = blockIdx.z * VC;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int wr = warp & 3, wc = warp >> 2, g = lane >> 2, t4 = lane & 3;
    const int dim = DIM ? DIM : a.dim, vdim = a.vdim, ksteps = dim / 16;
    const int k_row = dim * 2 + 16, pieces = dim / 8;
    extern __shared__ __align__(16) uint8_t sm[];
    const int tile = CH * k_row;
    const int stage_bytes = 2 * tile + CH * V_ROW + 2 * CH * 4;
    uint8_t* st_hi = sm + 2 * stage_bytes;             // [dim][V_ROW]: the state, split
    uint8_t* st_lo = st_hi + dim * V_ROW;
    uint8_t* w_hi = st_lo + dim * V_ROW;               // [CH][V_ROW]: weighted values, split
    uint8_t* w_lo = w_hi + CH * V_ROW;
    float* share = (float*)(w_lo + CH * V_ROW);        // [CH][VC + 2]: the read-out's second share
    float* gates = share + CH * (VC + 2) + warp * 2 * CH;  // this warp's L_i and b_i - L_i
    pdl_wait();
    const int first = a.q_start[s], n = a.q_start[s + 1] - first;
    if (n <= 0) return;
    const __nv_bfloat16* qp = a.q + (size_t)first * a.q_ld + (size_t)h * dim;
    const __nv_bfloat16* kp = a.k + (size_t)first * a.k_ld + (size_t)h * dim;
    const __nv_bfloat16* vp = a.v + (size_t)first * a.v_ld + (size_t)h * vdim;
    const float* lk = a.log_keep + (size_t)first * a.heads + h;
    const float* la = a.log_add + (size_t)first * a.heads + h;
    const int chunks = (n + CH - 1) / CH;

    // the columns no value lies in never change: the normaliser's ones, zeros behind it
    for (int i = tid; i < 2 * CH * (VC / 8); i += MC_THREADS) {
        const int stage = i / (CH * (VC / 8)), r = i / (VC / 8) % CH, c = i % (VC / 8) * 8;
        if (col0 + c >= vdim)
            *reinterpret_cast<uint4*>(sm + stage * stage_bytes + 2 * tile + r * V_ROW + c * 2) = make_uint4(col0 + c == vdim ? 0x3f80u : 0u, 0u, 0u, 0u);
    }
    const int shift = pieces > 8 ? 4 : pieces > 4 ? 3 : pieces > 2 ? 2 : 1;  // 2^shift threads a row of queries and keys
    const int piece = tid & ((1 << shift) - 1), row_of = tid >> shift, rows_a_pass = MC_THREADS >> shift;
    auto load = [&](int chunk, int stage) {
        uint8_t* base = sm + stage * stage_bytes;
        const int row0 = chunk * CH, count = min(CH, n - row0);
        if (piece < pieces) {
            uint8_t* to = base + row_of * k_row + piece * 16;
            const __nv_bfloat16* from_q = qp + (size_t)(row0 + row_of) * a.q_ld + piece * 8;
            const __nv_bfloat16* from_k = kp + (size_t)(row0 + row_of) * a.k_ld + piece * 8;
#pragma unroll
            for (int r = row_of; r < CH; r += rows_a_pass) {
                const bool ok = r < count;
                cp_async16(to, ok ? from_q : qp, ok);
                cp_async16(to + tile, ok ? from_k : kp, ok);
                to += rows_a_pass * k_row;
                from_q += rows_a_pass * a.q_ld;
                from_k += rows_a_pass * a.k_ld;
            }
        }
        static_assert(VC == 16 && MC_THREADS >= 2 * CH, "two threads a row of values");
        if (tid < 2 * CH && col0 + (tid & 1) * 8 < vdim) {
            const int r = tid >> 1, c = (tid & 1) * 8;
            const bool ok = r < count;
            cp_async16(base + 2 * tile + r * V_ROW + c * 2, vp + (size_t)(row0 + (ok ? r : 0)) * a.v_ld + col0 + c, ok);
        }
        float* f = (float*)(base + 2 * tile + CH * V_ROW);
        if (tid < 2 * CH) {
            const int r = tid % CH;
            if (r < count) cp_async4(f + tid, (tid < CH ? lk : la) + (size_t)(row0 + r) * a.heads);
            else f[tid] = tid < CH ? 0.0f : -INFINITY;  // rows beyond the portion neither forget nor write
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0, 0);

    // ---- the state: warp w holds key channels 16 w .. + 15 (rows g and g + 8), columns 8 j + 2 t4 and the next
    float* slot = a.state + (size_t)a.state_slots[s] * a.state_stride + (size_t)h * dim * vdim;
    float* nslot = a.normaliser + (size_t)a.state_slots[s] * a.norm_stride + (size_t)h * dim;
    const bool holds = warp < ksteps;
    float S[VC / 8][4];
    auto place = [&](int j, int e, int& row, int& col) {
        row = warp * 16 + g + (e >> 1) * 8;
        col = col0 + j * 8 + t4 * 2 + (e & 1);
    };
    auto publish = [&]() {  // the state into shared memory, split
        if (!holds) return;
#pragma unroll
        for (int j = 0; j < VC / 8; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t hi, lo;
                split2(S[j][half * 2], S[j][half * 2 + 1], hi, lo);
                const int at = (warp * 16 + g + half * 8) * V_ROW + (j * 8 + t4 * 2) * 2;
                *reinterpret_cast<uint32_t*>(st_hi + at) = hi;
                *reinterpret_cast<uint32_t*>(st_lo + at) = lo;
            }
    };
#pragma unroll
    for (int j = 0; j < VC / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            int row, col;
            place(j, e, row, col);
            S[j][e] = holds && col <= vdim ? (col < vdim ? slot[(size_t)row * vdim + col] : nslot[row]) : 0.0f;
        }
    publish();

    const int half_steps = (ksteps + 1) / 2;  // wc shares out the channels of S^T q: each its own first
    const int kk_first = wc ? half_steps : 0;
    const int reads_steps = wc ? ksteps - half_steps : half_steps;
    for (int chunk = 0; chunk < chunks; ++chunk) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the chunk has landed, the state is published, nobody reads the other stage any more
        if (chunk + 1 < chunks) load(chunk + 1, (chunk + 1) & 1);
        const uint8_t* base = sm + (chunk & 1) * stage_bytes;
        const uint8_t *qs = base, *ks = base + tile, *vs = base + 2 * tile;
        const float* f = (const float*)(vs + CH * V_ROW);
        // ---- L_i, by every warp for itself: lane l has rows l and l + 32
        float l0 = f[lane], l1 = f[lane + 32];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float p0 = __shfl_up_sync(0xffffffffu, l0, o), p1 = __shfl_up_sync(0xffffffffu, l1, o);
            if (lane >= o) l0 += p0, l1 += p1;
        }
        l1 += __shfl_sync(0xffffffffu, l0, 31);
        const float last = __shfl_sync(0xffffffffu, l1, 31);
        gates[lane] = l0, gates[lane + 32] = l1;
        gates[CH + lane] = f[CH + lane] - l0, gates[CH + lane + 32] = f[CH + lane + 32] - l1;
        __syncwarp();
        const float row_l[2] = {gates[wr * 16 + g], gates[wr * 16 + g + 8]};
        // ---- dot products of 16 rows and 32 columns, and this warp's share of S^T q
        float acc[VC / 8][4], dot[4][4];
#pragma unroll
        for (int j = 0; j < VC / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j) dot[j][0] = dot[j][1] = dot[j][2] = dot[j][3] = 0.0f;
        const bool sees = wc * 32 <= wr * 16 + 15;  // some column is not behind every row
        const uint32_t q_base = smem_addr(qs + (wr * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * k_row + (lane >> 4) * 16);
        const uint32_t k_base = smem_addr(ks + (wc * 32 + (lane & 7) + (lane >> 4) * 8) * k_row + ((lane >> 3) & 1) * 16);
        const uint32_t s_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * V_ROW + (lane >> 4) * 16;
#pragma unroll 4
        for (int step = 0; step < ksteps; ++step) {
            const bool reads = step < reads_steps;
            if (!sees && !reads) break;
            int kk = kk_first + step;
            if (kk >= ksteps) kk -= ksteps;
            uint32_t qf[4];
            ldmatrix_x4(q_base + kk * 32, qf[0], qf[1], qf[2], qf[3]);
            if (sees) {
#pragma unroll
                for (int j = 0; j < 4; j += 2) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4(k_base + j * 8 * k_row + kk * 32, b0, b1, b2, b3);
                    mma_bf16(dot[j], qf, b0, b1);
                    mma_bf16(dot[j + 1], qf, b2, b3);
                }
            }
            if (reads) {
#pragma unroll
                for (int j = 0; j < VC / 8; j += 2) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4_trans(smem_addr(st_hi) + s_off + kk * 16 * V_ROW + j * 16, b0, b1, b2, b3);
                    mma_bf16(acc[j], qf, b0, b1);
                    mma_bf16(acc[j + 1], qf, b2, b3);
                    ldmatrix_x4_trans(smem_addr(st_lo) + s_off + kk * 16 * V_ROW + j * 16, b0, b1, b2, b3);
                    mma_bf16(acc[j], qf, b0, b1);
                    mma_bf16(acc[j + 1], qf, b2, b3);
                }
            }
        }
        const float decay[2] = {ex2(row_l[0]), ex2(row_l[1])};
#pragma unroll
        for (int j = 0; j < VC / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[j][e] *= decay[e >> 1];
        // ---- weighted dot products times the values
        if (sees) {
#pragma unroll
            for (int kk = 0; kk < 2; ++kk) {  // 16 columns each
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int j = kk * 2 + half, c = wc * 32 + j * 8 + t4 * 2;
                    const float b0 = gates[CH + c], b1 = gates[CH + c + 1];
                    float m[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int row = wr * 16 + g + (e >> 1) * 8;
                        m[e] = c + (e & 1) <= row ? dot[j][e] * ex2(row_l[e >> 1] + ((e & 1) ? b1 : b0)) : 0.0f;
                    }
                    split2(m[0], m[1], hi[half * 2], lo[half * 2]);
                    split2(m[2], m[3], hi[half * 2 + 1], lo[half * 2 + 1]);
                }
#pragma unroll
                for (int j = 0; j < VC / 8; j += 2) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4_trans(smem_addr(vs) + s_off + (wc * 32 + kk * 16) * V_ROW + j * 16, b0, b1, b2, b3);
                    mma_bf16(acc[j], hi, b0, b1);
                    mma_bf16(acc[j + 1], hi, b2, b3);
                    mma_bf16(acc[j], lo, b0, b1);
                    mma_bf16(acc[j + 1], lo, b2, b3);
                }
            }
        }
        if (wc == 1) {
#pragma unroll
            for (int j = 0; j < VC / 8; ++j)
#pragma unroll
                for (int half = 0; half < 2; ++half)
                    *reinterpret_cast<float2*>(share + (wr * 16 + g + half * 8) * (VC + 2) + j * 8 + t4 * 2) = make_float2(acc[j][half * 2], acc[j][half * 2 + 1]);
        }
        // ---- the values, weighted for the state behind the chunk
        {
            static_assert(MC_THREADS == 4 * CH, "four threads a row of four columns each");
            const int r = tid >> 2, at = r * V_ROW + (tid & 3) * 8;
            const uint2 raw = *reinterpret_cast<const uint2*>(vs + at);
            const float w = ex2(last + gates[CH + r]);
            uint2 hi, lo;
            split2(w * __uint_as_float(raw.x << 16), w * __uint_as_float(raw.x & 0xffff0000u), hi.x, lo.x);
            split2(w * __uint_as_float(raw.y << 16), w * __uint_as_float(raw.y & 0xffff0000u), hi.y, lo.y);
            *reinterpret_cast<uint2*>(w_hi + at) = hi;
            *reinterpret_cast<uint2*>(w_lo + at) = lo;
        }
        __syncthreads();  // shares and weighted values are written, the published state has been read
        if (wc == 0) {
#pragma unroll
            for (int j = 0; j < VC / 8; ++j)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int r = wr * 16 + g + half * 8, row = chunk * CH + r, c = j * 8 + t4 * 2, col = col0 + c;
                    if (row >= n || col > vdim) continue;
                    const float2 other = *reinterpret_cast<const float2*>(share + r * (VC + 2) + c);
                    const float x = acc[j][half * 2] + other.x, y = acc[j][half * 2 + 1] + other.y;
                    const size_t t = (size_t)(first + row);
                    if (col < vdim) *reinterpret_cast<float2*>(a.out + (t * a.heads + h) * vdim + col) = make_float2(x, y);
                    else a.norm_out[t * a.heads + h] = x;  // (vdim is even: its column is the first of a pair)
                }
        }
        // ---- the state
        if (holds) {
            const float keep = ex2(last);
#pragma unroll
            for (int j = 0; j < VC / 8; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[j][e] *= keep;
            const uint32_t kt_base = smem_addr(ks + ((lane & 7) + (lane >> 4) * 8) * k_row + warp * 32 + ((lane >> 3) & 1) * 16);
#pragma unroll
            for (int kk = 0; kk < CH / 16; ++kk) {
                uint32_t kf[4];
                ldmatrix_a_trans(kt_base + kk * 16 * k_row, kf);
#pragma unroll
                for (int j = 0; j < VC / 8; j += 2) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4_trans(smem_addr(w_hi) + s_off + kk * 16 * V_ROW + j * 16, b0, b1, b2, b3);
                    mma_bf16(S[j], kf, b0, b1);
                    mma_bf16(S[j + 1], kf, b2, b3);
                    ldmatrix_x4_trans(smem_addr(w_lo) + s_off + kk * 16 * V_ROW + j * 16, b0, b1, b2, b3);
                    mma_bf16(S[j], kf, b0, b1);
                    mma_bf16(S[j + 1], kf, b2, b3);
                }
            }
            if (chunk + 1 < chunks) publish();
        }
    }
    pdl_trigger();
#pragma unroll
    for (int j = 0; j < VC / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            int row, col;
            place(j, e, row, col);
            if (!holds || col > vdim) continue;
            if (col < vdim) slot[(size_t)row * vdim + col] = S[j][e];
            else nslot[row] = S[j][e];
        }
}

}  // namespace

// Whether the chunked kernel takes these sizes (others take the kernel for scalar-decay recurrences).
SHISO_API int shiso_memory_chunks_supported(int dim, int vdim) { return dim >= 16 && dim <= MC_MAX_DIM && dim % 16 == 0 && vdim >= 8 && vdim % 8 == 0; }

// bfloat16 rows; log_keep and log_add float [T, heads]; state [slots, heads, dim, vdim], normaliser [slots, heads, dim];
// out float [T, heads * vdim], norm_out float [T, heads].
SHISO_API int shiso_memory_chunks(const void* q, const void* k, const void* v, long long q_ld, long long k_ld, long long v_ld,
                                  const float* log_keep, const float* log_add, float* state, long long state_stride, float* normaliser,
                                  long long norm_stride, const int* q_start, const int* state_slots, float* out, float* norm_out, int num_seqs,
                                  int heads, int dim, int vdim, cudaStream_t stream) {
    if (num_seqs <= 0) return SHISO_OK;
    if (heads <= 0 || num_seqs > 65535) return SHISO_ERR_SHAPE;
    if (!shiso_memory_chunks_supported(dim, vdim)) return SHISO_ERR_UNSUPPORTED;
    if ((((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15) || q_ld % 8 || k_ld % 8 || v_ld % 8 || ((uintptr_t)out & 7)) return SHISO_ERR_ALIGN;
    const int k_row = dim * 2 + 16;
    const size_t smem = (size_t)2 * (2 * CH * k_row + CH * V_ROW + 2 * CH * 4) + 2 * dim * V_ROW + 2 * CH * V_ROW + CH * (VC + 2) * 4 + 8 * 2 * CH * 4;
    auto kernel = dim == 128 ? memory_chunks_kernel<128> : dim == 64 ? memory_chunks_kernel<64> : memory_chunks_kernel<0>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024);
        if (e != cudaSuccess) return (int)e;
    }
    if (smem > 112 * 1024) return SHISO_ERR_SHAPE;
    const ChunkArgs a = {(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, q_ld, k_ld, v_ld, log_keep, log_add, state,
                         normaliser, state_stride, norm_stride, q_start, state_slots, out, norm_out, heads, dim, vdim};
    // (without the dependent-launch attribute: CTAs that become resident under the tail of the kernel
    // before them pile up on the SMs that have room first, and a CTA here runs as long as the portion)
    kernel<<<dim3(heads, num_seqs, (vdim + 1 + VC - 1) / VC), MC_THREADS, smem, stream>>>(a);
    return launch_status();
}
