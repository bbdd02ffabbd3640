// The gated delta rule: a matrix state S[dim, vdim] per head that forgets by a factor g and is
// corrected towards each new value,
//
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q,
//
// with q and k brought to unit length per head (q times q_scale as well), beta = sigmoid(b) and
// g = exp(-exp(a_log_h) softplus(a + dt_bias_h)) from one logit each per row and head.  q and k may
// be shared by the heads of a group (head h reads group h / (heads / groups)).
//
// Steps with portions of prompts: the rows of a sequence are taken EIGHT at a time.  Unrolled over
// a block of rows with old state S, and with G_i = g_1 .. g_i and D_ij = g_(j+1) .. g_i (products, never
// quotients),
//
//     u_i = beta_i (v_i - G_i S^T k_i - sum_(j<i) D_ij (k_i . k_j) u_j)
//     o_i = G_i S^T q_i + sum_(j<=i) D_ij (q_i . k_j) u_j
//     S  <- G_8 S + sum_j D_8j k_j u_j^T.
//
// With A_ij = beta_i D_ij (k_i . k_j) below the diagonal, w_i = beta_i v_i - beta_i G_i S^T k_i and
// T = (I + A)^-1 (a unit triangle, by substitution) this is u = T w and o = G S^T q + M w with
// M = (D o (Q K^T)) T: everything that couples the rows is eight-by-eight, the same for all columns
// of the state, and found beforehand.
//
//   delta_prepare_kernel  per (block of rows, group): unit vectors, the dot products between them,
//                         decays, the two triangles per head, beta v; float, in the order the next reads.
//   delta_blocks_kernel   per (head, sequence, range of value columns), block after block: S^T k and
//                         S^T q of all eight rows from the old state, ONE exchange across lanes for the
//                         sixteen results, the triangles, the state.  Walked row by row the state waits
//                         for an exchange across lanes per row; and a lane that holds four columns uses
//                         each key and query it reads from shared memory four times.
//   delta_output_kernel   each head's outputs divided by their root mean square, times a weight shared
//                         by the heads, times silu(gate).
//
// Blocks are counted from a portion's start, so another cut of a prompt adds the same numbers up in
// another order (float throughout; a sequence's sums never depend on the rest of the batch).
//
// Steps of single rows (decode): delta_step_kernel, ONE launch for the convolutions of q, k and v with
// silu and their windows, unit vectors, the state, the output norm and the gate.
#include "common.cuh"

namespace {

constexpr int DB = 8;            // rows a block
constexpr int DC = 2 * DB * DB + 2 * DB + 4;  // a (head, block)'s coefficients: D_8i T_ij, M_ij, beta_i G_i, G_i, G_8 (and padding)
constexpr int D_MAX_DIM = 256;

__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t pair_of(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void halves_of(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }

__device__ __forceinline__ void cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

__device__ __forceinline__ float decay_of(float a_logit, float dt_bias, float rate) {
    const float z = a_logit + dt_bias;
    const float softplus = z > 20.0f ? z : log1pf(expf(z));
    return expf(-rate * softplus);
}
__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_of(float z) { return z / (1.0f + expf(-z)); }
// The same with the special-function unit's exponential and reciprocal: relative error about 2^-21, for
// results that are rounded to bfloat16 at once.
__device__ __forceinline__ float silu_sfu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// Block b of sequence s is number q_start[s] / 8 + s + b of the step: enough room for every sequence's
// last, ragged block, and no prefix sum to find it.
__device__ __forceinline__ int first_block(const int* q_start, int s) { return q_start[s] / DB + s; }

// --------------------------------------------------------------------------- what couples a block's rows

struct PrepareArgs {
    const void *q, *k, *v, *b, *a;
    long long q_ld, k_ld, v_ld, b_ld, a_ld;
    const float *dt_bias, *a_log;
    const int* q_start;
    float* kq;    // [groups][blocks][k: 8 x DP | q: 8 x DP]
    float* coef;  // [heads][blocks][DC]
    float* bv;    // [heads][blocks][chunks of 8 columns][8 rows][8 columns]: beta v
    int num_seqs, blocks, heads, groups, dim, dp, vdim, chunks;
    float q_scale, unit_eps;
};

// PER: entries of a query or key a lane holds (dim in multiples of 32, divided by 32).
template <typename AT, int PER>
__global__ void __launch_bounds__(DB * 32) delta_prepare_kernel(const PrepareArgs a) {
    __shared__ float ks[DB][32 * PER];
    __shared__ float kk[DB][DB], qk[DB][DB];
    __shared__ float gs[DB][DB], bs[DB][DB];               // decay and beta of eight heads' rows
    __shared__ float sA[DB][DB * DB], sD[DB][DB * DB], sT[DB][DB * DB];  // a warp's head: A, D, (I + A)^-1
    __shared__ int s_seq;
    pdl_begin();
    const int blk = blockIdx.x, g = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (threadIdx.x == 0) s_seq = -1;
    __syncthreads();
    for (int s = threadIdx.x; s < a.num_seqs; s += blockDim.x)
        if (first_block(a.q_start, s) <= blk && blk < first_block(a.q_start, s) + (a.q_start[s + 1] - a.q_start[s] + DB - 1) / DB) s_seq = s;
    __syncthreads();
    const int s = s_seq;
    if (s < 0) return;
    const int base = a.q_start[s] + (blk - first_block(a.q_start, s)) * DB;
    const int count = min(DB, a.q_start[s + 1] - base);
    const int per = a.heads / a.groups;
    // decays and betas of eight heads, a thread a (head, row); rows beyond the portion neither forget nor write
    auto gates = [&](int hh0) {
        const int hh = hh0 + threadIdx.x / DB, t = threadIdx.x % DB;
        if (threadIdx.x < DB * DB && hh < per) {
            const int h = g * per + hh;
            float decay = 1.0f, beta = 0.0f;
            if (t < count) {
                decay = decay_of(to_f32(((const AT*)a.a)[((size_t)base + t) * a.a_ld + h]), a.dt_bias[h], expf(a.a_log[h]));
                beta = sigmoid_of(to_f32(((const AT*)a.b)[((size_t)base + t) * a.b_ld + h]));
            }
            gs[hh - hh0][t] = decay;
            bs[hh - hh0][t] = beta;
        }
    };
    gates(0);
    // a warp a row: unit vectors (rows beyond the portion are zeros)
    const size_t row = (size_t)base + min(warp, count - 1);
    const bool mine = warp < count;
    const AT* qp = (const AT*)a.q + row * a.q_ld + (size_t)g * a.dim;
    const AT* kp = (const AT*)a.k + row * a.k_ld + (size_t)g * a.dim;
    float qv[PER], kv[PER];
    float qq = 0.0f, kn = 0.0f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int c = lane + 32 * i;
        const bool ok = mine && c < a.dim;
        qv[i] = ok ? to_f32(qp[c]) : 0.0f;
        kv[i] = ok ? to_f32(kp[c]) : 0.0f;
        qq += qv[i] * qv[i];
        kn += kv[i] * kv[i];
    }
    const float iq = rsqrtf(warp_sum(qq) + a.unit_eps) * a.q_scale, ik = rsqrtf(warp_sum(kn) + a.unit_eps);
    float* kq = a.kq + ((size_t)g * a.blocks + blk) * 2 * DB * a.dp;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int c = lane + 32 * i;
        qv[i] *= iq;
        kv[i] *= ik;
        ks[warp][c] = kv[i];
        if (c < a.dp) {
            kq[warp * a.dp + c] = kv[i];
            kq[(DB + warp) * a.dp + c] = qv[i];
        }
    }
    for (int c = 32 * PER + lane; c < a.dp; c += 32) kq[warp * a.dp + c] = kq[(DB + warp) * a.dp + c] = 0.0f;
    __syncthreads();
    // the products between the rows, row `warp` against all eight: sixteen sums, one exchange (lane l
    // ends up with sum l / 2: of k for l < 16, of q behind)
    {
        float x[2 * DB];
#pragma unroll
        for (int j = 0; j < DB; ++j) {
            x[j] = x[DB + j] = 0.0f;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const float other = ks[j][lane + 32 * i];
                x[j] = fmaf(kv[i], other, x[j]);
                x[DB + j] = fmaf(qv[i], other, x[DB + j]);
            }
        }
#pragma unroll
        for (int o = 16; o > 1; o >>= 1) {
            const bool upper = (lane & o) != 0;
#pragma unroll
            for (int i = 0; i < o / 2; ++i) {
                const float keep = upper ? x[i + o / 2] : x[i], send = upper ? x[i] : x[i + o / 2];
                x[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        }
        const float sum = x[0] + __shfl_xor_sync(0xffffffffu, x[0], 1);
        const int e = lane >> 1;
        if ((lane & 1) == 0) (e < DB ? kk : qk)[warp][e % DB] = sum;
    }
    for (int hh0 = 0; hh0 < per; hh0 += DB) {
        if (hh0 > 0) {
            __syncthreads();  // the heads before these are done with their gates
            gates(hh0);
        }
        __syncthreads();
        const int here = min(DB, per - hh0);
        if (warp < here) {  // a warp a head
            const int h = g * per + hh0 + warp;
            float *A = sA[warp], *D = sD[warp], *T = sT[warp];
            const float* gw = gs[warp];
#pragma unroll
            for (int e = lane; e < DB * DB; e += 32) {
                const int i = e / DB, j = e % DB;
                float d = 1.0f;  // g_(j+1) .. g_i
#pragma unroll
                for (int m = 1; m < DB; ++m)
                    if (m > j && m <= i) d *= gw[m];
                D[e] = d;
                A[e] = j < i ? bs[warp][i] * d * kk[i][j] : 0.0f;
            }
            __syncwarp();
            if (lane < DB) {  // column `lane` of (I + A)^-1
                float x[DB];
#pragma unroll
                for (int i = 0; i < DB; ++i) {
                    x[i] = i == lane ? 1.0f : 0.0f;
#pragma unroll
                    for (int j = 0; j < i; ++j) x[i] = fmaf(-A[i * DB + j], x[j], x[i]);
                    T[i * DB + lane] = x[i];
                }
            }
            __syncwarp();
            float* out = a.coef + ((size_t)h * a.blocks + blk) * DC;
#pragma unroll
            for (int e = lane; e < DB * DB; e += 32) {
                const int i = e / DB, j = e % DB;
                out[e] = D[(DB - 1) * DB + i] * T[e];
                float m = 0.0f;
#pragma unroll
                for (int l = 0; l < DB; ++l)  // (T is zero above the diagonal)
                    if (l <= i) m = fmaf(D[i * DB + l] * qk[i][l], T[l * DB + j], m);
                out[DB * DB + e] = m;
            }
            if (lane < DB) {
                const float so_far = D[lane * DB] * gw[0];
                out[2 * DB * DB + lane] = bs[warp][lane] * so_far;
                out[2 * DB * DB + DB + lane] = so_far;
                if (lane == DB - 1) out[2 * DB * DB + 2 * DB] = so_far;
            }
        }
        // beta v of these heads, by everybody
        for (int hh = 0; hh < here; ++hh) {
            const int h = g * per + hh0 + hh;
            const AT* vp = (const AT*)a.v + (size_t)base * a.v_ld + (size_t)h * a.vdim;
            float* bv = a.bv + ((size_t)h * a.blocks + blk) * a.chunks * DB * DB;
            for (int e = threadIdx.x; e < a.chunks * DB * DB; e += blockDim.x) {
                const int t = e / (a.chunks * DB), c = e - t * a.chunks * DB;
                bv[(c / DB) * DB * DB + t * DB + c % DB] = t < count && c < a.vdim ? bs[hh][t] * to_f32(vp[(size_t)t * a.v_ld + c]) : 0.0f;
            }
        }
    }
}

template <typename AT>
int launch_delta_prepare(const PrepareArgs& a, cudaStream_t stream) {
    const dim3 grid(a.blocks, a.groups);
    const int per = (a.dim + 31) / 32;
#define DP_GO(P) launch_kernel(delta_prepare_kernel<AT, P>, grid, DB * 32, 0, stream, a)
    if (per <= 1) DP_GO(1);
    else if (per <= 2) DP_GO(2);
    else if (per <= 4) DP_GO(4);
    else DP_GO(8);
#undef DP_GO
    return launch_status();
}

// --------------------------------------------------------------------------- the state, block after block

struct BlocksArgs {
    const float *kq, *coef, *bv;
    float* state;
    long long slot_stride;
    const int *q_start, *state_slots;
    float* out;  // [T, heads * vdim]
    int blocks, heads, groups, dim, vdim, chunks;
    int wide;  // a state row's four neighbouring columns may be moved at once
};

constexpr int D_STAGES = 3;

// A run of RUN neighbouring floats as pairs.
template <int RUN>
__device__ __forceinline__ void read_run(const float* p, uint64_t* pairs) {
    if constexpr (RUN == 4) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
        pairs[0] = v.x, pairs[1] = v.y;
    } else {
        pairs[0] = *reinterpret_cast<const uint64_t*>(p);
    }
}

// RPL: key rows a lane holds.  A warp holds four columns, half a chunk; a lane's rows come in runs of four
// (rows 128 j + 4 lane .. + 3, 16-byte words of shared memory) or, where RPL is no multiple of four, of two.
template <int RPL>
__global__ void __launch_bounds__(256) delta_blocks_kernel(const BlocksArgs a) {
    constexpr int DP = 32 * RPL, KQ = 2 * DB * DP, RUN = RPL % 4 == 0 ? 4 : 2;
    const int h = blockIdx.x, s = blockIdx.y, warps = blockDim.x >> 5;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad = warp & 1;
    const int chunk0 = blockIdx.z * (warps / 2), chunk = chunk0 + (warp >> 1);
    const int col0 = chunk * DB + quad * 4;
    const int dim = a.dim, vdim = a.vdim, g = h / (a.heads / a.groups);
    extern __shared__ __align__(16) float sm[];
    const int stage_floats = KQ + DC + warps / 2 * DB * DB;
    float* wsm = sm + D_STAGES * stage_floats + warp * 3 * DB * 4;  // this warp's w: [4 columns][8 rows]
    float* usm = wsm + DB * 4;                                      // and D_8 u: [8 rows][4 columns] twice over, (u, u)
    pdl_wait();
    const int first = a.q_start[s], n = a.q_start[s + 1] - first;
    if (n <= 0) return;
    const int nb = (n + DB - 1) / DB;
    const size_t blk0 = (size_t)first_block(a.q_start, s);
    const float* kq_src = a.kq + ((size_t)g * a.blocks + blk0) * KQ;
    const float* coef_src = a.coef + ((size_t)h * a.blocks + blk0) * DC;
    const float* bv_src = a.bv + (((size_t)h * a.blocks + blk0) * a.chunks + chunk0) * DB * DB;
    const int my_chunks = min(warps / 2, a.chunks - chunk0);
    auto load = [&](int b) {
        if (b < nb) {
            float* st = sm + (b % D_STAGES) * stage_floats;
            const float* src = kq_src + (size_t)b * KQ;
            for (int i = threadIdx.x; i < KQ / 4; i += blockDim.x) cp16(st + 4 * i, src + 4 * i);
            src = coef_src + (size_t)b * DC;
            for (int i = threadIdx.x; i < DC / 4; i += blockDim.x) cp16(st + KQ + 4 * i, src + 4 * i);
            src = bv_src + (size_t)b * a.chunks * DB * DB;
            for (int i = threadIdx.x; i < my_chunks * DB * DB / 4; i += blockDim.x) cp16(st + KQ + DC + 4 * i, src + 4 * i);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int b = 0; b < D_STAGES - 1; ++b) load(b);

    const bool live = chunk < a.chunks && col0 < vdim;
    float* slot = a.state + (size_t)a.state_slots[s] * a.slot_stride + (size_t)h * dim * vdim;
    uint64_t S[4][RPL / 2];
#pragma unroll
    for (int r = 0; r < RPL; r += 2) {
        float v[2][4];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int row = r / RUN * (32 * RUN) + lane * RUN + r % RUN + e;
            v[e][0] = v[e][1] = v[e][2] = v[e][3] = 0.0f;
            if (live && row < dim) {
                if (a.wide) {
                    const float4 x = *reinterpret_cast<const float4*>(slot + (size_t)row * vdim + col0);
                    v[e][0] = x.x, v[e][1] = x.y, v[e][2] = x.z, v[e][3] = x.w;
                } else {
#pragma unroll
                    for (int c = 0; c < 4; ++c)
                        if (col0 + c < vdim) v[e][c] = slot[(size_t)row * vdim + col0 + c];
                }
            }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) S[c][r / 2] = pair_of(v[0][c], v[1][c]);
    }
    const int tok = lane >> 2, mine = lane & 3;  // this lane's row and column between exchange and update
    float* out = a.out + (size_t)first * a.heads * vdim + (size_t)h * vdim + col0 + mine;
    const bool writes = chunk < a.chunks && col0 + mine < vdim;

    for (int b = 0; b < nb; ++b) {
        asm volatile("cp.async.wait_group %0;" ::"n"(D_STAGES - 2) : "memory");
        __syncthreads();  // block b has landed for everybody, and nobody reads block b - 1 any more
        load(b + D_STAGES - 1);
        const float* st = sm + (b % D_STAGES) * stage_floats;
        const float* kt = st + lane * RUN;  // row t's run j: kt[t * DP + 32 * RUN * j]
        const float* qt = kt + DB * DP;
        const float* coef = st + KQ;
        if (chunk < a.chunks) {
            // ---- S^T k and S^T q of the eight rows: this lane's share of 8 x 4 columns x 2.  Place t holds row
            // t ^ tok: the rows a lane keeps in the exchange stand in the first places whatever the lane
            float val[64];
#pragma unroll
            for (int t = 0; t < DB; ++t) {
                uint64_t K[RPL / 2], Q[RPL / 2];
#pragma unroll
                for (int j = 0; j < RPL / RUN; ++j) {
                    read_run<RUN>(kt + (t ^ tok) * DP + 32 * RUN * j, K + j * (RUN / 2));
                    read_run<RUN>(qt + (t ^ tok) * DP + 32 * RUN * j, Q + j * (RUN / 2));
                }
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    uint64_t p = mul2(S[c][0], K[0]), r = mul2(S[c][0], Q[0]);
#pragma unroll
                    for (int j = 1; j < RPL / 2; ++j) {
                        p = fma2(S[c][j], K[j], p);
                        r = fma2(S[c][j], Q[j], r);
                    }
                    float lo, hi;
                    halves_of(p, lo, hi);
                    val[(t * 4 + c) * 2] = lo + hi;
                    halves_of(r, lo, hi);
                    val[(t * 4 + c) * 2 + 1] = lo + hi;
                }
            }
            // ---- one exchange: every step sends half of what a lane still holds; lane l ends up with the sums 2 l and 2 l + 1
#pragma unroll
            for (int o = 16; o > 2; o >>= 1)  // over the rows
#pragma unroll
                for (int i = 0; i < 2 * o; ++i) val[i] += __shfl_xor_sync(0xffffffffu, val[i + 2 * o], o);
#pragma unroll
            for (int o = 2; o > 0; o >>= 1) {  // over the columns
                const bool upper = (lane & o) != 0;
#pragma unroll
                for (int i = 0; i < 2 * o; ++i) {
                    const float keep = upper ? val[i + 2 * o] : val[i], send = upper ? val[i] : val[i + 2 * o];
                    val[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
            // ---- the triangles: row `tok`, column `mine`
            const float bv = st[KQ + DC + (warp >> 1) * DB * DB + tok * DB + quad * 4 + mine];
            wsm[mine * DB + tok] = fmaf(-coef[2 * DB * DB + tok], val[0], bv);
            __syncwarp();
            float u = 0.0f, o = coef[2 * DB * DB + DB + tok] * val[1];
            const float4* t4 = reinterpret_cast<const float4*>(coef + tok * DB);
            const float4* m4 = reinterpret_cast<const float4*>(coef + DB * DB + tok * DB);
            const float4* w4 = reinterpret_cast<const float4*>(wsm + mine * DB);
#pragma unroll
            for (int j = 0; j < DB / 4; ++j) {
                const float4 t = t4[j], m = m4[j], x = w4[j];
                u = fmaf(t.x, x.x, fmaf(t.y, x.y, fmaf(t.z, x.z, fmaf(t.w, x.w, u))));
                o = fmaf(m.x, x.x, fmaf(m.y, x.y, fmaf(m.z, x.z, fmaf(m.w, x.w, o))));
            }
            *reinterpret_cast<float2*>(usm + (tok * 4 + mine) * 2) = make_float2(u, u);
            if (writes && b * DB + tok < n) out[(size_t)(b * DB + tok) * a.heads * vdim] = o;
            __syncwarp();
            // ---- the state
            const float last = coef[2 * DB * DB + 2 * DB];
            const uint64_t last2 = pair_of(last, last);
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
                for (int j = 0; j < RPL / 2; ++j) S[c][j] = mul2(S[c][j], last2);
#pragma unroll
            for (int t = 0; t < DB; ++t) {
                const ulonglong2* up = reinterpret_cast<const ulonglong2*>(usm + t * 4 * 2);
                const ulonglong2 ua = up[0], ub = up[1];
                const uint64_t u[4] = {ua.x, ua.y, ub.x, ub.y};
#pragma unroll
                for (int j = 0; j < RPL / RUN; ++j) {
                    uint64_t k2[RUN / 2];
                    read_run<RUN>(kt + t * DP + 32 * RUN * j, k2);
#pragma unroll
                    for (int i = 0; i < RUN / 2; ++i)
#pragma unroll
                        for (int c = 0; c < 4; ++c) S[c][j * (RUN / 2) + i] = fma2(k2[i], u[c], S[c][j * (RUN / 2) + i]);
                }
            }
        }
    }
    pdl_trigger();
    if (!live) return;
#pragma unroll
    for (int r = 0; r < RPL; r += 2) {
        float v[2][4];
#pragma unroll
        for (int c = 0; c < 4; ++c) halves_of(S[c][r / 2], v[0][c], v[1][c]);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int row = r / RUN * (32 * RUN) + lane * RUN + r % RUN + e;
            if (row >= dim) continue;
            if (a.wide) {
                *reinterpret_cast<float4*>(slot + (size_t)row * vdim + col0) = make_float4(v[e][0], v[e][1], v[e][2], v[e][3]);
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (col0 + c < vdim) slot[(size_t)row * vdim + col0 + c] = v[e][c];
            }
        }
    }
}

template <int RPL>
int launch_delta_blocks(const BlocksArgs& a, int num_seqs, int sm_count, cudaStream_t stream) {
    // a CTA's warps share the keys and queries they bring in: as many as leave a CTA for every SM, at least four
    int warps = 8;
    while (warps > 4 && (long long)a.heads * num_seqs * ((2 * a.chunks + warps - 1) / warps) < sm_count) warps /= 2;
    while (warps > 2 && warps / 2 >= 2 * a.chunks) warps /= 2;
    const size_t smem = (size_t)(D_STAGES * (2 * DB * 32 * RPL + DC + warps / 2 * DB * DB) + warps * 3 * DB * 4) * sizeof(float);
    auto kern = delta_blocks_kernel<RPL>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    // (without the dependent-launch attribute: CTAs that become resident under the tail of the kernel
    // before them pile up on the SMs that have room first, and a CTA here runs as long as the portion)
    kern<<<dim3(a.heads, num_seqs, (2 * a.chunks + warps - 1) / warps), dim3(warps * 32), smem, stream>>>(a);
    return launch_status();
}

// --------------------------------------------------------------------------- steps of single rows

struct StepArgs {
    const void *x, *gate, *b, *a;  // x: the columns [q | k | v] before their convolution
    long long ld;                  // between two rows of all four
    const float *taps, *dt_bias, *a_log, *norm_w;
    float *window, *state;
    long long window_stride, slot_stride;
    const int *q_start, *state_slots;
    void* out;
    long long out_ld;
    int heads, groups, dim, vdim, n_taps;
    float q_scale, unit_eps, eps;
};

constexpr int DS_THREADS = 256;
constexpr int DS_HELD = 16;  // state rows a thread keeps between its two passes

// One CTA per (group, sequence): the group's q and k channels and its heads' v channels are nobody
// else's, so their windows move on here.  N: value columns a thread takes at once.
template <typename AT, int N>
__global__ void __launch_bounds__(DS_THREADS, 2) delta_step_kernel(const StepArgs a) {
    __shared__ float scratch[33];
    __shared__ float red[2][DS_THREADS * N];
    extern __shared__ __align__(16) float ch[];  // q [dim], k [dim], v [heads of the group][vdim], then u and o of a head [vdim] each
    pdl_wait();
    const int g = blockIdx.x, s = blockIdx.y, tid = threadIdx.x;
    const int row = a.q_start[s];
    if (a.q_start[s + 1] <= row) return;
    const int dim = a.dim, vdim = a.vdim, per = a.heads / a.groups, channels = 2 * a.groups * dim + a.heads * vdim;
    const int slot = a.state_slots[s], mine = 2 * dim + per * vdim;
    float* su = ch + mine;
    float* so = su + vdim;
    const AT* x = (const AT*)a.x + (size_t)row * a.ld;
    float* window = a.window + (size_t)slot * a.window_stride;
    float qq = 0.0f, kn = 0.0f;
    for (int i = tid; i < mine; i += DS_THREADS) {
        const int c = i < dim ? g * dim + i : i < 2 * dim ? (a.groups + g) * dim + i - dim : 2 * a.groups * dim + g * per * vdim + i - 2 * dim;
        const float* taps = a.taps + (size_t)c * a.n_taps;
        const float in = to_f32(x[c]);
        float acc = taps[a.n_taps - 1] * in;
        for (int j = 0; j < a.n_taps - 1; ++j) {
            float* at = window + (size_t)j * channels + c;
            acc = fmaf(taps[j], *at, acc);
            if (j > 0) at[-(long long)channels] = *at;
        }
        window[(size_t)(a.n_taps - 2) * channels + c] = in;
        acc = to_f32(from_f32<AT>(silu_of(acc)));  // (rounded where the convolution's own kernel rounds)
        ch[i] = acc;
        if (i < dim) qq += acc * acc;
        else if (i < 2 * dim) kn += acc * acc;
    }
    qq = block_sum(qq, scratch);
    kn = block_sum(kn, scratch);
    const float iq = rsqrtf(qq + a.unit_eps) * a.q_scale, ik = rsqrtf(kn + a.unit_eps);
    float qk = 0.0f;
    for (int i = tid; i < dim; i += DS_THREADS) {
        const float q = ch[i] * iq, k = ch[dim + i] * ik;
        ch[i] = q;
        ch[dim + i] = k;
        qk += q * k;
    }
    qk = block_sum(qk, scratch);  // (its barriers stand between the writes above and the reads below)
    const float *sq = ch, *sk = ch + dim;
    const int spans = (vdim + N - 1) / N;
    const int lanes = min(spans, DS_THREADS), parts = DS_THREADS / lanes;  // threads over the columns, and shares of the key rows
    const int span = tid % lanes, part = tid / lanes;
    for (int hh = 0; hh < per; ++hh) {
        const int h = g * per + hh;
        const float decay = decay_of(to_f32(((const AT*)a.a)[(size_t)row * a.ld + h]), a.dt_bias[h], expf(a.a_log[h]));
        const float beta = sigmoid_of(to_f32(((const AT*)a.b)[(size_t)row * a.ld + h]));
        const float* sv = ch + 2 * dim + hh * vdim;
        float* S = a.state + (size_t)slot * a.slot_stride + (size_t)h * dim * vdim;
        for (int base = 0; base < spans; base += lanes) {
            const int c0 = (base + span) * N;
            const bool live = part < parts && base + span < spans;
            auto fetch = [&](int r, float (&v)[N]) {
                if constexpr (N == 4) {
                    const float4 f = *reinterpret_cast<const float4*>(S + (size_t)r * vdim + c0);
                    v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
                } else {
                    v[0] = S[(size_t)r * vdim + c0];
                }
            };
            float held[DS_HELD][N], p[N], o[N];
#pragma unroll
            for (int e = 0; e < N; ++e) p[e] = o[e] = 0.0f;
            if (live) {
#pragma unroll
                for (int i = 0; i < DS_HELD; ++i) {
                    const int r = part + i * parts;
#pragma unroll
                    for (int e = 0; e < N; ++e) held[i][e] = 0.0f;
                    if (r < dim) fetch(r, held[i]);
                }
#pragma unroll
                for (int i = 0; i < DS_HELD; ++i) {
                    const int r = part + i * parts;
                    const float k = r < dim ? sk[r] : 0.0f, q = r < dim ? sq[r] : 0.0f;
#pragma unroll
                    for (int e = 0; e < N; ++e) p[e] = fmaf(held[i][e], k, p[e]), o[e] = fmaf(held[i][e], q, o[e]);
                }
                for (int r = part + DS_HELD * parts; r < dim; r += parts) {
                    float v[N];
                    fetch(r, v);
#pragma unroll
                    for (int e = 0; e < N; ++e) p[e] = fmaf(v[e], sk[r], p[e]), o[e] = fmaf(v[e], sq[r], o[e]);
                }
#pragma unroll
                for (int e = 0; e < N; ++e) red[0][(part * lanes + span) * N + e] = p[e], red[1][(part * lanes + span) * N + e] = o[e];
            }
            __syncthreads();
            for (int i = tid; i < lanes * N; i += DS_THREADS) {
                const int c = base * N + i;
                if (c >= vdim) continue;
                float ps = 0.0f, os = 0.0f;
                for (int j = 0; j < parts; ++j) ps += red[0][j * lanes * N + i], os += red[1][j * lanes * N + i];
                const float u = beta * fmaf(-decay, ps, sv[c]);
                su[c] = u;
                so[c] = fmaf(u, qk, decay * os);
            }
            __syncthreads();
            if (live) {
                float u[N];
#pragma unroll
                for (int e = 0; e < N; ++e) u[e] = su[c0 + e];
                auto put = [&](int r, const float (&v)[N]) {
                    const float k = sk[r];
                    if constexpr (N == 4)
                        *reinterpret_cast<float4*>(S + (size_t)r * vdim + c0) =
                            make_float4(fmaf(k, u[0], decay * v[0]), fmaf(k, u[1], decay * v[1]), fmaf(k, u[2], decay * v[2]), fmaf(k, u[3], decay * v[3]));
                    else
                        S[(size_t)r * vdim + c0] = fmaf(k, u[0], decay * v[0]);
                };
#pragma unroll
                for (int i = 0; i < DS_HELD; ++i) {
                    const int r = part + i * parts;
                    if (r < dim) put(r, held[i]);
                }
                for (int r = part + DS_HELD * parts; r < dim; r += parts) {
                    float v[N];
                    fetch(r, v);
                    put(r, v);
                }
            }
        }
        // the head's output norm and gate
        float ss = 0.0f;
        for (int c = tid; c < vdim; c += DS_THREADS) ss += so[c] * so[c];
        const float inv = rsqrtf(block_sum(ss, scratch) / (float)vdim + a.eps);
        const AT* gate = (const AT*)a.gate + (size_t)row * a.ld + (size_t)h * vdim;
        AT* out = (AT*)a.out + (size_t)row * a.out_ld + (size_t)h * vdim;
        for (int c = tid; c < vdim; c += DS_THREADS) out[c] = from_f32<AT>(so[c] * inv * a.norm_w[c] * silu_of(to_f32(gate[c])));
        __syncthreads();  // u, o and the shares are written again by the next head
    }
    pdl_trigger();
}

template <typename AT>
int launch_delta_step(const StepArgs& a, int num_seqs, cudaStream_t stream) {
    const size_t smem = (size_t)(2 * a.dim + (a.heads / a.groups + 2) * a.vdim) * sizeof(float);
    if (smem > 160 * 1024) return SHISO_ERR_SHAPE;
    const bool wide = a.vdim % 4 == 0 && a.slot_stride % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    auto kern = wide ? delta_step_kernel<AT, 4> : delta_step_kernel<AT, 1>;
    if (smem > 32 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_kernel(kern, dim3(a.groups, num_seqs), dim3(DS_THREADS), smem, stream, a);
    return launch_status();
}

// --------------------------------------------------------------------------- output norm and gate

// out[t, h, c] = x[t, h, c] / sqrt(mean_c(x^2) + eps) * w[c] * silu(gate[t, h, c]).  `group` lanes (a
// power of two) a (row, head), each with four neighbouring columns at a time (N = 4) or one.
template <typename AT, int N>
__global__ void __launch_bounds__(256)
delta_output_kernel(const float* __restrict__ x, const AT* __restrict__ gate, long long gate_ld, const float* __restrict__ w,
                    AT* __restrict__ out, long long out_ld, int tokens, int heads, int vdim, int group, float eps) {
    pdl_begin();
    const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / group;
    const int sub = threadIdx.x % group;
    const bool live = item < (long long)tokens * heads;
    const int t = live ? (int)(item / heads) : 0, h = live ? (int)(item % heads) : 0;
    const float* xr = x + ((size_t)t * heads + h) * vdim;
    const AT* gr = gate + (size_t)t * gate_ld + (size_t)h * vdim;
    AT* o = out + (size_t)t * out_ld + (size_t)h * vdim;
    float ss = 0.0f;
    for (int c = sub * N; c < vdim; c += group * N) {
        if constexpr (N == 4) {
            const float4 v = *reinterpret_cast<const float4*>(xr + c);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        } else {
            ss += xr[c] * xr[c];
        }
    }
    for (int off = group >> 1; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    if (!live) return;
    const float inv = rsqrtf(ss / (float)vdim + eps);
    for (int c = sub * N; c < vdim; c += group * N) {
        if constexpr (N == 4) {
            const float4 v = *reinterpret_cast<const float4*>(xr + c), wv = *reinterpret_cast<const float4*>(w + c);
            if constexpr (sizeof(AT) == 2) {
                const uint2 raw = *reinterpret_cast<const uint2*>(gr + c);
                const float g0 = __uint_as_float(raw.x << 16), g1 = __uint_as_float(raw.x & 0xffff0000u);
                const float g2 = __uint_as_float(raw.y << 16), g3 = __uint_as_float(raw.y & 0xffff0000u);
                const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x * inv * wv.x * silu_sfu(g0), v.y * inv * wv.y * silu_sfu(g1));
                const __nv_bfloat162 hi = __floats2bfloat162_rn(v.z * inv * wv.z * silu_sfu(g2), v.w * inv * wv.w * silu_sfu(g3));
                *reinterpret_cast<uint2*>(o + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            } else {
                const float4 gv = *reinterpret_cast<const float4*>(gr + c);
                *reinterpret_cast<float4*>(o + c) = make_float4(v.x * inv * wv.x * silu_of(gv.x), v.y * inv * wv.y * silu_of(gv.y),
                                                                v.z * inv * wv.z * silu_of(gv.z), v.w * inv * wv.w * silu_of(gv.w));
            }
        } else {
            o[c] = from_f32<AT>(xr[c] * inv * w[c] * silu_of(to_f32(gr[c])));
        }
    }
}

}  // namespace


// q, k [T, groups * dim], v [T, heads * vdim], b, a [T, heads] (rows may be strided, `*_ld` elements
// apart); state float [slots, heads, dim, vdim]; out float [T, heads * vdim]; scratch: 16-byte aligned.
SHISO_API int shiso_delta_rule(const void* q, const void* k, const void* v, const void* b, const void* a_logit, long long q_ld,
                               long long k_ld, long long v_ld, long long b_ld, long long a_ld, int act_dtype, const float* dt_bias,
                               const float* a_log, float* state, long long slot_stride, const int* q_start, const int* state_slots,
                               float* scratch, float* out, int tokens, int num_seqs, int heads, int groups, int dim, int vdim,
                               float q_scale, float unit_eps, int sm_count, cudaStream_t stream) {
    if (tokens <= 0 || num_seqs <= 0) return SHISO_OK;
    if (heads <= 0 || groups <= 0 || heads % groups || dim <= 0 || dim > D_MAX_DIM || vdim <= 0 || num_seqs > 65535 || groups > 65535)
        return SHISO_ERR_SHAPE;
    if (((uintptr_t)scratch | (uintptr_t)out) & 15) return SHISO_ERR_ALIGN;
    const int blocks = tokens / DB + num_seqs, dp = (dim + 63) / 64 * 64, chunks = (vdim + DB - 1) / DB;
    float* kq = scratch;
    float* coef = kq + (size_t)groups * blocks * 2 * DB * dp;
    float* bv = coef + (size_t)heads * blocks * DC;
    const PrepareArgs prep = {q, k, v, b, a_logit, q_ld, k_ld, v_ld, b_ld, a_ld, dt_bias, a_log, q_start, kq, coef, bv,
                              num_seqs, blocks, heads, groups, dim, dp, vdim, chunks, q_scale, unit_eps};
    int status = SHISO_ERR_DTYPE;
    if (act_dtype == SHISO_F32) status = launch_delta_prepare<float>(prep, stream);
    else if (act_dtype == SHISO_BF16) status = launch_delta_prepare<__nv_bfloat16>(prep, stream);
    if (status != SHISO_OK) return status;
    const int wide = vdim % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    const BlocksArgs walk = {kq, coef, bv, state, slot_stride, q_start, state_slots, out, blocks, heads, groups, dim, vdim, chunks, wide};
    switch (dp) {
        case 64: return launch_delta_blocks<2>(walk, num_seqs, sm_count, stream);
        case 128: return launch_delta_blocks<4>(walk, num_seqs, sm_count, stream);
        case 192: return launch_delta_blocks<6>(walk, num_seqs, sm_count, stream);
        default: return launch_delta_blocks<8>(walk, num_seqs, sm_count, stream);
    }
}

// A step of one row per sequence.  x: the columns [q | k | v] of the projected rows, gate, b and a further
// columns of the same rows (`ld` elements apart); taps float [channels, n_taps]; window float
// [slots, n_taps - 1, channels]; out [T, heads * vdim], rows out_ld apart.
SHISO_API int shiso_delta_step(const void* x, const void* gate, const void* b, const void* a_logit, long long ld, int act_dtype,
                               const float* taps, const float* dt_bias, const float* a_log, const float* norm_w, float* window,
                               long long window_stride, float* state, long long slot_stride, const int* q_start,
                               const int* state_slots, void* out, long long out_ld, int num_seqs, int heads, int groups, int dim,
                               int vdim, int n_taps, float q_scale, float unit_eps, float eps, cudaStream_t stream) {
    if (num_seqs <= 0) return SHISO_OK;
    if (heads <= 0 || groups <= 0 || heads % groups || dim <= 0 || vdim <= 0 || n_taps < 2 || num_seqs > 65535) return SHISO_ERR_SHAPE;
    const StepArgs args = {x, gate, b, a_logit, ld, taps, dt_bias, a_log, norm_w, window, state, window_stride, slot_stride, q_start,
                           state_slots, out, out_ld, heads, groups, dim, vdim, n_taps, q_scale, unit_eps, eps};
    if (act_dtype == SHISO_F32) return launch_delta_step<float>(args, num_seqs, stream);
    if (act_dtype == SHISO_BF16) return launch_delta_step<__nv_bfloat16>(args, num_seqs, stream);
    return SHISO_ERR_DTYPE;
}

SHISO_API int shiso_delta_output(const float* x, const void* gate, long long gate_ld, int act_dtype, const float* w, void* out,
                                 long long out_ld, int tokens, int heads, int vdim, float eps, cudaStream_t stream) {
    if (tokens <= 0) return SHISO_OK;
    if (heads <= 0 || vdim <= 0) return SHISO_ERR_SHAPE;
    const uintptr_t all = (uintptr_t)x | (uintptr_t)gate | (uintptr_t)w | (uintptr_t)out;
    const bool wide = vdim % 4 == 0 && gate_ld % 4 == 0 && out_ld % 4 == 0 && (all & 15) == 0;
    const int n = wide ? 4 : 1;
    int group = 1;
    while (group < 32 && group * n < vdim) group *= 2;
    const unsigned blocks = ceil_div_u((long long)tokens * heads * group, 256);
#define DO_GO(AT, N) \
    launch_kernel(delta_output_kernel<AT, N>, blocks, 256, 0, stream, x, (const AT*)gate, gate_ld, w, (AT*)out, out_ld, tokens, heads, vdim, group, eps)
    if (act_dtype == SHISO_F32) {
        if (wide) DO_GO(float, 4);
        else DO_GO(float, 1);
    } else if (act_dtype == SHISO_BF16) {
        if (wide) DO_GO(__nv_bfloat16, 4);
        else DO_GO(__nv_bfloat16, 1);
    } else {
        return SHISO_ERR_DTYPE;
    }
#undef DO_GO
    return launch_status();
}
