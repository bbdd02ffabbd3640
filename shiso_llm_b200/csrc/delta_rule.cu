// The gated delta rule: a matrix state S[dim, vdim] per head that forgets by a factor g and is
// corrected towards each new value,
//
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q,
//
// with q and k brought to unit length per head (q times q_scale as well), beta = sigmoid(b) and
// g = exp(-exp(a_log_h) softplus(a + dt_bias_h)) from one logit each per row and head.  q and k may
// be shared by the heads of a group (head h reads group h / (heads / groups)).
//
// A column of S needs both S^T k and S^T q; they are taken in ONE pass over the old state, since
//     u = beta (v - g p),   o = g r + u (k . q)   with p = S_old^T k, r = S_old^T q,
// so a row costs one exchange across lanes, not two that wait for one another.
//
// delta_rule_kernel: one CTA walks the rows of one (head, sequence, range of value columns) in
// order.  Eight lanes hold a column, each dim / 8 of its rows in runs of four (rows 32 j + 4 lane .. + 3:
// 16-byte words of shared memory, eight lanes a full 128-byte line, the columns of a warp reading the
// same words), as pairs of floats for the two-wide multiply-add.  What is added to what depends on
// dim only - never on how the sequence was cut into steps, on the batch, or on how many columns a CTA
// was given.  Four warps that hold no state stage the rows sixteen at a time, a warp a row: copies
// (cp.async) of the rows after next are on their way while the next are normalised and the current
// ones walked; outputs leave through shared memory, written by the same warps.
//
// delta_output_kernel: each head's float outputs divided by their root mean square, times a weight
// shared by the heads, times silu(gate).
//
// delta_step_kernel: a step of single rows (decode) in ONE launch: the causal convolutions of q, k and
// v with silu and their windows, unit vectors, the state, the output norm and the gate.
#include "common.cuh"

namespace {

constexpr int DR_ROWS = 16;      // rows a stage holds
constexpr int DR_STAGERS = 128;  // threads behind the ones that hold state
constexpr int DR_STAGE_WARPS = DR_STAGERS / 32;

struct DeltaArgs {
    const void *q, *k, *v, *b, *a;
    long long q_ld, k_ld, v_ld, b_ld, a_ld;
    const float *dt_bias, *a_log;
    float* state;
    long long slot_stride;
    const int *q_start, *state_slots;
    float* out;
    int heads, groups, dim, vdim, cols;
    int bulk;  // rows may be fetched 16 bytes at a time (widths, strides and addresses allow it)
    float q_scale, unit_eps;
};

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

__device__ __forceinline__ void cp16(void* dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}

__device__ __forceinline__ float decay_of(float a_logit, float dt_bias, float rate) {
    const float z = a_logit + dt_bias;
    const float softplus = z > 20.0f ? z : log1pf(expf(z));
    return expf(-rate * softplus);
}
__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_of(float z) { return z / (1.0f + expf(-z)); }

// RPT: key rows a lane holds (dim rounded up to a multiple of 32, divided by 8).
template <typename AT, int RPT>
__global__ void __launch_bounds__(RPT > 16 ? 256 : RPT > 8 ? 384 : 640) delta_rule_kernel(const DeltaArgs a) {
    constexpr int DP = 8 * RPT;  // key rows with padding (zeros: their state stays zero)
    constexpr int EPV = 16 / (int)sizeof(AT);
    const int h = blockIdx.x, s = blockIdx.y, col0 = blockIdx.z * a.cols;
    const int workers = a.cols * 8;
    const bool stager = (int)threadIdx.x >= workers;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int part = lane & 7, local = warp * 4 + (lane >> 3), col = col0 + local;
    const int dim = a.dim, vdim = a.vdim, cols = a.cols, g = h / (a.heads / a.groups);
    extern __shared__ __align__(16) float sm[];
    // two stages: q [ROWS][DP], k [ROWS][DP], v [ROWS][cols], (g, beta, k . q, -) [ROWS][4]; two blocks of outputs
    // [ROWS][cols]; two raw areas: q [ROWS][dim], k [ROWS][dim], v [ROWS][cols] as they came
    const int stage_floats = DR_ROWS * (2 * DP + cols + 4);
    float* outs = sm + 2 * stage_floats;
    AT* raw = reinterpret_cast<AT*>(outs + 2 * DR_ROWS * cols);
    const int raw_elems = DR_ROWS * (2 * dim + cols);
    __shared__ float logits[2][DR_ROWS][2];
    const float rate = expf(a.a_log[h]), dt_bias = a.dt_bias[h];
    pdl_wait();
    const int first = a.q_start[s], n = a.q_start[s + 1] - first;
    if (n <= 0) return;
    const int batches = (n + DR_ROWS - 1) / DR_ROWS;
    const AT* qp = (const AT*)a.q + (size_t)first * a.q_ld + (size_t)g * dim;
    const AT* kp = (const AT*)a.k + (size_t)first * a.k_ld + (size_t)g * dim;
    const AT* vp = (const AT*)a.v + (size_t)first * a.v_ld + (size_t)h * vdim + col0;

    if (stager) {
        const int me = (int)threadIdx.x - workers, mywarp = me >> 5;
        const AT* bp = (const AT*)a.b + (size_t)first * a.b_ld + h;
        const AT* ap = (const AT*)a.a + (size_t)first * a.a_ld + h;
        float* op = a.out + (size_t)first * a.heads * vdim + (size_t)h * vdim + col0;
        float b_logit = 0.0f, a_logit = 0.0f;
        auto fetch = [&](int batch) {
            const int base = batch * DR_ROWS, count = min(DR_ROWS, n - base);
            if (a.bulk) {
                AT* rq = raw + (batch & 1) * raw_elems;
                AT* rk = rq + DR_ROWS * dim;
                AT* rv = rk + DR_ROWS * dim;
                const int pieces = dim / EPV, vpieces = cols / EPV;
                for (int i = me; i < DR_ROWS * pieces; i += DR_STAGERS) {
                    const int t = i / pieces, c = (i - t * pieces) * EPV;
                    const bool ok = t < count;
                    cp16(rq + t * dim + c, ok ? qp + (size_t)(base + t) * a.q_ld + c : qp, ok);
                    cp16(rk + t * dim + c, ok ? kp + (size_t)(base + t) * a.k_ld + c : kp, ok);
                }
                for (int i = me; i < DR_ROWS * vpieces; i += DR_STAGERS) {
                    const int t = i / vpieces, c = (i - t * vpieces) * EPV;
                    const bool ok = t < count && col0 + c < vdim;
                    cp16(rv + t * cols + c, ok ? vp + (size_t)(base + t) * a.v_ld + c : vp, ok);
                }
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
            if (me < count) {
                b_logit = to_f32(bp[(size_t)(base + me) * a.b_ld]);
                a_logit = to_f32(ap[(size_t)(base + me) * a.a_ld]);
            }
        };
        auto convert = [&](int batch) {  // a warp a row
            const int base = batch * DR_ROWS, count = min(DR_ROWS, n - base);
            const AT* rq = raw + (batch & 1) * raw_elems;
            const AT* rk = rq + DR_ROWS * dim;
            const AT* rv = rk + DR_ROWS * dim;
            float* sq = sm + (batch & 1) * stage_floats;
            float* sk = sq + DR_ROWS * DP;
            float* sv = sk + DR_ROWS * DP;
            float* sc = sv + DR_ROWS * cols;
            for (int t = mywarp; t < count; t += DR_STAGE_WARPS) {
                const AT* q_row = a.bulk ? rq + t * dim : qp + (size_t)(base + t) * a.q_ld;
                const AT* k_row = a.bulk ? rk + t * dim : kp + (size_t)(base + t) * a.k_ld;
                const AT* v_row = a.bulk ? rv + t * cols : vp + (size_t)(base + t) * a.v_ld;
                float qv[RPT / 4], kv[RPT / 4];
                float qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
                for (int i = 0; i < RPT / 4; ++i) {
                    const int c = lane + 32 * i;
                    qv[i] = c < dim ? to_f32(q_row[c]) : 0.0f;
                    kv[i] = c < dim ? to_f32(k_row[c]) : 0.0f;
                    qq += qv[i] * qv[i];
                    kk += kv[i] * kv[i];
                    qk += qv[i] * kv[i];
                }
                qq = warp_sum(qq);
                kk = warp_sum(kk);
                qk = warp_sum(qk);
                const float iq = rsqrtf(qq + a.unit_eps) * a.q_scale, ik = rsqrtf(kk + a.unit_eps);
#pragma unroll
                for (int i = 0; i < RPT / 4; ++i) {
                    sq[t * DP + lane + 32 * i] = qv[i] * iq;
                    sk[t * DP + lane + 32 * i] = kv[i] * ik;
                }
                for (int c = lane; c < cols; c += 32) sv[t * cols + c] = col0 + c < vdim ? to_f32(v_row[c]) : 0.0f;
                if (lane == 0)
                    *reinterpret_cast<float4*>(sc + t * 4) = make_float4(decay_of(logits[batch & 1][t][1], dt_bias, rate),
                                                                         sigmoid_of(logits[batch & 1][t][0]), qk * iq * ik, 0.0f);
            }
        };
        auto flush = [&](int batch) {
            const int base = batch * DR_ROWS, count = min(DR_ROWS, n - base);
            const float* so = outs + (batch & 1) * DR_ROWS * cols;
            for (int i = me; i < count * cols; i += DR_STAGERS) {
                const int t = i / cols, c = i - t * cols;
                if (col0 + c < vdim) op[(size_t)(base + t) * a.heads * vdim + c] = so[i];
            }
        };
        fetch(0);
        for (int batch = 0; batch < batches; ++batch) {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            if (me < DR_ROWS) logits[batch & 1][me][0] = b_logit, logits[batch & 1][me][1] = a_logit;
            asm volatile("bar.sync 1, %0;" ::"n"(DR_STAGERS) : "memory");
            // (the other raw area was converted before the last of the block's barriers)
            if (batch + 1 < batches) fetch(batch + 1);
            convert(batch);
            if (batch >= 2) flush(batch - 2);
            __syncthreads();  // this batch is staged; the batch before it has been walked
        }
        if (batches >= 2) flush(batches - 2);
        __syncthreads();
        flush(batches - 1);
        pdl_trigger();
        return;
    }

    const bool live = col < vdim;
    float* slot = a.state + (size_t)a.state_slots[s] * a.slot_stride + (size_t)h * dim * vdim;
    uint64_t S[RPT / 2];
#pragma unroll
    for (int r = 0; r < RPT; r += 2) {
        const int row = (r >> 2) * 32 + part * 4 + (r & 3);
        S[r / 2] = pair_of(live && row < dim ? slot[(size_t)row * vdim + col] : 0.0f,
                           live && row + 1 < dim ? slot[(size_t)(row + 1) * vdim + col] : 0.0f);
    }
    for (int batch = 0; batch < batches; ++batch) {
        __syncthreads();
        const int count = min(DR_ROWS, n - batch * DR_ROWS);
        const float* sq = sm + (batch & 1) * stage_floats;
        const float* sk = sq + DR_ROWS * DP;
        const float* sv = sk + DR_ROWS * DP + local;
        const float4* sc = reinterpret_cast<const float4*>(sk + DR_ROWS * DP + DR_ROWS * cols);
        float* so = outs + (batch & 1) * DR_ROWS * cols + local;
        const ulonglong2* kt = reinterpret_cast<const ulonglong2*>(sk) + part;
        const ulonglong2* qt = reinterpret_cast<const ulonglong2*>(sq) + part;
        uint64_t K[RPT / 2], Q[RPT / 2];
#pragma unroll
        for (int j = 0; j < RPT / 4; ++j) {
            const ulonglong2 k2 = kt[8 * j], q2 = qt[8 * j];
            K[2 * j] = k2.x, K[2 * j + 1] = k2.y;
            Q[2 * j] = q2.x, Q[2 * j + 1] = q2.y;
        }
#pragma unroll 2
        for (int t = 0; t < count; ++t) {
            uint64_t p0 = 0, p1 = 0, r0 = 0, r1 = 0;  // (pairs of zeros)
#pragma unroll
            for (int j = 0; j < RPT / 2; j += 2) {
                p0 = fma2(S[j], K[j], p0);
                r0 = fma2(S[j], Q[j], r0);
                p1 = fma2(S[j + 1], K[j + 1], p1);
                r1 = fma2(S[j + 1], Q[j + 1], r1);
            }
            const float4 c4 = sc[t];  // decay, beta, k . q
            const float v = sv[t * cols];
            // the next row's keys and queries are asked for under the exchange below
            uint64_t Kn[RPT / 2];
            const int next = min(t + 1, count - 1);
#pragma unroll
            for (int j = 0; j < RPT / 4; ++j) {
                const ulonglong2 k2 = kt[next * (DP / 4) + 8 * j], q2 = qt[next * (DP / 4) + 8 * j];
                Kn[2 * j] = k2.x, Kn[2 * j + 1] = k2.y;
                Q[2 * j] = q2.x, Q[2 * j + 1] = q2.y;
            }
            float pa, pb, pc, pd, ra, rb, rc, rd;
            halves_of(p0, pa, pb);
            halves_of(p1, pc, pd);
            halves_of(r0, ra, rb);
            halves_of(r1, rc, rd);
            float p = (pa + pb) + (pc + pd), r = (ra + rb) + (rc + rd);
#pragma unroll
            for (int o = 1; o < 8; o <<= 1) {
                p += __shfl_xor_sync(0xffffffffu, p, o);
                r += __shfl_xor_sync(0xffffffffu, r, o);
            }
            const float u = c4.y * fmaf(-c4.x, p, v);
            if (part == 0) so[t * cols] = fmaf(u, c4.z, c4.x * r);
            const uint64_t u2 = pair_of(u, u), g2 = pair_of(c4.x, c4.x);
#pragma unroll
            for (int j = 0; j < RPT / 2; ++j) S[j] = fma2(K[j], u2, mul2(g2, S[j]));
#pragma unroll
            for (int j = 0; j < RPT / 2; ++j) K[j] = Kn[j];
        }
    }
    __syncthreads();
    pdl_trigger();
#pragma unroll
    for (int r = 0; r < RPT; r += 2) {
        const int row = (r >> 2) * 32 + part * 4 + (r & 3);
        float lo, hi;
        halves_of(S[r / 2], lo, hi);
        if (live && row < dim) slot[(size_t)row * vdim + col] = lo;
        if (live && row + 1 < dim) slot[(size_t)(row + 1) * vdim + col] = hi;
    }
}

template <typename AT>
int launch_delta_rule(const DeltaArgs& args, int num_seqs, int sm_count, cudaStream_t stream) {
    DeltaArgs a = args;
    const int rpt = (a.dim + 31) / 32 * 4;  // key rows in runs of 32: four to each of a column's eight lanes
    // value columns per CTA: fewer while SMs would stay idle, but at least 16 (every CTA's staging
    // warps bring and normalise its head's keys and queries themselves), or what the head has
    int cols = rpt > 16 ? 16 : rpt > 8 ? 32 : 64;  // (the registers of a lane bound the block)
    while (cols > 16 && (long long)a.heads * num_seqs * ((a.vdim + cols - 1) / cols) < sm_count) cols /= 2;
    while (cols > 8 && cols / 2 >= a.vdim) cols /= 2;
    a.cols = cols;
    const int epv = 16 / (int)sizeof(AT);
    a.bulk = a.dim % epv == 0 && a.vdim % epv == 0 && a.q_ld % epv == 0 && a.k_ld % epv == 0 && a.v_ld % epv == 0 &&
             (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v) & 15) == 0;
    const dim3 grid(a.heads, num_seqs, (a.vdim + cols - 1) / cols), block(cols * 8 + DR_STAGERS);
#define DR_CASE(R)                                                                                                    \
    if (rpt <= R) {                                                                                                   \
        const size_t smem = (size_t)2 * DR_ROWS * (2 * 8 * R + cols + 4 + cols) * sizeof(float) +                     \
                            (size_t)2 * DR_ROWS * (2 * a.dim + cols) * sizeof(AT);                                    \
        auto kern = delta_rule_kernel<AT, R>;                                                                         \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
        launch_kernel(kern, grid, block, smem, stream, a);                                                            \
        return launch_status();                                                                                       \
    }
    DR_CASE(4) DR_CASE(8) DR_CASE(12) DR_CASE(16) DR_CASE(24) DR_CASE(32)
#undef DR_CASE
    return SHISO_ERR_SHAPE;
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
                const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x * inv * wv.x * silu_of(g0), v.y * inv * wv.y * silu_of(g1));
                const __nv_bfloat162 hi = __floats2bfloat162_rn(v.z * inv * wv.z * silu_of(g2), v.w * inv * wv.w * silu_of(g3));
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
// apart); state float [slots, heads, dim, vdim]; out float [T, heads * vdim].
SHISO_API int shiso_delta_rule(const void* q, const void* k, const void* v, const void* b, const void* a_logit, long long q_ld,
                               long long k_ld, long long v_ld, long long b_ld, long long a_ld, int act_dtype, const float* dt_bias,
                               const float* a_log, float* state, long long slot_stride, const int* q_start, const int* state_slots,
                               float* out, int tokens, int num_seqs, int heads, int groups, int dim, int vdim, float q_scale,
                               float unit_eps, int sm_count, cudaStream_t stream) {
    if (tokens <= 0 || num_seqs <= 0) return SHISO_OK;
    if (heads <= 0 || groups <= 0 || heads % groups || dim <= 0 || dim > 256 || vdim <= 0 || num_seqs > 65535) return SHISO_ERR_SHAPE;
    const DeltaArgs args = {q, k, v, b, a_logit, q_ld, k_ld, v_ld, b_ld, a_ld, dt_bias, a_log, state, slot_stride,
                            q_start, state_slots, out, heads, groups, dim, vdim, 0, 0, q_scale, unit_eps};
    if (act_dtype == SHISO_F32) return launch_delta_rule<float>(args, num_seqs, sm_count, stream);
    if (act_dtype == SHISO_BF16) return launch_delta_rule<__nv_bfloat16>(args, num_seqs, sm_count, stream);
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
