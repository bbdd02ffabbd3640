// A matrix memory with exponential gating: per head a state S[dim, vdim], a normaliser n[dim] and a running
// maximum m, all float and carried per request,
//
//     i = cap tanh(zi / cap),  f = log sigmoid(cap tanh(zf / cap)),  m' = max(f + m, i),
//     S <- e^(f + m - m') S + e^(i - m') k v^T,   n <- e^(f + m - m') n + e^(i - m') k,
//     o = S^T (s q) / (max(|n . s q|, e^-m') + denominator_eps)       (s: the queries' scale)
//
// and the mixer's output o / rms(o) * w * sigmoid(gate), head by head.
//
//   memory_gates_kernel   the two factors e^(f + m - m') and e^(i - m') of every row and head, and e^-m', from
//                         the gates' logits: m' is a scan of maps m -> max(f + m, i), whose composition
//                         (F, I) then (f, i) is (F + f, max(I + f, i)).
//   memory_output_kernel  numerators and n . q to the output rows.
//   memory_step_kernel    steps of single rows: everything behind the projections in one launch, the two
//                         gate logits included.
//
// The rows between the two are taken 64 at a time on the tensor cores (matrix_memory_chunks.cu, which wants
// the logarithms of the two factors) or walked by the kernel for scalar-decay recurrences (state_recurrence.cu).
#include "common.cuh"

namespace {

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoid_of(float z) { return 1.0f / (1.0f + expf(-z)); }
// With the special-function unit's exponential and reciprocal, for results that are rounded to bfloat16 at once.
template <typename AT> __device__ __forceinline__ float gate_of(float z) {
    if constexpr (sizeof(AT) == 2) return __fdividef(1.0f, 1.0f + __expf(-z));
    else return sigmoid_of(z);
}

// --------------------------------------------------------------------------- the gates

constexpr int MG_THREADS = 512, MG_WARPS = MG_THREADS / 32;

struct GatesArgs {
    const float* logits;  // [T, 2 heads]: input gates, then forget gates
    float* top;           // [slots, heads], top_stride apart
    long long top_stride;
    const int *q_start, *state_slots;
    float *keep, *add, *floor;  // [T, heads]
    int heads, logs;  // logs: the two factors' base-2 logarithms
    float cap;
};

// One CTA per (head, sequence); 512 rows at a time, the next ones' logits on their way meanwhile.
__global__ void __launch_bounds__(MG_THREADS) memory_gates_kernel(const GatesArgs a) {
    __shared__ float sF[MG_WARPS], sI[MG_WARPS];
    pdl_begin();
    const int h = blockIdx.x, s = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int first = a.q_start[s], n = a.q_start[s + 1] - first;
    if (n <= 0) return;
    float* top = a.top + (size_t)a.state_slots[s] * a.top_stride + h;
    float m = *top;  // before this round's first row
    const float* z = a.logits + (size_t)first * 2 * a.heads + h;
    float zi = 0.0f, zf = 0.0f;
    auto fetch = [&](int t) {
        if (t < n) {
            zi = z[(size_t)t * 2 * a.heads];
            zf = z[(size_t)t * 2 * a.heads + a.heads];
        }
    };
    fetch(threadIdx.x);
    for (int base = 0; base < n; base += MG_THREADS) {
        const int t = base + threadIdx.x;
        float f = 0.0f, i = -INFINITY;  // rows beyond the portion change nothing
        if (t < n) {
            i = capped(zi, a.cap);
            f = log_sigmoid(capped(zf, a.cap));
        }
        fetch(t + MG_THREADS);
        float F = f, I = i;  // the composition of this warp's rows up to this one
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pF = __shfl_up_sync(0xffffffffu, F, o), pI = __shfl_up_sync(0xffffffffu, I, o);
            if (lane >= o) {
                I = fmaxf(pI + F, I);
                F += pF;
            }
        }
        if (lane == 31) sF[warp] = F, sI[warp] = I;
        __syncthreads();
        float before = m, all = m;  // before this warp's first row, and behind this round's last
#pragma unroll
        for (int w = 0; w < MG_WARPS; ++w) {
            if (w == warp) before = all;
            all = fmaxf(sF[w] + all, sI[w]);
        }
        const float now = fmaxf(F + before, I);
        float last = __shfl_up_sync(0xffffffffu, now, 1);
        if (lane == 0) last = before;
        if (t < n) {
            const size_t at = (size_t)(first + t) * a.heads + h;
            constexpr float LOG2E = 1.4426950408889634f;
            a.keep[at] = a.logs ? (f + (last - now)) * LOG2E : expf(f + (last - now));
            a.add[at] = a.logs ? (i - now) * LOG2E : expf(i - now);
            a.floor[at] = expf(-now);
        }
        m = all;
        __syncthreads();
    }
    if (threadIdx.x == 0) *top = m;
}

// --------------------------------------------------------------------------- quotient, norm and gate

struct OutputArgs {
    const float *raw, *nq, *floor, *w;  // [T, heads * vdim], [T, heads], [T, heads], [heads * vdim]
    long long gate_ld, out_ld;
    int tokens, heads, vdim, group;
    float q_scale, den_eps, eps;
};

// `group` lanes (a power of two) a (row, head), each with N neighbouring columns at a time.
template <typename AT, int N>
__global__ void __launch_bounds__(256) memory_output_kernel(const OutputArgs a, const AT* __restrict__ gate, AT* __restrict__ out) {
    pdl_begin();
    const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / a.group;
    const int sub = threadIdx.x % a.group;
    const bool live = item < (long long)a.tokens * a.heads;
    const int t = live ? (int)(item / a.heads) : 0, h = live ? (int)(item % a.heads) : 0;
    const float* x = a.raw + ((size_t)t * a.heads + h) * a.vdim;
    const AT* g = gate + (size_t)t * a.gate_ld + (size_t)h * a.vdim;
    AT* o = out + (size_t)t * a.out_ld + (size_t)h * a.vdim;
    const float* w = a.w + (size_t)h * a.vdim;
    float ss = 0.0f;
    for (int c = sub * N; c < a.vdim; c += a.group * N) {
        if constexpr (N == 4) {
            const float4 v = *reinterpret_cast<const float4*>(x + c);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        } else {
            ss += x[c] * x[c];
        }
    }
    for (int off = a.group >> 1; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    if (!live) return;
    const size_t th = (size_t)t * a.heads + h;
    const float quotient = a.q_scale / (fmaxf(fabsf(a.nq[th] * a.q_scale), a.floor[th]) + a.den_eps);
    const float f = quotient * rsqrtf(ss * quotient * quotient / (float)a.vdim + a.eps);
    for (int c = sub * N; c < a.vdim; c += a.group * N) {
        if constexpr (N == 4) {
            const float4 v = *reinterpret_cast<const float4*>(x + c), wv = *reinterpret_cast<const float4*>(w + c);
            if constexpr (sizeof(AT) == 2) {
                const uint2 raw = *reinterpret_cast<const uint2*>(g + c);
                const float g0 = __uint_as_float(raw.x << 16), g1 = __uint_as_float(raw.x & 0xffff0000u);
                const float g2 = __uint_as_float(raw.y << 16), g3 = __uint_as_float(raw.y & 0xffff0000u);
                const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x * f * wv.x * gate_of<AT>(g0), v.y * f * wv.y * gate_of<AT>(g1));
                const __nv_bfloat162 hi = __floats2bfloat162_rn(v.z * f * wv.z * gate_of<AT>(g2), v.w * f * wv.w * gate_of<AT>(g3));
                *reinterpret_cast<uint2*>(o + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            } else {
                const float4 gv = *reinterpret_cast<const float4*>(g + c);
                *reinterpret_cast<float4*>(o + c) = make_float4(v.x * f * wv.x * gate_of<AT>(gv.x), v.y * f * wv.y * gate_of<AT>(gv.y),
                                                                v.z * f * wv.z * gate_of<AT>(gv.z), v.w * f * wv.w * gate_of<AT>(gv.w));
            }
        } else {
            o[c] = from_f32<AT>(x[c] * f * w[c] * gate_of<AT>(to_f32(g[c])));
        }
    }
}

// --------------------------------------------------------------------------- steps of single rows

constexpr int MS_THREADS = 256;
constexpr int MS_HELD = 16;  // state rows a thread has in flight

struct StepArgs {
    const void *x, *gate_w;   // [T, hidden] rows the gates read, [2 heads, hidden]
    const float* gate_b;      // [2 heads]
    const void *q, *k, *v, *gate;  // columns of the projected rows, ld apart
    long long ld, out_ld;
    const float* w;           // [heads * vdim]
    float *state, *normaliser, *top;
    long long state_stride, norm_stride, top_stride;
    const int *q_start, *state_slots;
    void* out;
    int hidden, heads, dim, vdim;
    float cap, q_scale, den_eps, eps;
};

// One CTA per (head, sequence).  N: value columns a thread takes at once.  The state is asked for before
// anything else (no kernel of this step before this one writes it), goes through registers once, and the
// read-out comes from the new state's rows as they pass.
template <typename AT, int N>
__global__ void __launch_bounds__(MS_THREADS, 2) memory_step_kernel(const StepArgs a) {
    __shared__ float scratch[33];
    __shared__ float red[MS_THREADS * N];
    extern __shared__ __align__(16) float ch[];  // q [dim], k [dim], v [vdim], o [vdim]
    const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x;
    const int row = a.q_start[s];
    if (a.q_start[s + 1] <= row) return;
    const int dim = a.dim, vdim = a.vdim, slot = a.state_slots[s];
    float *sq = ch, *sk = ch + dim, *sv = sk + dim, *so = sv + vdim;
    float* S = a.state + (size_t)slot * a.state_stride + (size_t)h * dim * vdim;
    const int spans = (vdim + N - 1) / N;
    const int lanes = min(spans, MS_THREADS), parts = MS_THREADS / lanes;  // threads over the columns, and shares of the key rows
    const int span = tid % lanes, part = tid / lanes;
    float held[MS_HELD][N];
    auto fetch = [&](int r0, int c0, bool live) {
#pragma unroll
        for (int i = 0; i < MS_HELD; ++i) {
            const int r = r0 + part + i * parts;
#pragma unroll
            for (int e = 0; e < N; ++e) held[i][e] = 0.0f;
            if (live && r < dim) {
                if constexpr (N == 4) {
                    const float4 f = *reinterpret_cast<const float4*>(S + (size_t)r * vdim + c0);
                    held[i][0] = f.x, held[i][1] = f.y, held[i][2] = f.z, held[i][3] = f.w;
                } else {
                    held[i][0] = S[(size_t)r * vdim + c0];
                }
            }
        }
    };
    fetch(0, span * N, part < parts && span < spans);
    pdl_wait();
    // the gates
    float zi = 0.0f, zf = 0.0f;
    {
        const AT* x = (const AT*)a.x + (size_t)row * a.hidden;
        const AT* wi = (const AT*)a.gate_w + (size_t)h * a.hidden;
        const AT* wf = (const AT*)a.gate_w + (size_t)(a.heads + h) * a.hidden;
        for (int c = tid; c < a.hidden; c += MS_THREADS) {
            const float v = to_f32(x[c]);
            zi = fmaf(v, to_f32(wi[c]), zi);
            zf = fmaf(v, to_f32(wf[c]), zf);
        }
    }
    const AT* q = (const AT*)a.q + (size_t)row * a.ld + (size_t)h * dim;
    const AT* k = (const AT*)a.k + (size_t)row * a.ld + (size_t)h * dim;
    const AT* v = (const AT*)a.v + (size_t)row * a.ld + (size_t)h * vdim;
    for (int c = tid; c < dim; c += MS_THREADS) sq[c] = to_f32(q[c]), sk[c] = to_f32(k[c]);
    for (int c = tid; c < vdim; c += MS_THREADS) sv[c] = to_f32(v[c]);
    zi = block_sum(zi, scratch) + a.gate_b[h];
    zf = block_sum(zf, scratch) + a.gate_b[a.heads + h];
    float* top = a.top + (size_t)slot * a.top_stride + h;
    const float i = capped(zi, a.cap), f = log_sigmoid(capped(zf, a.cap)), m = *top;
    const float now = fmaxf(f + m, i), keep = expf(f + m - now), add = expf(i - now);
    // the normaliser
    float nq = 0.0f;
    float* nrm = a.normaliser + (size_t)slot * a.norm_stride + (size_t)h * dim;
    for (int c = tid; c < dim; c += MS_THREADS) {
        const float x = fmaf(add, sk[c], keep * nrm[c]);
        nrm[c] = x;
        nq = fmaf(x, sq[c], nq);
    }
    nq = block_sum(nq, scratch);  // (its barriers stand behind the reads of *top)
    if (tid == 0) *top = now;
    // the state
    for (int base = 0; base < spans; base += lanes) {
        const int c0 = (base + span) * N;
        const bool live = part < parts && base + span < spans;
        float o[N];
#pragma unroll
        for (int e = 0; e < N; ++e) o[e] = 0.0f;
        for (int r0 = 0; r0 < dim; r0 += MS_HELD * parts) {
            if (base > 0 || r0 > 0) fetch(r0, c0, live);
            if (!live) continue;
#pragma unroll
            for (int j = 0; j < MS_HELD; ++j) {
                const int r = r0 + part + j * parts;
                if (r >= dim) continue;
                const float ak = add * sk[r], qr = sq[r];
#pragma unroll
                for (int e = 0; e < N; ++e) {
                    held[j][e] = fmaf(ak, sv[c0 + e], keep * held[j][e]);
                    o[e] = fmaf(held[j][e], qr, o[e]);
                }
                if constexpr (N == 4)
                    *reinterpret_cast<float4*>(S + (size_t)r * vdim + c0) = make_float4(held[j][0], held[j][1], held[j][2], held[j][3]);
                else
                    S[(size_t)r * vdim + c0] = held[j][0];
            }
        }
        if (live) {
#pragma unroll
            for (int e = 0; e < N; ++e) red[(part * lanes + span) * N + e] = o[e];
        }
        __syncthreads();
        for (int c = tid; c < lanes * N; c += MS_THREADS) {
            if (base * N + c >= vdim) continue;
            float sum = 0.0f;
            for (int j = 0; j < parts; ++j) sum += red[j * lanes * N + c];
            so[base * N + c] = sum;
        }
        __syncthreads();
    }
    pdl_trigger();
    // quotient, norm and gate
    float ss = 0.0f;
    for (int c = tid; c < vdim; c += MS_THREADS) ss += so[c] * so[c];
    ss = block_sum(ss, scratch);
    const float quotient = a.q_scale / (fmaxf(fabsf(nq * a.q_scale), expf(-now)) + a.den_eps);
    const float factor = quotient * rsqrtf(ss * quotient * quotient / (float)vdim + a.eps);
    const AT* gate = (const AT*)a.gate + (size_t)row * a.ld + (size_t)h * vdim;
    AT* out = (AT*)a.out + (size_t)row * a.out_ld + (size_t)h * vdim;
    for (int c = tid; c < vdim; c += MS_THREADS)
        out[c] = from_f32<AT>(so[c] * factor * a.w[(size_t)h * vdim + c] * gate_of<AT>(to_f32(gate[c])));
}

template <typename AT>
int launch_memory_step(const StepArgs& a, int num_seqs, cudaStream_t stream) {
    const size_t smem = (size_t)(2 * a.dim + 2 * a.vdim) * sizeof(float);
    if (smem > 96 * 1024) return SHISO_ERR_SHAPE;
    const bool wide = a.vdim % 4 == 0 && a.state_stride % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    auto kern = wide ? memory_step_kernel<AT, 4> : memory_step_kernel<AT, 1>;
    if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_kernel(kern, dim3(a.heads, num_seqs), dim3(MS_THREADS), smem, stream, a);
    return launch_status();
}

}  // namespace

SHISO_API int shiso_memory_gates(const float* logits, float cap, float* top, long long top_stride, const int* q_start, const int* state_slots,
                                 float* keep, float* add, float* floor, int num_seqs, int heads, int logs, cudaStream_t stream) {
    if (num_seqs <= 0) return SHISO_OK;
    if (heads <= 0 || num_seqs > 65535 || cap <= 0.0f) return SHISO_ERR_SHAPE;
    const GatesArgs a = {logits, top, top_stride, q_start, state_slots, keep, add, floor, heads, logs, cap};
    launch_kernel(memory_gates_kernel, dim3(heads, num_seqs), MG_THREADS, 0, stream, a);
    return launch_status();
}

SHISO_API int shiso_memory_output(const float* raw, const float* nq, const float* floor, const void* gate, long long gate_ld, int act_dtype,
                                  const float* w, void* out, long long out_ld, int tokens, int heads, int vdim, float q_scale,
                                  float den_eps, float eps, cudaStream_t stream) {
    if (tokens <= 0) return SHISO_OK;
    if (heads <= 0 || vdim <= 0) return SHISO_ERR_SHAPE;
    const uintptr_t all = (uintptr_t)raw | (uintptr_t)gate | (uintptr_t)w | (uintptr_t)out;
    const bool wide = vdim % 4 == 0 && gate_ld % 4 == 0 && out_ld % 4 == 0 && (all & 15) == 0;
    const int n = wide ? 4 : 1;
    int group = 1;
    while (group < 32 && group * n < vdim) group *= 2;
    const OutputArgs a = {raw, nq, floor, w, gate_ld, out_ld, tokens, heads, vdim, group, q_scale, den_eps, eps};
    const unsigned blocks = ceil_div_u((long long)tokens * heads * group, 256);
#define MO_GO(AT, N) launch_kernel(memory_output_kernel<AT, N>, blocks, 256, 0, stream, a, (const AT*)gate, (AT*)out)
    if (act_dtype == SHISO_F32) {
        if (wide) MO_GO(float, 4);
        else MO_GO(float, 1);
    } else if (act_dtype == SHISO_BF16) {
        if (wide) MO_GO(__nv_bfloat16, 4);
        else MO_GO(__nv_bfloat16, 1);
    } else {
        return SHISO_ERR_DTYPE;
    }
#undef MO_GO
    return launch_status();
}

// A step of one row per sequence.  x [T, hidden] and gate_w [2 heads, hidden] in the activation type; q, k, v and
// gate are columns of rows `ld` elements apart; state [slots, heads, dim, vdim], normaliser [slots, heads, dim] and
// top [slots, heads] float; out [T, heads * vdim], rows out_ld apart.
SHISO_API int shiso_memory_step(const void* x, const void* gate_w, const float* gate_b, const void* q, const void* k, const void* v,
                                const void* gate, long long ld, int act_dtype, const float* w, float* state, long long state_stride,
                                float* normaliser, long long norm_stride, float* top, long long top_stride, const int* q_start,
                                const int* state_slots, void* out, long long out_ld, int num_seqs, int hidden, int heads, int dim, int vdim,
                                float cap, float q_scale, float den_eps, float eps, cudaStream_t stream) {
    if (num_seqs <= 0) return SHISO_OK;
    if (heads <= 0 || dim <= 0 || vdim <= 0 || hidden <= 0 || num_seqs > 65535 || cap <= 0.0f) return SHISO_ERR_SHAPE;
    const StepArgs a = {x, gate_w, gate_b, q, k, v, gate, ld, out_ld, w, state, normaliser, top, state_stride, norm_stride, top_stride,
                        q_start, state_slots, out, hidden, heads, dim, vdim, cap, q_scale, den_eps, eps};
    if (act_dtype == SHISO_F32) return launch_memory_step<float>(a, num_seqs, stream);
    if (act_dtype == SHISO_BF16) return launch_memory_step<__nv_bfloat16>(a, num_seqs, stream);
    return SHISO_ERR_DTYPE;
}
