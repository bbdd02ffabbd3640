// What turns the outputs of two softmax maps over the same values into a differential attention layer's
// output: d = a_1 - second * a_2 per head, d / rms(d) * factor * sigmoid(gate), entry by entry.
//
// The maps' outputs are float rows in the order (key head, map, query head of the group); the output
// rows are head by head.  `group` lanes (a power of two) a (row, head), each with N neighbouring columns at a
// time; sums in an order that depends on vdim only.
#include "common.cuh"

namespace {

struct DifferenceArgs {
    const float* maps;  // [T, 2 heads * vdim]
    long long gate_ld, out_ld;
    int tokens, heads, per, vdim, group;  // per: query heads a key head
    float second, factor, eps;
};

template <int N> __device__ __forceinline__ void load_cols(const float* p, float (&v)[N]) {
    if constexpr (N == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
    } else {
        v[0] = p[0];
    }
}

template <typename AT, int N>
__global__ void __launch_bounds__(256) map_difference_kernel(const DifferenceArgs a, const AT* __restrict__ gate, AT* __restrict__ out) {
    pdl_begin();
    const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / a.group;
    const int sub = threadIdx.x % a.group;
    const bool live = item < (long long)a.tokens * a.heads;
    const int t = live ? (int)(item / a.heads) : 0, h = live ? (int)(item % a.heads) : 0;
    const int at1 = 2 * (h / a.per) * a.per + h % a.per;
    const float* m1 = a.maps + ((size_t)t * 2 * a.heads + at1) * a.vdim;
    const float* m2 = m1 + (size_t)a.per * a.vdim;
    float ss = 0.0f;
    for (int c = sub * N; c < a.vdim; c += a.group * N) {
        float x[N], y[N];
        load_cols<N>(m1 + c, x);
        load_cols<N>(m2 + c, y);
#pragma unroll
        for (int e = 0; e < N; ++e) {
            const float d = fmaf(-a.second, y[e], x[e]);
            ss += d * d;
        }
    }
    for (int off = a.group >> 1; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    if (!live) return;
    const float f = rsqrtf(ss / (float)a.vdim + a.eps) * a.factor;
    const AT* g = gate + (size_t)t * a.gate_ld + (size_t)h * a.vdim;
    AT* o = out + (size_t)t * a.out_ld + (size_t)h * a.vdim;
    for (int c = sub * N; c < a.vdim; c += a.group * N) {
        float x[N], y[N];
        load_cols<N>(m1 + c, x);
        load_cols<N>(m2 + c, y);
#pragma unroll
        for (int e = 0; e < N; ++e) x[e] = fmaf(-a.second, y[e], x[e]) * f * (1.0f / (1.0f + expf(-to_f32(g[c + e]))));
        if constexpr (N == 4 && sizeof(AT) == 2) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(x[0], x[1]), hi = __floats2bfloat162_rn(x[2], x[3]);
            *reinterpret_cast<uint2*>(o + c) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        } else {
#pragma unroll
            for (int e = 0; e < N; ++e) o[c + e] = from_f32<AT>(x[e]);
        }
    }
}

}  // namespace

// maps float [T, 2 heads * vdim]; gate and out [T, heads * vdim] in the activation type, rows gate_ld / out_ld apart.
SHISO_API int shiso_map_difference(const float* maps, const void* gate, long long gate_ld, int act_dtype, void* out, long long out_ld,
                                   int tokens, int heads, int kv_heads, int vdim, float second, float factor, float eps,
                                   cudaStream_t stream) {
    if (tokens <= 0) return SHISO_OK;
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || vdim <= 0) return SHISO_ERR_SHAPE;
    const bool wide = vdim % 4 == 0 && out_ld % 4 == 0 && (((uintptr_t)maps | (uintptr_t)out) & 15) == 0;
    const int n = wide ? 4 : 1;
    int group = 1;
    while (group < 32 && group * n < vdim) group *= 2;
    const DifferenceArgs a = {maps, gate_ld, out_ld, tokens, heads, heads / kv_heads, vdim, group, second, factor, eps};
    const unsigned blocks = ceil_div_u((long long)tokens * heads * group, 256);
#define MD_GO(AT, N) launch_kernel(map_difference_kernel<AT, N>, blocks, 256, 0, stream, a, (const AT*)gate, (AT*)out)
    if (act_dtype == SHISO_F32) {
        if (wide) MD_GO(float, 4);
        else MD_GO(float, 1);
    } else if (act_dtype == SHISO_BF16) {
        if (wide) MD_GO(__nv_bfloat16, 4);
        else MD_GO(__nv_bfloat16, 1);
    } else {
        return SHISO_ERR_DTYPE;
    }
#undef MD_GO
    return launch_status();
}
