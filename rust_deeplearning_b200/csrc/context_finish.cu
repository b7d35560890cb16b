// From attention (or recurrence) results to the rows of the output product, for one mixer or for several mixers side by side
// whose output products are one.  Per side, head h of a token:
//   o = x                               the head's result, or
//   o = x_1 - lambda x_2                the difference of its two maps (differential attention)
//   o = o / sqrt(mean(o^2) + eps)       (optional)
//   o = o * weight[h, i] * factor       (the weight optional)
//   o = o * sigmoid(gate)               a gate per head or per value (optional)
// rounded once into the side's columns of the output rows.  Columns that carry the output product's bias (`ones`) are set to
// one, the columns after them up to the rows' width to zero.
// A team of LANES lanes takes one head of one token, in pieces of 16 bytes of the result where sizes and addresses allow; the order
// of its sums depends on the head's size alone.
#include "api.h"
#include "common.cuh"
#include "launch.cuh"

namespace {

constexpr int CF_WARPS = 8;
constexpr int CF_MAX_DIM = 512;

template <int VEC> __device__ __forceinline__ void cf_load(const void* p, long long i, int dtype, float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        f[0] = rdl_load(p, i, dtype);
    } else if (dtype == RDL_BF16) {
        if constexpr (VEC == 8) {
            const uint4 raw = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)p + i);
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
            for (int k = 0; k < 4; ++k) { const float2 v = __bfloat1622float2(h[k]); f[2 * k] = v.x; f[2 * k + 1] = v.y; }
        }
    } else {
#pragma unroll
        for (int k = 0; k < VEC; k += 4) {
            const float4 v = *reinterpret_cast<const float4*>((const float*)p + i + k);
            f[k] = v.x; f[k + 1] = v.y; f[k + 2] = v.z; f[k + 3] = v.w;
        }
    }
}
template <typename T, int VEC> __device__ __forceinline__ void cf_store(T* p, const float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        *p = from_float<T>(f[0]);
    } else if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int k = 0; k < 4; ++k) h[k] = __floats2bfloat162_rn(f[2 * k], f[2 * k + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    }
}
// results that are rounded to bfloat16 take the hardware's exponential and reciprocal
template <typename T> __device__ __forceinline__ float cf_sigmoid(float z) {
    return sizeof(T) == 2 ? __fdividef(1.0f, 1.0f + __expf(fminf(-z, 80.0f))) : 1.0f / (1.0f + expf(-z));
}

template <typename T, int VEC, int NP, int LANES>
__global__ void __launch_bounds__(CF_WARPS * 32) context_finish_kernel(ContextFinishArgs a) {
    rdl_grid_wait();
    rdl_grid_launch_dependents();
    constexpr int TEAMS = CF_WARPS * 32 / LANES;
    const int team = threadIdx.x / LANES, lane = threadIdx.x % LANES;
    const unsigned mask = LANES == 32 ? 0xffffffffu : ((1u << (LANES & 31)) - 1u) << ((threadIdx.x & 31) / LANES * LANES);
    const ContextSide& s = a.side[blockIdx.y];
    const long long item = (long long)blockIdx.x * TEAMS + team;
    if (item >= (long long)a.n_tokens * s.n_heads) return;
    const int t = (int)(item / s.n_heads), h = (int)(item - (long long)t * s.n_heads);
    T* out = (T*)a.out + (long long)t * a.out_stride;
    const int x_dtype = s.x_f32 ? RDL_F32 : a.dtype;
    const long long x0 = (long long)t * s.x_stride + (long long)h * s.maps * s.x_head;
    const float one_gate = s.gate_kind == RDL_CONTEXT_GATE_HEAD ? rdl_load(s.gate, (long long)t * s.gate_stride + h, a.dtype) : 0.f;
    float v[NP][VEC], x2[NP][VEC], gv[NP][VEC], wv[NP][VEC];
#pragma unroll
    for (int p = 0; p < NP; ++p) {
        const int e = (p * LANES + lane) * VEC;
#pragma unroll
        for (int i = 0; i < VEC; ++i) { v[p][i] = 0.f; x2[p][i] = 0.f; gv[p][i] = 0.f; wv[p][i] = 1.f; }
        if (e < s.vdim) {
            cf_load<VEC>(s.x, x0 + e, x_dtype, v[p]);
            if (s.maps == 2) cf_load<VEC>(s.x, x0 + s.x_head + e, x_dtype, x2[p]);
            if (s.gate_kind == RDL_CONTEXT_GATE_VALUE) cf_load<VEC>(s.gate, (long long)t * s.gate_stride + (long long)h * s.vdim + e, a.dtype, gv[p]);
            if (s.weight) cf_load<VEC>(s.weight, (long long)h * s.vdim + e, RDL_F32, wv[p]);
        }
    }
    float inv = s.factor;
    if (s.maps == 2) {
#pragma unroll
        for (int p = 0; p < NP; ++p)
#pragma unroll
            for (int i = 0; i < VEC; ++i) v[p][i] = fmaf(-s.lambda, x2[p][i], v[p][i]);
    }
    if (s.norm) {
        float ss = 0.f;
#pragma unroll
        for (int p = 0; p < NP; ++p)
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss = fmaf(v[p][i], v[p][i], ss);
#pragma unroll
        for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
        inv *= 1.0f / sqrtf(ss / (float)s.vdim + s.eps);
    }
    if (s.gate_kind == RDL_CONTEXT_GATE_HEAD) inv *= cf_sigmoid<T>(one_gate);
#pragma unroll
    for (int p = 0; p < NP; ++p) {
        const int e = (p * LANES + lane) * VEC;
        if (e >= s.vdim) continue;
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            v[p][i] *= inv;
            if (s.weight) v[p][i] *= wv[p][i];
            if (s.gate_kind == RDL_CONTEXT_GATE_VALUE) v[p][i] *= cf_sigmoid<T>(gv[p][i]);
        }
        cf_store<T, VEC>(out + s.out_col + h * s.vdim + e, v[p]);
    }
    if (blockIdx.y == 0 && h == 0)
        for (int c = a.ones_col + lane; c < a.out_width; c += LANES) out[c] = from_float<T>(c < a.ones_col + a.n_ones ? 1.f : 0.f);
}

template <typename T, int VEC, int NP, int LANES>
cudaError_t launch_as(const ContextFinishArgs& a, long long items, cudaStream_t st) {
    constexpr int TEAMS = CF_WARPS * 32 / LANES;
    return rdl_launch(context_finish_kernel<T, VEC, NP, LANES>, dim3((unsigned)((items + TEAMS - 1) / TEAMS), a.n_sides), dim3(CF_WARPS * 32), 0, st, a);
}

// items: heads of the side that has most, over all tokens
template <typename T>
cudaError_t launch_finish(const ContextFinishArgs& a, bool wide, int widest, long long items, cudaStream_t st) {
    constexpr int VEC = 16 / (int)sizeof(T);
    if (wide) {
        if (widest <= 8 * VEC) return launch_as<T, VEC, 1, 8>(a, items, st);
        if (widest <= 16 * VEC) return launch_as<T, VEC, 1, 16>(a, items, st);
        if (widest <= 32 * VEC) return launch_as<T, VEC, 1, 32>(a, items, st);
        return launch_as<T, VEC, CF_MAX_DIM / (32 * VEC), 32>(a, items, st);
    }
    return widest <= 128 ? launch_as<T, 1, 4, 32>(a, items, st) : launch_as<T, 1, 16, 32>(a, items, st);
}

}  // namespace

extern "C" int rdl_context_finish(const ContextFinishArgs* p, void* stream) {
    const ContextFinishArgs& a = *p;
    RDL_REQUIRE(rdl_valid_dtype(a.dtype) && a.n_tokens >= 0 && (a.n_sides == 1 || a.n_sides == 2) && a.out, "context_finish: bad arguments");
    const int es = a.dtype == RDL_BF16 ? 2 : 4;
    const int per = 16 / es;                    // values of a 16-byte piece of the result
    bool wide = a.out_stride % per == 0 && ((uintptr_t)a.out & 15) == 0;
    int widest = 0, used = 0, heads = 0;
    for (int i = 0; i < a.n_sides; ++i) {
        const ContextSide& s = a.side[i];
        RDL_REQUIRE(s.x && s.n_heads > 0 && s.vdim > 0 && s.vdim <= CF_MAX_DIM && (s.maps == 1 || s.maps == 2) && s.x_head >= s.vdim,
                    "context_finish: bad side %d (heads of %d values in steps of %d, %d maps; at most %d values and 2 maps)", i, s.vdim, s.x_head, s.maps, CF_MAX_DIM);
        RDL_REQUIRE(s.gate_kind == RDL_CONTEXT_GATE_NONE || (s.gate && (s.gate_kind == RDL_CONTEXT_GATE_HEAD || s.gate_kind == RDL_CONTEXT_GATE_VALUE)),
                    "context_finish: bad gate of side %d", i);
        RDL_REQUIRE(!s.norm || s.eps > 0.f, "context_finish: the norm needs eps > 0");
        RDL_REQUIRE(s.out_col >= used && s.out_col + (long long)s.n_heads * s.vdim <= a.out_width, "context_finish: the sides' columns overlap or leave the rows");
        used = s.out_col + s.n_heads * s.vdim;
        if (s.vdim > widest) widest = s.vdim;
        if (s.n_heads > heads) heads = s.n_heads;
        wide = wide && s.vdim % per == 0 && s.x_head % per == 0 && s.x_stride % per == 0 && s.out_col % per == 0 && ((uintptr_t)s.x & 15) == 0 &&
               (s.gate_kind != RDL_CONTEXT_GATE_VALUE || (s.gate_stride % per == 0 && ((uintptr_t)s.gate & 15) == 0)) && ((uintptr_t)s.weight & 15) == 0;
    }
    RDL_REQUIRE(a.ones_col >= used && a.n_ones >= 0 && a.ones_col + a.n_ones <= a.out_width && a.out_width <= a.out_stride, "context_finish: bad columns of ones");
    if (a.n_tokens == 0) return 0;
    const long long items = (long long)heads * a.n_tokens;
    RDL_REQUIRE(items / CF_WARPS < 2147483647LL, "context_finish: too many heads for one grid");
    cudaStream_t st = (cudaStream_t)stream;
    cudaError_t e = a.dtype == RDL_BF16 ? launch_finish<__nv_bfloat16>(a, wide, widest, items, st) : launch_finish<float>(a, wide, widest, items, st);
    RDL_CHECK_EX(e, "context_finish");
    return 0;
}
