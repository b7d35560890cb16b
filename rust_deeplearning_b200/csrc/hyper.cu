// Hyper-connections: a residual stream of S copies x_1 .. x_S per token instead of one.  A sublayer reads a weighted
// sum of the copies and writes its result back into all of them:
//   u = sum_s read[s] x_s;   y = sublayer(norm(u));   x_t <- sum_s mix[s][t] x_s + write[t] y     (all t at once)
// One kernel stands between two sublayers: it forms the copies after the first one's result, the weighted sum the second
// one reads and its norm, in float, in one pass over the token's copies:
//   y   = a + b * sigmoid(gate)             (a, b in the activations' type; b and its gate, a number per token, optional)
//   x_t = sum_s mix[s][t] x_s + write[t] y  (left out without a: the copies stay as they are)
//   out = norm(sum_t read[t] x_t)           (left out without out; without a norm's weight the plain sum)
// The copies of a token lie one after another, [rows][S][width]; at the start of a model all are equal, and the first
// kernel reads the one row ([rows][width], in_copies = 1).  A row's sums run in an order that depends on its width alone.
#include "api.h"
#include "common.cuh"
#include "launch.cuh"

namespace {

constexpr int HY_MAX_STREAMS = 8, HY_MAX_IT = 8;

__device__ __forceinline__ void hy_load4(const void* p, long long i, int dtype, float (&f)[4]) {
    if (dtype == RDL_BF16) {
        const uint2 raw = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)p + i);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
    } else {
        const float4 v = *reinterpret_cast<const float4*>((const float*)p + i);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    }
}
__device__ __forceinline__ void hy_store4(void* p, long long i, int dtype, const float (&f)[4]) {
    if (dtype == RDL_BF16) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<const uint32_t*>(&a); raw.y = *reinterpret_cast<const uint32_t*>(&b);
        *reinterpret_cast<uint2*>((__nv_bfloat16*)p + i) = raw;
    } else {
        *reinterpret_cast<float4*>((float*)p + i) = make_float4(f[0], f[1], f[2], f[3]);
    }
}

// Four values at a time, the weighted sum held in registers until its norm is known; S copies, NIT groups of four a thread
// (all loads of a thread are asked for before the first is used while they are few).
template <int S, int NIT>
__global__ void __launch_bounds__(256) hyper_vec_kernel(HyperArgs a) {
    __shared__ float scratch[33];
    rdl_grid_wait();
    rdl_grid_launch_dependents();
    const int r = blockIdx.x, W = a.width;
    const long long src = a.row_index ? a.row_index[r] : r;
    const float* xin = a.x_in + src * (a.in_copies == 1 ? 1 : S) * W;
    const bool one = a.in_copies == 1, update = a.a != nullptr;
    float mix[S][S], wr[S], rd[S];
#pragma unroll
    for (int t = 0; t < S; ++t) {
        rd[t] = a.out ? a.read[t] : 0.f;
        wr[t] = update ? a.write[t] : 0.f;
#pragma unroll
        for (int s = 0; s < S; ++s) mix[s][t] = update ? a.mix[s * S + t] : (s == t ? 1.f : 0.f);
    }
    const float gate = a.b && a.b_gate ? 1.0f / (1.0f + expf(-a.b_gate[src * a.gate_stride])) : 1.0f;
    float u[NIT][4];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < NIT; ++it) {
        const int e = (threadIdx.x + it * blockDim.x) * 4;
        if (e < W) {
            float x[S][4], y[4] = {0.f, 0.f, 0.f, 0.f}, b[4];
            if (one) {
                hy_load4(xin, e, RDL_F32, x[0]);
#pragma unroll
                for (int s = 1; s < S; ++s)
#pragma unroll
                    for (int k = 0; k < 4; ++k) x[s][k] = x[0][k];
            } else {
#pragma unroll
                for (int s = 0; s < S; ++s) hy_load4(xin, (long long)s * W + e, RDL_F32, x[s]);
            }
            if (update) {
                hy_load4(a.a, src * W + e, a.branch_dtype, y);
                if (a.b) {
                    hy_load4(a.b, src * W + e, a.branch_dtype, b);
#pragma unroll
                    for (int k = 0; k < 4; ++k) y[k] = fmaf(b[k], gate, y[k]);
                }
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) u[it][k] = 0.f;
#pragma unroll
            for (int t = 0; t < S; ++t) {
                float n[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    if (update) {
                        float v = wr[t] * y[k];
#pragma unroll
                        for (int s = 0; s < S; ++s) v = fmaf(mix[s][t], x[s][k], v);
                        n[k] = v;
                    } else {
                        n[k] = x[t][k];
                    }
                    u[it][k] = fmaf(rd[t], n[k], u[it][k]);
                }
                if (a.x_out) hy_store4(a.x_out, ((long long)r * S + t) * W + e, RDL_F32, n);
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) ss = fmaf(u[it][k], u[it][k], ss);
        }
    }
    if (!a.out) return;
    float inv = 1.f;
    if (a.w) inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + a.eps);
#pragma unroll
    for (int it = 0; it < NIT; ++it) {
        const int e = (threadIdx.x + it * blockDim.x) * 4;
        if (e < W) {
            float o[4], wv[4];
            if (a.w) hy_load4(a.w, e, a.w_dtype, wv);
#pragma unroll
            for (int k = 0; k < 4; ++k) o[k] = a.w ? u[it][k] * inv * (wv[k] + a.off) : u[it][k];
            hy_store4(a.out, (long long)r * W + e, a.out_dtype, o);
        }
    }
}

// any number of copies up to HY_MAX_STREAMS, any width: value by value, the weighted sum in shared memory
__global__ void __launch_bounds__(256) hyper_kernel(HyperArgs a) {
    extern __shared__ float u_row[];           // [width]
    __shared__ float scratch[33];
    rdl_grid_wait();
    rdl_grid_launch_dependents();
    const int r = blockIdx.x, W = a.width, S = a.n_copies;
    const long long src = a.row_index ? a.row_index[r] : r;
    const bool one = a.in_copies == 1, update = a.a != nullptr;
    const float* xin = a.x_in + src * (one ? 1 : S) * W;
    const float gate = a.b && a.b_gate ? 1.0f / (1.0f + expf(-a.b_gate[src * a.gate_stride])) : 1.0f;
    float ss = 0.f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
        float x[HY_MAX_STREAMS];
        for (int s = 0; s < S; ++s) x[s] = xin[one ? i : (long long)s * W + i];
        float y = 0.f, u = 0.f;
        if (update) {
            y = rdl_load(a.a, src * W + i, a.branch_dtype);
            if (a.b) y = fmaf(rdl_load(a.b, src * W + i, a.branch_dtype), gate, y);
        }
        for (int t = 0; t < S; ++t) {
            float n = x[t];
            if (update) {
                n = a.write[t] * y;
                for (int s = 0; s < S; ++s) n = fmaf(a.mix[s * S + t], x[s], n);
            }
            if (a.out) u = fmaf(a.read[t], n, u);
            if (a.x_out) a.x_out[((long long)r * S + t) * W + i] = n;
        }
        if (a.out) u_row[i] = u;
        ss = fmaf(u, u, ss);
    }
    if (!a.out) return;
    float inv = 1.f;
    if (a.w) inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + a.eps);
    for (int i = threadIdx.x; i < W; i += blockDim.x)      // this thread wrote the value it reads
        rdl_store(a.out, (long long)r * W + i, a.out_dtype, a.w ? u_row[i] * inv * (rdl_load(a.w, i, a.w_dtype) + a.off) : u_row[i]);
}

template <int S>
cudaError_t launch_hyper(const HyperArgs& a, int threads, int depth, cudaStream_t st) {
    const dim3 grid(a.n_rows), block(threads);
    switch (depth) {
        case 1: return rdl_launch(hyper_vec_kernel<S, 1>, grid, block, 0, st, a);
        case 2: return rdl_launch(hyper_vec_kernel<S, 2>, grid, block, 0, st, a);
        case 4: return rdl_launch(hyper_vec_kernel<S, 4>, grid, block, 0, st, a);
        default: return rdl_launch(hyper_vec_kernel<S, 8>, grid, block, 0, st, a);
    }
}

}  // namespace

extern "C" int rdl_hyper(const HyperArgs* p, void* stream) {
    const HyperArgs& a = *p;
    RDL_REQUIRE(a.n_rows >= 0 && a.width > 0 && a.n_copies >= 1 && a.n_copies <= HY_MAX_STREAMS,
                "hyper: bad sizes rows=%d width=%d copies=%d (1 to %d)", a.n_rows, a.width, a.n_copies, HY_MAX_STREAMS);
    RDL_REQUIRE(a.x_in && (a.in_copies == 1 || a.in_copies == a.n_copies), "hyper: missing stream, or %d copies for %d", a.in_copies, a.n_copies);
    RDL_REQUIRE(!a.a || (a.mix && a.write && rdl_valid_dtype(a.branch_dtype)), "hyper: a result to write back comes with its matrices");
    RDL_REQUIRE(a.a || !a.b, "hyper: the second part of a result comes with the first");
    RDL_REQUIRE(!a.out || (a.read && rdl_valid_dtype(a.out_dtype)), "hyper: the weighted sum needs its weights");
    RDL_REQUIRE(!a.w || rdl_valid_dtype(a.w_dtype), "hyper: bad dtype of the norm's weight");
    RDL_REQUIRE(a.out || a.x_out, "hyper: nothing to write");
    RDL_REQUIRE(!(a.row_index && a.x_out), "hyper: chosen rows are read, not written back");
    RDL_REQUIRE(!(a.x_out && a.in_copies == 1 && a.n_copies > 1 && a.x_out == a.x_in), "hyper: copies cannot be made in the place of the row they are made from");
    if (a.n_rows == 0) return 0;
    cudaStream_t st = (cudaStream_t)stream;
    const int W = a.width, groups = W / 4;
    // as many threads as keep two groups of four each while a block holds them: a choice by the width alone
    int threads = (groups + 1) / 2;
    threads = (threads + 31) / 32 * 32;
    threads = threads > 256 ? 256 : (threads < 32 ? 32 : threads);
    const int need = (groups + threads - 1) / threads;
    const bool aligned = (((uintptr_t)a.x_in | (uintptr_t)a.x_out | (uintptr_t)a.a | (uintptr_t)a.b | (uintptr_t)a.w | (uintptr_t)a.out) & 15) == 0;
    if (W % 4 == 0 && need <= HY_MAX_IT && aligned && a.n_copies <= 4) {
        const int depth = need <= 1 ? 1 : (need <= 2 ? 2 : (need <= 4 ? 4 : 8));
        cudaError_t e;
        switch (a.n_copies) {
            case 1: e = launch_hyper<1>(a, threads, depth, st); break;
            case 2: e = launch_hyper<2>(a, threads, depth, st); break;
            case 3: e = launch_hyper<3>(a, threads, depth, st); break;
            default: e = launch_hyper<4>(a, threads, depth, st); break;
        }
        RDL_CHECK_EX(e, "hyper");
        return 0;
    }
    const size_t smem = a.out ? (size_t)W * sizeof(float) : 0;
    RDL_REQUIRE(smem <= 48 * 1024, "hyper: rows of %d values that are no multiple of 4 (or more than 4 copies) exceed the plain kernel's 12,288", W);
    RDL_CHECK_EX(rdl_launch(hyper_kernel, dim3(a.n_rows), dim3(W >= 1024 ? 256 : 128), smem, st, a), "hyper");
    return 0;
}
