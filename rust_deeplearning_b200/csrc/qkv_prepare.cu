// Everything between the q/k/v product and attention for designs with a short convolution on the projections, in one pass:
//   u   = row + bias                                        (the projection; the bias optional)
//   c_t = sum_j conv[:, j] u_(t - (taps - 1) + j)           per channel along the sequence, zeros before its start (optional)
//   q   = c / sqrt(sum over ALL query channels of c^2 / q_count + eps) * wq,   k likewise with k_count and wk   (optional)
//   v   = (1 - lambda) c + lambda first                     (another layer's values of the same token; optional)
// and the cache write of k and v.  All in float; every value is rounded once, on its way into the packed rows the attention
// kernels read and into the cache.  q_count and k_count are the projections' sizes without any zero padding of their heads.
//
// A sequence's last taps - 1 values of u are state per slot (float [slots][taps - 1][channels]): a step's first tokens read
// what the step before left, and the block of a sequence's first tokens leaves the last ones.
//
// A block takes a group of TAPS consecutive tokens of one sequence (groups start at multiples of TAPS within the step's rows of
// the sequence), NT of them at a time; a thread owns the same channels for all of them, so a row that several outputs need is
// loaded once, and the state is read and written by the thread that owns the channel: the first group reads all the state
// a step's tokens need (they are fewer than TAPS) before it writes.
// Blocks and groups: sequence s owns the block numbers from seq_start[s] / TAPS + s on, at least as many as it has groups, so that
// a block finds its sequence by a search in that rising list; steps of single tokens have a block per token.
// The sums of squares are formed thread by thread, across each warp, and across the warps' sums by one warp (which forms the factors): an order that depends
// on the number of channels alone, never on the step's rows, on the cut or on NT.
#include "api.h"
#include "common.cuh"
#include "launch.cuh"

namespace {

constexpr int QP_MAX_TAPS = 8;

template <typename T> struct Piece;
template <> struct Piece<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[8]) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 v = __bfloat1622float2(h[i]); f[2 * i] = v.x; f[2 * i + 1] = v.y; }
    }
    static __device__ __forceinline__ uint4 pack(const float (&f)[8]) {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
        return raw;
    }
};
template <> struct Piece<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(const float* p, float (&f)[4]) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    }
    static __device__ __forceinline__ uint4 pack(const float (&f)[4]) {
        return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
    }
};

// The sums of V values over a warp at once: after each of the first log2(V) exchanges a lane goes on with half of the values,
// so that V = 8 takes 9 shuffles instead of 40.  Every value's sum is formed in the order of warp_sum.  Returns the lane's
// value; `which` is its number.
template <int V>
__device__ __forceinline__ float warp_sums(float (&v)[V], int lane, int& which) {
    which = 0;
#pragma unroll
    for (int o = 16, n = V; o > 0; o >>= 1) {
        if (n > 1) {
            n >>= 1;
            const bool upper = (lane & o) != 0;
#pragma unroll
            for (int i = 0; i < V / 2; ++i) {
                if (i < n) {
                    const float send = upper ? v[i] : v[i + n], mine = upper ? v[i + n] : v[i];
                    v[i] = mine + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
            which += upper ? n : 0;
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
        }
    }
    return v[0];
}

// VEC: pieces of 16 bytes (head_dim a whole number of them), else single values.  CPT: pieces a thread owns.  NT: tokens at a
// time.  TAPS: the most taps this instance takes.  SINGLE: a block per token (a step of single tokens).
template <typename T, bool VEC, int CPT, int NT, int TAPS, bool SINGLE>
__global__ void __launch_bounds__(VEC ? 512 : 1024) qkv_prepare_kernel(QkvPrepareArgs a) {
    constexpr int N = VEC ? Piece<T>::N : 1;
    __shared__ float part[2 * NT][32], total[2 * NT];
    __shared__ long long cache_at[NT];                      // where a token's key and value rows of head 0 lie in the cache
    __shared__ int cache_row[NT];                           // the row's place in its page; -1: not written
    int seq, r0, past;
    if (SINGLE) {
        const int t = blockIdx.x, pos = a.tok_pos[t];
        seq = a.tok_seq[t];
        if (pos < 0) return;                                // a padding row of a fixed-size batch
        r0 = t - a.seq_start[seq];
        if (r0 % TAPS) return;                              // the block of the group's first token takes it
        past = pos - r0;
    } else {
        int lo = 0, hi = a.n_seqs - 1;                      // the last sequence whose blocks start at or before this one
        while (lo < hi) {
            const int mid = (lo + hi + 1) >> 1;
            if (a.seq_start[mid] / TAPS + mid <= (int)blockIdx.x) lo = mid;
            else hi = mid - 1;
        }
        seq = lo;
        const int start = a.seq_start[seq];
        r0 = ((int)blockIdx.x - (start / TAPS + seq)) * TAPS;
        if (start + r0 >= a.seq_start[seq + 1]) return;     // a number the sequence has no group for
        past = a.tok_pos[start];
    }
    const int row0 = a.seq_start[seq], n = a.seq_start[seq + 1] - row0;
    const int C = a.n_channels, D = a.head_dim, qw = a.n_heads * D, kw = a.n_kv_heads * D;
    const int taps = a.conv ? a.taps : 1, keep = taps - 1;
    const T* rows = (const T*)a.rows + (long long)row0 * a.row_stride;      // the sequence's rows of this step
    T* out = (T*)a.out + (long long)row0 * a.out_stride;
    const T* first = a.v_first ? (const T*)a.v_first + (long long)row0 * a.v_first_stride : nullptr;
    const T* conv = (const T*)a.conv;
    float* st = keep > 0 ? a.state + (long long)a.slots[seq] * keep * C : nullptr;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
    auto load = [](const T* p, float (&f)[N]) {
        if constexpr (VEC) Piece<T>::load(p, f);
        else f[0] = to_float(*p);
    };
    auto floats = [](const float* p, float (&f)[N]) {
        if constexpr (VEC) {
#pragma unroll
            for (int e = 0; e < N; e += 4) {
                const float4 v = *reinterpret_cast<const float4*>(p + e);
                f[e] = v.x; f[e + 1] = v.y; f[e + 2] = v.z; f[e + 3] = v.w;
            }
        } else {
            f[0] = *p;
        }
    };
    auto keep_floats = [](float* p, const float (&f)[N]) {
        if constexpr (VEC) {
#pragma unroll
            for (int e = 0; e < N; e += 4) *reinterpret_cast<float4*>(p + e) = make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]);
        } else {
            *p = f[0];
        }
    };
    auto store = [](T* p, const float (&f)[N]) {
        if constexpr (VEC) *reinterpret_cast<uint4*>(p) = Piece<T>::pack(f);
        else *p = from_float<T>(f[0]);
    };
    // u of the step's row `src` (below zero: from the state, or zeros before the sequence's start)
    auto projected = [&](int src, int c, const float (&bias)[N], float (&u)[N]) {
        if (src >= 0) {
            load(rows + (long long)src * a.row_stride + c, u);
#pragma unroll
            for (int e = 0; e < N; ++e) u[e] += bias[e];
        } else if (past + src >= 0) {
            floats(st + (long long)(keep + src) * C + c, u);
        } else {
#pragma unroll
            for (int e = 0; e < N; ++e) u[e] = 0.f;
        }
    };
    // w[k]: the weight of the value k tokens back
    auto constants = [&](int c, float (&bias)[N], float (&w)[TAPS][N]) {
#pragma unroll
        for (int e = 0; e < N; ++e) bias[e] = 0.f;
        if (a.bias) floats(a.bias + c, bias);
#pragma unroll
        for (int k = 0; k < TAPS; ++k) {
            if (k <= keep && conv) load(conv + (long long)(keep - k) * C + c, w[k]);
            else
#pragma unroll
                for (int e = 0; e < N; ++e) w[k][e] = k == 0 ? 1.f : 0.f;
        }
    };
    const int end = min(r0 + TAPS, n);
    // where the cache rows of the tokens from rb on lie
    auto places = [&](int rb) {
        if (threadIdx.x >= NT) return;
        const int p = past + rb + threadIdx.x;
        // In a ring a later token of this step may land on the same row: only the last writer writes.
        const bool write = a.do_write && rb + (int)threadIdx.x < end && (long long)p + (long long)a.ring_pages * a.page_size >= (long long)a.seq_end[seq];
        cache_row[threadIdx.x] = write ? p % a.page_size : -1;
        cache_at[threadIdx.x] = write ? rdl_cache_offset(a.tables + (long long)seq * a.table_width, p, a.page_size, a.ring_pages, a.n_kv_heads, 0, D) : 0;
    };
    // What no kernel of this step has written is fetched while the product before this kernel is still running: the model's
    // constants, the page lists and, for single tokens, the state (the step before left it, many kernels ago).
    constexpr bool EARLY = CPT == 1;
    float bias[N], w[TAPS][N], norm0[N], old[SINGLE && EARLY ? TAPS - 1 : 1][N];
    if (EARLY) {
        const int c = threadIdx.x * N;
        if (c < C) {
            constants(c, bias, w);
            if (SINGLE && r0 == 0) {
#pragma unroll
                for (int k = 1; k < TAPS; ++k) {
                    if (k <= keep && past - k >= 0) floats(st + (long long)(keep - k) * C + c, old[SINGLE ? k - 1 : 0]);
                    else
#pragma unroll
                        for (int e = 0; e < N; ++e) old[SINGLE ? k - 1 : 0][e] = 0.f;
                }
            }
            if (a.wq && c < qw + kw) floats(c < qw ? a.wq + c : a.wk + (c - qw), norm0);
        }
    }
    places(r0);
    rdl_grid_wait();
    rdl_grid_launch_dependents();
    for (int rb = r0; rb < end; rb += NT) {
        float acc[NT][CPT][N];
        float sums[2 * NT];
        if (rb != r0) {
            __syncthreads();                                // what the tokens before left in shared memory is no longer read
            places(rb);
        }
#pragma unroll
        for (int i = 0; i < 2 * NT; ++i) sums[i] = 0.f;
#pragma unroll
        for (int it = 0; it < CPT; ++it) {
            const int c = (threadIdx.x + it * blockDim.x) * N;
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int e = 0; e < N; ++e) acc[i][it][e] = 0.f;
            if (c < C) {
                if (!EARLY) constants(c, bias, w);
#pragma unroll
                for (int rr = -(TAPS - 1); rr < NT; ++rr) {
                    const int src = rb + rr;
                    if (rr < -keep || src >= n) continue;
                    float u[N];
                    if (SINGLE && EARLY && rr < 0 && rb == 0) {
#pragma unroll
                        for (int e = 0; e < N; ++e) u[e] = old[SINGLE && EARLY && rr < 0 ? -rr - 1 : 0][e];
                    } else {
                        projected(src, c, bias, u);
                    }
#pragma unroll
                    for (int i = 0; i < NT; ++i) {
                        const int k = i - rr;               // row rr counts k tokens back for token i
                        if (k >= 0 && k < TAPS)
#pragma unroll
                            for (int e = 0; e < N; ++e) acc[i][it][e] = fmaf(w[k][e], u[e], acc[i][it][e]);
                    }
                }
                if (c < qw + kw) {
#pragma unroll
                    for (int i = 0; i < NT; ++i) {
                        float s = 0.f;
#pragma unroll
                        for (int e = 0; e < N; ++e) s = fmaf(acc[i][it][e], acc[i][it][e], s);
                        sums[2 * i] += c < qw ? s : 0.f;
                        sums[2 * i + 1] += c < qw ? 0.f : s;
                    }
                } else if (first) {
                    float f[NT][N];
#pragma unroll
                    for (int i = 0; i < NT; ++i)
                        if (rb + i < end) load(first + (long long)(rb + i) * a.v_first_stride + (c - qw - kw), f[i]);
#pragma unroll
                    for (int i = 0; i < NT; ++i)
#pragma unroll
                        for (int e = 0; e < N; ++e) acc[i][it][e] = (1.0f - a.v_lambda) * acc[i][it][e] + a.v_lambda * f[i][e];
                }
            }
        }
        float inv[2 * NT];
        if (a.wq) {
            int which;
            const float s = warp_sums(sums, lane, which);
            if ((lane & (16 / NT - 1)) == 0) part[which][warp] = s;
        }
        __syncthreads();
        if (a.wq) {
            for (int i = warp; i < 2 * NT; i += n_warps) {
                const float s = warp_sum(lane < n_warps ? part[i][lane] : 0.f);
                if (lane == 0) total[i] = 1.0f / sqrtf(s / ((i & 1) ? a.k_count : a.q_count) + a.eps);
            }
            __syncthreads();
#pragma unroll
            for (int i = 0; i < 2 * NT; ++i) inv[i] = total[i];
        }
#pragma unroll
        for (int it = 0; it < CPT; ++it) {
            const int c = (threadIdx.x + it * blockDim.x) * N;
            if (c >= C) continue;
            const bool is_q = c < qw, is_k = !is_q && c < qw + kw;
            float wn[N];
            if (a.wq && (is_q || is_k)) {
                if constexpr (EARLY) {
#pragma unroll
                    for (int e = 0; e < N; ++e) wn[e] = norm0[e];
                } else {
                    floats(is_q ? a.wq + c : a.wk + (c - qw), wn);
                }
            }
            const int head = is_q ? 0 : (is_k ? c - qw : c - qw - kw) / D;
            const int d = is_q ? 0 : (is_k ? c - qw : c - qw - kw) - head * D;
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int r = rb + i;
                if (r >= end) continue;
                float (&v)[N] = acc[i][it];
                if (is_q || is_k) {
                    if (a.wq) {
                        const float s = is_q ? inv[2 * i] : inv[2 * i + 1];
#pragma unroll
                        for (int e = 0; e < N; ++e) v[e] = v[e] * s * wn[e];
                    }
                }
                store(out + (long long)r * a.out_stride + c, v);
                const int pr = cache_row[i];
                if (is_q || pr < 0) continue;
                // chunks of a cache row are stored swizzled by its place in the page
                T* dst = (T*)(is_k ? a.k_cache : a.v_cache) + cache_at[i] + (long long)head * a.page_size * D;
                store(dst + (VEC ? rdl_swizzled_chunk(pr, d / N, D / N) * N : rdl_cache_col<T>(pr, d, D)), v);
            }
        }
    }
    if (r0 == 0 && keep > 0) {
        // the sequence's last taps - 1 values of u, in rising order: an entry is read before it is written (row j takes an
        // older entry j + n > j, or a row of the step)
#pragma unroll
        for (int it = 0; it < CPT; ++it) {
            const int c = (threadIdx.x + it * blockDim.x) * N;
            if (c >= C) continue;
            if (CPT > 1) {
#pragma unroll
                for (int e = 0; e < N; ++e) bias[e] = 0.f;
                if (a.bias) floats(a.bias + c, bias);
            }
            if (SINGLE && EARLY && n == 1) {                // one token moves the state on by one row, and the rows are at hand
                float u[N];
                projected(0, c, bias, u);
#pragma unroll
                for (int k = 0; k < TAPS - 1; ++k)
                    if (k < keep) {
                        if (k == 0) keep_floats(st + (long long)(keep - 1) * C + c, u);
                        else keep_floats(st + (long long)(keep - 1 - k) * C + c, old[SINGLE && EARLY && k > 0 ? k - 1 : 0]);
                    }
                continue;
            }
            for (int j = 0; j < keep; ++j) {
                float u[N];
                projected(n - keep + j, c, bias, u);
                keep_floats(st + (long long)j * C + c, u);
            }
        }
    }
}

template <typename T, bool VEC, int CPT, int NT, bool SINGLE>
cudaError_t launch_prepare(const QkvPrepareArgs& a, int threads, cudaStream_t st) {
    if (a.conv && a.taps > 4) {
        const int blocks = SINGLE ? a.n_tokens : a.n_tokens / QP_MAX_TAPS + a.n_seqs;
        return rdl_launch(qkv_prepare_kernel<T, VEC, CPT, NT, QP_MAX_TAPS, SINGLE>, dim3(blocks), dim3(threads), 0, st, a);
    }
    const int blocks = SINGLE ? a.n_tokens : a.n_tokens / 4 + a.n_seqs;
    return rdl_launch(qkv_prepare_kernel<T, VEC, CPT, NT, 4, SINGLE>, dim3(blocks), dim3(threads), 0, st, a);
}

// steps of single tokens have a block per token; prompts take several tokens at a time where a thread's registers hold them
template <typename T>
cudaError_t launch_prepare_for(const QkvPrepareArgs& a, bool vec, int pieces, cudaStream_t st) {
    const bool single = a.n_tokens <= a.n_seqs;
    auto threads_for = [&](int cpt) { const int t = ((pieces + cpt - 1) / cpt + 31) / 32 * 32; return t < 64 ? 64 : t; };
    if (vec) {
        if (pieces <= 512) return single ? launch_prepare<T, true, 1, 1, true>(a, threads_for(1), st) : launch_prepare<T, true, 1, 4, false>(a, threads_for(1), st);
        if (pieces <= 1024) return single ? launch_prepare<T, true, 2, 1, true>(a, threads_for(2), st) : launch_prepare<T, true, 2, 2, false>(a, threads_for(2), st);
        return single ? launch_prepare<T, true, 4, 1, true>(a, threads_for(4), st) : launch_prepare<T, true, 4, 1, false>(a, threads_for(4), st);
    }
    if (pieces <= 1024) return single ? launch_prepare<T, false, 1, 1, true>(a, threads_for(1), st) : launch_prepare<T, false, 1, 1, false>(a, threads_for(1), st);
    return single ? launch_prepare<T, false, 16, 1, true>(a, threads_for(16), st) : launch_prepare<T, false, 16, 1, false>(a, threads_for(16), st);
}

}  // namespace

extern "C" int rdl_qkv_prepare(const QkvPrepareArgs* p, void* stream) {
    QkvPrepareArgs a = *p;
    RDL_REQUIRE(rdl_valid_dtype(a.dtype), "qkv_prepare: bad dtype %d", a.dtype);
    RDL_REQUIRE(a.n_tokens >= 0 && a.n_seqs >= 0 && a.n_heads > 0 && a.n_kv_heads > 0 && a.head_dim > 0,
                "qkv_prepare: bad sizes tokens=%d heads=%d kv_heads=%d head_dim=%d", a.n_tokens, a.n_heads, a.n_kv_heads, a.head_dim);
    a.n_channels = (a.n_heads + 2 * a.n_kv_heads) * a.head_dim;
    RDL_REQUIRE(a.rows && a.out && a.rows != a.out && a.row_stride >= a.n_channels && a.out_stride >= a.n_channels,
                "qkv_prepare: rows in and out must be different buffers at least as wide as the heads");
    RDL_REQUIRE(a.tok_seq && a.tok_pos && a.seq_start && a.slots && a.seq_end, "qkv_prepare: missing batch description");
    RDL_REQUIRE(!a.conv || (a.taps >= 1 && a.taps <= QP_MAX_TAPS), "qkv_prepare: %d taps, the kernel takes 1 to %d", a.taps, QP_MAX_TAPS);
    RDL_REQUIRE(!a.conv || a.taps == 1 || a.state, "qkv_prepare: more than one tap needs the slots' state");
    RDL_REQUIRE((a.wq == nullptr) == (a.wk == nullptr) && (!a.wq || (a.eps > 0.f && a.q_count > 0.f && a.k_count > 0.f)),
                "qkv_prepare: the norms need both weights, eps > 0 and the projections' true sizes");
    RDL_REQUIRE(!a.v_first || a.v_first_stride >= (long long)a.n_kv_heads * a.head_dim, "qkv_prepare: the first values' rows are narrower than the heads");
    RDL_REQUIRE(!a.do_write || (a.k_cache && a.v_cache && a.tables && a.page_size > 0 && a.ring_pages > 0 && a.ring_pages <= a.table_width),
                "qkv_prepare: cache write needs storage and page tables");
    if (a.n_tokens == 0) return 0;
    const int per = a.dtype == RDL_BF16 ? 8 : 4;
    const bool vec = a.head_dim % per == 0 && a.row_stride % per == 0 && a.out_stride % per == 0 && a.v_first_stride % per == 0 &&
                     a.n_channels / per <= 2048 &&
                     (((uintptr_t)a.rows | (uintptr_t)a.out | (uintptr_t)a.bias | (uintptr_t)a.conv | (uintptr_t)a.state | (uintptr_t)a.wq |
                       (uintptr_t)a.wk | (uintptr_t)a.v_first | (uintptr_t)a.k_cache | (uintptr_t)a.v_cache) & 15) == 0;
    const int pieces = vec ? a.n_channels / per : a.n_channels;
    RDL_REQUIRE(pieces <= 16384, "qkv_prepare: %d channels exceed the 16,384 the kernel holds", a.n_channels);
    cudaStream_t st = (cudaStream_t)stream;
    cudaError_t e = a.dtype == RDL_BF16 ? launch_prepare_for<__nv_bfloat16>(a, vec, pieces, st) : launch_prepare_for<float>(a, vec, pieces, st);
    RDL_CHECK_EX(e, "qkv_prepare");
    return 0;
}
