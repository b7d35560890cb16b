// Everything between a q/k/v product and attention for designs that treat the projections head by head, in one pass:
//   u   = row + bias                                        (queries and keys; the bias optional)
//   c_t = sum_j conv[:, j] u_(t - (taps - 1) + j)           per channel along the sequence, zeros before its start (optional)
//   v   = the keys' c, where a design's values are its keys; else columns of the row of their own
//   n   = c / sqrt(mean(c^2) + eps) * w                     per head, one weight for all query heads and one for all key heads (optional)
//   r   = n with its first rot_n values rotated (half-split pairs, float tables)                           (optional)
//   q   = r * q_factor[position]                            (queries only; optional)
// and the cache write of k and v.  All in float; every value is rounded once, on its way into the packed rows the attention
// kernels read and into the cache.
//
// A head may have several maps (differential attention: two softmaxes over the same values).  The maps of a key head lie
// next to each other in ONE row of the cache, and a query head's map m is laid out as a query of its own that is zero
// outside map m's columns:
//   k = [k^1 | k^2],   q^1 = [q^1 | 0],   q^2 = [0 | q^2]     so that  q^m . k  is map m's score.
// The attention kernels then see heads * maps query heads on kv_heads key heads whose values are shared by both maps, and
// read every key and value once.  Everything above (norm, rotation) is done per map.
//
// A warp takes one map of a head (or a value head) for a group of TAPS consecutive tokens of one sequence, NT of them at a time,
// so that a row that several outputs of the convolution need is loaded once.  TAPS is the most taps an instance takes, so
// that only a sequence's first group looks back beyond the step's rows.  That group reads the state (the last taps - 1 values of u
// per slot, float [slots][taps - 1][channels]) before it writes it.  Steps of single tokens (SINGLE) have a group a sequence.
// The sums of squares are formed lane by lane and across the warp: an order that depends on the head's size alone.
#include "api.h"
#include "common.cuh"
#include "launch.cuh"

namespace {

constexpr int HP_WARPS = 4;
constexpr int HP_MAX_TAPS = 8;
constexpr int HP_MAX_DIM = 512;

template <typename T, int VEC> __device__ __forceinline__ void hp_load(const T* p, float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        f[0] = to_float(*p);
    } else if constexpr (sizeof(T) == 4) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    } else {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
    }
}
template <typename T, int VEC> __device__ __forceinline__ void hp_store(T* p, const float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        *p = from_float<T>(f[0]);
    } else if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
        const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<const uint32_t*>(&a);
        raw.y = *reinterpret_cast<const uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    }
}

// VEC values a piece (4 where sizes and addresses allow, else 1), NP pieces a lane.
template <typename T, int VEC, int NP, int NT, int TAPS, bool SINGLE>
__global__ void __launch_bounds__(HP_WARPS * 32) head_prepare_kernel(HeadPrepareArgs a) {
    __shared__ float turn[HP_WARPS][VEC * NP * 32];          // a warp's row while its pairs are rotated
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int NQ = a.n_heads * a.maps, NK = a.n_kv_heads * a.maps;
    const int item = blockIdx.y * HP_WARPS + warp;
    if (item >= NQ + NK + (a.v_col >= 0 ? a.n_kv_heads : 0)) return;
    int seq, r0, n, row0;
    if (SINGLE) {
        seq = blockIdx.x;
        row0 = a.seq_start[seq];
        n = a.seq_start[seq + 1] - row0;
        r0 = 0;
        if (n <= 0) return;                                  // a padding sequence of a fixed-size batch
    } else {
        int lo = 0, hi = a.n_seqs - 1;                       // sequence s owns the groups from seq_start[s] / TAPS + s on
        while (lo < hi) {
            const int mid = (lo + hi + 1) >> 1;
            if (a.seq_start[mid] / TAPS + mid <= (int)blockIdx.x) lo = mid;
            else hi = mid - 1;
        }
        seq = lo;
        row0 = a.seq_start[seq];
        n = a.seq_start[seq + 1] - row0;
        r0 = ((int)blockIdx.x - (row0 / TAPS + seq)) * TAPS;
        if (r0 >= n) return;                                 // a number the sequence has no group for
    }
    const int past = a.tok_pos[row0];
    if (past < 0) return;
    const int end = SINGLE ? n : min(r0 + TAPS, n);
    const bool is_q = item < NQ, is_k = !is_q && item < NQ + NK, is_v = !is_q && !is_k;
    const int kk = item - NQ;
    const int map = is_q ? item % a.maps : (is_k ? kk % a.maps : 0);
    const int g = is_k ? kk / a.maps : (is_v ? kk - NK : 0);
    const int width = is_v ? a.vdim : a.dim;
    const int col = is_q ? a.q_col + item * a.dim : (is_k ? a.k_col + kk * a.dim : a.v_col + g * a.vdim);
    const int ch = item * a.dim;                             // the first channel of the convolution (queries, then keys)
    const int C = (NQ + NK) * a.dim, taps = (a.conv && !is_v) ? a.taps : 1, keep = taps - 1;
    const int D = a.pad, at = map * a.dim;                   // where the map lies in its laid-out head
    const T* rows = (const T*)a.rows + (long long)row0 * a.row_stride + col;
    T* out = (T*)a.out + (long long)row0 * a.out_stride;
    const int o_col = is_q ? item * D : (NQ + g) * D, v_out = (NQ + a.n_kv_heads + g) * D;
    float* st = keep > 0 ? a.state + (long long)a.slots[seq] * keep * C + ch : nullptr;
    const int* table = a.do_write ? a.tables + (long long)seq * a.table_width : nullptr;
    const float* nw = is_q ? a.wq : (is_k ? a.wk : nullptr);
    float bias[NP][VEC], w[TAPS][NP][VEC], wn[NP][VEC], old[SINGLE ? TAPS - 1 : 1][NP][VEC];
    // the model's constants, and for single tokens the state (left many kernels ago): fetched while the product before this
    // kernel is still running
#pragma unroll
    for (int p = 0; p < NP; ++p) {
        const int e = (p * 32 + lane) * VEC;
#pragma unroll
        for (int i = 0; i < VEC; ++i) { bias[p][i] = 0.f; wn[p][i] = 1.f; }
#pragma unroll
        for (int k = 0; k < TAPS; ++k)
#pragma unroll
            for (int i = 0; i < VEC; ++i) w[k][p][i] = k == 0 ? 1.f : 0.f;
        if (e < width) {
            if (a.bias && !is_v) hp_load<float, VEC>(a.bias + ch + e, bias[p]);
            if (nw) hp_load<float, VEC>(nw + e, wn[p]);
            if (a.conv && !is_v) {
#pragma unroll
                for (int k = 0; k < TAPS; ++k)
                    if (k <= keep) hp_load<T, VEC>((const T*)a.conv + (long long)(keep - k) * C + ch + e, w[k][p]);
            }
        }
        if (SINGLE) {
#pragma unroll
            for (int k = 1; k < TAPS; ++k) {
#pragma unroll
                for (int i = 0; i < VEC; ++i) old[SINGLE ? k - 1 : 0][p][i] = 0.f;
                if (k <= keep && past - k >= 0 && e < width) hp_load<float, VEC>(st + (long long)(keep - k) * C + e, old[SINGLE ? k - 1 : 0][p]);
            }
        }
    }
    rdl_grid_wait();
    rdl_grid_launch_dependents();
    // u of the step's row `src` (below zero: from the state, or zeros before the sequence's start)
    auto projected = [&](int src, int p, float (&u)[VEC]) {
        const int e = (p * 32 + lane) * VEC;
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = 0.f;
        if (e >= width) return;
        if (src >= 0) {
            hp_load<T, VEC>(rows + (long long)src * a.row_stride + e, u);
#pragma unroll
            for (int i = 0; i < VEC; ++i) u[i] += bias[p][i];
        } else if (past + src >= 0) {
            hp_load<float, VEC>(st + (long long)(keep + src) * C + e, u);
        }
    };
    // a head's values [0, width) at `at` of its D laid-out ones; zeros where no map of the head lies
    auto put = [&](T* dst, int at_, int width_, bool others, const float (&v)[NP][VEC], int swizzle_row) {
#pragma unroll
        for (int p = 0; p < NP; ++p) {
            const int e = (p * 32 + lane) * VEC;
            if (e < width_) hp_store<T, VEC>(dst + (swizzle_row < 0 ? at_ + e : rdl_cache_col<T>(swizzle_row, at_ + e, D)), v[p]);
        }
        if (!others) return;
        const float zero[VEC] = {};
        for (int e = lane * VEC; e < D; e += 32 * VEC)
            if (is_q ? (e < at_ || e >= at_ + width_) : e >= at_ + width_)
                hp_store<T, VEC>(dst + (swizzle_row < 0 ? e : rdl_cache_col<T>(swizzle_row, e, D)), zero);
    };
    for (int rb = r0; rb < end; rb += NT) {
        float acc[NT][NP][VEC];
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int p = 0; p < NP; ++p)
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[i][p][e] = 0.f;
#pragma unroll
        for (int rr = -(TAPS - 1); rr < NT; ++rr) {
            const int src = rb + rr;
            if (rr < -keep || src >= end) continue;
#pragma unroll
            for (int p = 0; p < NP; ++p) {
                float u[VEC];
                if (SINGLE && rr < 0 && rb == 0) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) u[e] = old[SINGLE && rr < 0 ? -rr - 1 : 0][p][e];
                } else {
                    projected(src, p, u);
                }
#pragma unroll
                for (int i = 0; i < NT; ++i) {
                    const int k = i - rr;                    // row rr lies k tokens before token i
                    if (k >= 0 && k < TAPS)
#pragma unroll
                        for (int e = 0; e < VEC; ++e) acc[i][p][e] = fmaf(w[k][p][e], u[e], acc[i][p][e]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            const int r = rb + i, pos = past + r;
            if (r >= end) continue;
            float (&v)[NP][VEC] = acc[i];
            // In a ring a later token of this step may land on the same row: only the last writer writes.
            const bool write = a.do_write && !is_q && (long long)pos + (long long)a.ring_pages * a.page_size >= (long long)a.seq_end[seq];
            const int page_row = write ? pos % a.page_size : 0;
            const long long place = write ? rdl_cache_offset(table, pos, a.page_size, a.ring_pages, a.n_kv_heads, g, D) : 0;
            if (is_v || (is_k && a.v_col < 0)) {             // the values: the row's own, or the keys as the convolution left them
                if (a.write_kv) put(out + (long long)r * a.out_stride + v_out, 0, width, true, v, -1);
                if (write) put((T*)a.v_cache + place, 0, width, true, v, page_row);
                if (is_v) continue;
            }
            if (nw) {
                float ss = 0.f;
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) ss = fmaf(v[p][e], v[p][e], ss);
                ss = warp_sum(ss);
                const float inv = 1.0f / sqrtf(ss / (float)a.dim + a.eps);
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) v[p][e] = v[p][e] * inv * wn[p][e];
            }
            if (a.rot_n > 0) {
                const int half = a.rot_n >> 1;
                const float* cs = a.cos_t + (long long)pos * half;
                const float* sn = a.sin_t + (long long)pos * half;
                __syncwarp();
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) turn[warp][(p * 32 + lane) * VEC + e] = v[p][e];
                __syncwarp();
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        const int x = (p * 32 + lane) * VEC + e;
                        if (x < a.rot_n) {
                            const bool lower = x < half;
                            const float other = turn[warp][lower ? x + half : x - half];
                            const float c = cs[lower ? x : x - half], s = sn[lower ? x : x - half];
                            v[p][e] = lower ? v[p][e] * c - other * s : v[p][e] * c + other * s;
                        }
                    }
            }
            if (is_q && a.q_factor) {
                const float f = a.q_factor[pos];
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) v[p][e] *= f;
            }
            const bool others = is_q || map == a.maps - 1;
            if (is_q || a.write_kv) put(out + (long long)r * a.out_stride + o_col, at, width, others, v, -1);
            if (write) put((T*)a.k_cache + place, at, width, others, v, page_row);
        }
    }
    if (r0 == 0 && keep > 0) {
        // the sequence's last taps - 1 values of u, in rising order: an entry is read before it is written (row j takes an
        // older entry j + n > j, or a row of the step)
#pragma unroll
        for (int p = 0; p < NP; ++p) {
            const int e = (p * 32 + lane) * VEC;
            if (e >= width) continue;
            for (int j = 0; j < keep; ++j) {
                float u[VEC];
                projected(n - keep + j, p, u);
                hp_store<float, VEC>(st + (long long)j * C + e, u);
            }
        }
    }
}

template <typename T, int VEC, int NP>
cudaError_t launch_heads(const HeadPrepareArgs& a, cudaStream_t st) {
    const int items = (a.n_heads + a.n_kv_heads) * a.maps + (a.v_col >= 0 ? a.n_kv_heads : 0);
    const int taps = a.conv ? a.taps : 1;
    const dim3 block(HP_WARPS * 32);
    const unsigned gy = (unsigned)((items + HP_WARPS - 1) / HP_WARPS);
    if (a.n_tokens <= a.n_seqs) {
        if (taps <= 4) return rdl_launch(head_prepare_kernel<T, VEC, NP, 1, 4, true>, dim3(a.n_seqs, gy), block, 0, st, a);
        return rdl_launch(head_prepare_kernel<T, VEC, NP, 1, HP_MAX_TAPS, true>, dim3(a.n_seqs, gy), block, 0, st, a);
    }
    constexpr int NT = VEC * NP <= 4 ? 4 : (VEC * NP <= 8 ? 2 : 1);          // as many tokens as a lane's registers hold
    if (taps <= 4) return rdl_launch(head_prepare_kernel<T, VEC, NP, NT, 4, false>, dim3(a.n_tokens / 4 + a.n_seqs, gy), block, 0, st, a);
    return rdl_launch(head_prepare_kernel<T, VEC, NP, NT, HP_MAX_TAPS, false>, dim3(a.n_tokens / HP_MAX_TAPS + a.n_seqs, gy), block, 0, st, a);
}

template <typename T>
cudaError_t launch_heads_for(const HeadPrepareArgs& a, bool vec, cudaStream_t st) {
    const int widest = a.dim > a.vdim ? a.dim : a.vdim;
    if (vec) {
        if (widest <= 128) return launch_heads<T, 4, 1>(a, st);
        if (widest <= 256) return launch_heads<T, 4, 2>(a, st);
        return launch_heads<T, 4, 4>(a, st);
    }
    return widest <= 128 ? launch_heads<T, 1, 4>(a, st) : launch_heads<T, 1, 16>(a, st);
}

}  // namespace

extern "C" int rdl_head_prepare(const HeadPrepareArgs* p, void* stream) {
    const HeadPrepareArgs& a = *p;
    RDL_REQUIRE(rdl_valid_dtype(a.dtype), "head_prepare: bad dtype %d", a.dtype);
    RDL_REQUIRE(a.n_tokens >= 0 && a.n_seqs >= 0 && a.n_heads > 0 && a.n_kv_heads > 0 && a.n_heads % a.n_kv_heads == 0 && a.maps >= 1 && a.dim > 0 && a.vdim > 0,
                "head_prepare: bad sizes tokens=%d heads=%d kv_heads=%d maps=%d dim=%d vdim=%d", a.n_tokens, a.n_heads, a.n_kv_heads, a.maps, a.dim, a.vdim);
    RDL_REQUIRE(a.dim <= HP_MAX_DIM && a.vdim <= HP_MAX_DIM, "head_prepare: heads of %d and %d values, the kernel takes up to %d", a.dim, a.vdim, HP_MAX_DIM);
    RDL_REQUIRE(a.pad >= a.maps * a.dim && a.pad >= a.vdim, "head_prepare: heads are laid out with %d values, %d maps of %d and %d values do not fit",
                a.pad, a.maps, a.dim, a.vdim);
    RDL_REQUIRE(a.v_col >= 0 || (a.maps == 1 && a.vdim == a.dim), "head_prepare: keys serve as values with one map of the values' size only");
    RDL_REQUIRE(a.rows && a.out && a.rows != a.out && a.out_stride >= (long long)(a.n_heads * a.maps + 2 * a.n_kv_heads) * a.pad,
                "head_prepare: rows in and out must be different buffers, the latter as wide as the laid-out heads");
    RDL_REQUIRE(a.tok_pos && a.seq_start && a.slots && a.seq_end, "head_prepare: missing batch description");
    RDL_REQUIRE(!a.conv || (a.taps >= 1 && a.taps <= HP_MAX_TAPS), "head_prepare: %d taps, the kernel takes 1 to %d", a.taps, HP_MAX_TAPS);
    RDL_REQUIRE(!a.conv || a.taps == 1 || a.state, "head_prepare: more than one tap needs the slots' state");
    RDL_REQUIRE((a.wq == nullptr) == (a.wk == nullptr) && (!a.wq || a.eps > 0.f), "head_prepare: the norms need both weights and eps > 0");
    RDL_REQUIRE(a.rot_n >= 0 && a.rot_n % 2 == 0 && a.rot_n <= a.dim && (a.rot_n == 0 || (a.cos_t && a.sin_t)),
                "head_prepare: the rotated dimensions (%d) must be even, at most dim (%d) and come with tables", a.rot_n, a.dim);
    RDL_REQUIRE(!a.do_write || (a.k_cache && a.v_cache && a.tables && a.page_size > 0 && a.ring_pages > 0 && a.ring_pages <= a.table_width),
                "head_prepare: cache write needs storage and page tables");
    if (a.n_tokens == 0 || a.n_seqs == 0) return 0;
    const int items = (a.n_heads + a.n_kv_heads) * a.maps + (a.v_col >= 0 ? a.n_kv_heads : 0);
    RDL_REQUIRE((items + HP_WARPS - 1) / HP_WARPS <= 65535, "head_prepare: too many heads for one grid");
    const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.pad % 4 == 0 && a.row_stride % 4 == 0 && a.out_stride % 4 == 0 && a.q_col % 4 == 0 &&
                     a.k_col % 4 == 0 && (a.v_col < 0 || a.v_col % 4 == 0) && (a.dtype == RDL_F32 || a.pad % 8 == 0) &&
                     (((uintptr_t)a.rows | (uintptr_t)a.out | (uintptr_t)a.bias | (uintptr_t)a.conv | (uintptr_t)a.state | (uintptr_t)a.wq |
                       (uintptr_t)a.wk | (uintptr_t)a.k_cache | (uintptr_t)a.v_cache) & 15) == 0;
    cudaStream_t st = (cudaStream_t)stream;
    cudaError_t e = a.dtype == RDL_BF16 ? launch_heads_for<__nv_bfloat16>(a, vec, st) : launch_heads_for<float>(a, vec, st);
    RDL_CHECK_EX(e, "head_prepare");
    return 0;
}
