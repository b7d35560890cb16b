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
// A team of LANES lanes takes one map of a head (or a piece of a value head) for a group of HP_GROUP consecutive tokens of one
// sequence, NT of them at a time: the weights are loaded once a group, and the rows the convolution looks back on stay in
// registers from one NT to the next.  HP_GROUP is at least the most taps, so that only a sequence's first group looks back beyond
// the step's rows.  That group reads the state (the last taps - 1 values of u per slot, float [slots][taps - 1][channels])
// before it writes it.  Steps of single tokens (SINGLE) have a group a sequence.  Values move in pieces of 16 bytes where sizes
// and addresses allow.
// The sums of squares are formed lane by lane and across the lanes: an order that depends on the head's size alone.
#include "api.h"
#include "common.cuh"
#include "launch.cuh"

namespace {

constexpr int HP_WARPS = 4;
constexpr int HP_MAX_TAPS = 8;
constexpr int HP_MAX_DIM = 512;
constexpr int HP_GROUP = 8;

template <typename T, int VEC> __device__ __forceinline__ void hp_load(const T* p, float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        f[0] = to_float(*p);
    } else if constexpr (sizeof(T) == 4) {
#pragma unroll
        for (int i = 0; i < VEC; i += 4) {
            const float4 v = *reinterpret_cast<const float4*>(p + i);
            f[i] = v.x; f[i + 1] = v.y; f[i + 2] = v.z; f[i + 3] = v.w;
        }
    } else {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 v = __bfloat1622float2(h[i]); f[2 * i] = v.x; f[2 * i + 1] = v.y; }
    }
}
template <typename T, int VEC> __device__ __forceinline__ void hp_store(T* p, const float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        *p = from_float<T>(f[0]);
    } else if constexpr (sizeof(T) == 4) {
#pragma unroll
        for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
    } else {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    }
}

// VEC values a piece (16 bytes, or 1), NP pieces a lane; TAPS is the most taps an instance takes.
template <typename T, int VEC, int NP, int LANES, int NT, int TAPS, bool SINGLE>
__global__ void __launch_bounds__(HP_WARPS * 32) head_prepare_kernel(HeadPrepareArgs a) {
    constexpr int TEAMS = HP_WARPS * 32 / LANES, SPAN = LANES * VEC * NP;      // teams of a block; values a team holds
    constexpr bool WIDE = VEC > 1;
    __shared__ float turn[WIDE ? 1 : TEAMS][WIDE ? 1 : SPAN];                  // a team's row while its pairs are rotated
    __shared__ long long place_s[HP_GROUP];                 // where a token's cache rows of head 0 lie
    __shared__ int row_s[HP_GROUP];                         // the row's place in its page; -1: not written
    const int team = threadIdx.x / LANES, lane = threadIdx.x % LANES;
    const unsigned mask = LANES == 32 ? 0xffffffffu : ((1u << (LANES & 31)) - 1u) << ((threadIdx.x & 31) / LANES * LANES);
    const int NQ = a.n_heads * a.maps, NK = a.n_kv_heads * a.maps;
    const int v_pieces = a.v_col >= 0 ? (a.vdim + SPAN - 1) / SPAN : 0;         // values are only copied: piece by piece
    int seq, r0, n, row0;
    if (SINGLE) {
        seq = blockIdx.x;
        row0 = a.seq_start[seq];
        n = a.seq_start[seq + 1] - row0;
        r0 = 0;
        if (n <= 0) return;                                  // a padding sequence of a fixed-size batch
    } else {
        int lo = 0, hi = a.n_seqs - 1;                       // sequence s owns the groups from seq_start[s] / HP_GROUP + s on
        while (lo < hi) {
            const int mid = (lo + hi + 1) >> 1;
            if (a.seq_start[mid] / HP_GROUP + mid <= (int)blockIdx.x) lo = mid;
            else hi = mid - 1;
        }
        seq = lo;
        row0 = a.seq_start[seq];
        n = a.seq_start[seq + 1] - row0;
        r0 = ((int)blockIdx.x - (row0 / HP_GROUP + seq)) * HP_GROUP;
        if (r0 >= n) return;                                 // a number the sequence has no group for
    }
    const int past = a.tok_pos[row0];
    if (past < 0) return;
    const int end = SINGLE ? n : min(r0 + HP_GROUP, n);
    const int D = a.pad;
    const int* table = a.do_write ? a.tables + (long long)seq * a.table_width : nullptr;
    auto find_place = [&](int r, long long& place, int& page_row) {
        const int pos = past + r;
        // In a ring a later token of this step may land on the same row: only the last writer writes.
        const bool write = a.do_write && (long long)pos + (long long)a.ring_pages * a.page_size >= (long long)a.seq_end[seq];
        page_row = write ? pos % a.page_size : -1;
        place = write ? rdl_cache_offset(table, pos, a.page_size, a.ring_pages, a.n_kv_heads, 0, D) : 0;
    };
    if (threadIdx.x < HP_GROUP && r0 + (int)threadIdx.x < end) find_place(r0 + threadIdx.x, place_s[threadIdx.x], row_s[threadIdx.x]);
    __syncthreads();
    const int item = blockIdx.y * TEAMS + team;
    if (item >= NQ + NK + a.n_kv_heads * v_pieces) return;
    const bool is_q = item < NQ, is_k = !is_q && item < NQ + NK, is_v = !is_q && !is_k;
    const int kk = item - NQ, vi = kk - NK;
    const int map = is_q ? item % a.maps : (is_k ? kk % a.maps : 0);
    const int g = is_k ? kk / a.maps : (is_v ? vi / v_pieces : 0);
    const int v0 = is_v ? (vi - g * v_pieces) * SPAN : 0;    // where a value piece begins
    const int width = is_v ? min(SPAN, a.vdim - v0) : a.dim;
    const int col = is_q ? a.q_col + item * a.dim : (is_k ? a.k_col + kk * a.dim : a.v_col + g * a.vdim + v0);
    const int ch = item * a.dim;                             // the first channel of the convolution (queries, then keys)
    const int C = (NQ + NK) * a.dim, keep = (a.conv && !is_v) ? a.taps - 1 : 0;
    const int at = map * a.dim;                              // where the map lies in its laid-out head
    const T* rows = (const T*)a.rows + (long long)row0 * a.row_stride + col;
    T* out = (T*)a.out + (long long)row0 * a.out_stride;
    const int o_col = is_q ? item * D : (NQ + g) * D, v_out = (NQ + a.n_kv_heads + g) * D;
    const long long head_at = (long long)g * a.page_size * D;
    float* st = keep > 0 ? a.state + (long long)a.slots[seq] * keep * C + ch : nullptr;
    const float* nw = is_q ? a.wq : (is_k ? a.wk : nullptr);
    float bias[NP][VEC], w[TAPS][NP][VEC], wn[NP][VEC];
    float u[TAPS - 1 + NT][NP][VEC];                         // u of the TAPS - 1 rows before the ones being worked on, oldest first
    auto from_state = [&](int src, int p, float (&f)[VEC]) { // u of a row before the step's: the state's, or zeros before the sequence's start
        const int e = (p * LANES + lane) * VEC;
#pragma unroll
        for (int i = 0; i < VEC; ++i) f[i] = 0.f;
        if (e < width && src >= -keep && past + src >= 0) hp_load<float, VEC>(st + (long long)(keep + src) * C + e, f);
    };
    auto from_rows = [&](int src, int p, float (&f)[VEC]) {
        const int e = (p * LANES + lane) * VEC;
        if (e < width) {
            hp_load<T, VEC>(rows + (long long)src * a.row_stride + e, f);
#pragma unroll
            for (int i = 0; i < VEC; ++i) f[i] += bias[p][i];
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) f[i] = 0.f;
        }
    };
    // the model's constants and the state (left many kernels ago): fetched while the product before this kernel is still running
#pragma unroll
    for (int p = 0; p < NP; ++p) {
        const int e = (p * LANES + lane) * VEC;
#pragma unroll
        for (int i = 0; i < VEC; ++i) { bias[p][i] = 0.f; wn[p][i] = 1.f; }
#pragma unroll
        for (int k = 0; k < TAPS; ++k)
#pragma unroll
            for (int i = 0; i < VEC; ++i) w[k][p][i] = k == 0 ? 1.f : 0.f;
        if (e < width && !is_v) {
            if (a.bias) hp_load<float, VEC>(a.bias + ch + e, bias[p]);
            if (nw) hp_load<float, VEC>(nw + e, wn[p]);
            if (TAPS > 1 && a.conv) {
#pragma unroll
                for (int k = 0; k < TAPS; ++k)
                    if (k <= keep) hp_load<T, VEC>((const T*)a.conv + (long long)(keep - k) * C + ch + e, w[k][p]);
            } else if (a.conv) {
                hp_load<T, VEC>((const T*)a.conv + ch + e, w[0][p]);
            }
        }
        if (r0 == 0)
#pragma unroll
            for (int k = 0; k < TAPS - 1; ++k) from_state(k - (TAPS - 1), p, u[k][p]);
    }
    rdl_grid_wait();
    rdl_grid_launch_dependents();
    if (r0 > 0) {
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
            for (int p = 0; p < NP; ++p) from_rows(r0 + k - (TAPS - 1), p, u[k][p]);
    }
    // the head's values [0, width) at `at_` of its D laid-out ones; zeros where none of the head's values lie
    auto put = [&](T* dst, int at_, const float (&v)[NP][VEC], int swizzle_row, bool others) {
#pragma unroll
        for (int p = 0; p < NP; ++p) {
            const int e = (p * LANES + lane) * VEC;
            if (e < width) hp_store<T, VEC>(dst + (swizzle_row < 0 ? at_ + e : rdl_cache_col<T>(swizzle_row, at_ + e, D)), v[p]);
        }
        if (!others) return;
        const float zero[VEC] = {};
        for (int e = lane * VEC; e < D; e += LANES * VEC)
            if (is_q ? (e < at_ || e >= at_ + width) : e >= at_ + width)
                hp_store<T, VEC>(dst + (swizzle_row < 0 ? e : rdl_cache_col<T>(swizzle_row, e, D)), zero);
    };
    const float inv_dim = 1.0f / (float)a.dim;
    const bool k_others = is_q ? width < D : (map == a.maps - 1 && at + width < D);
    const bool v_others = (is_v ? v0 + width == a.vdim : true) && a.vdim < D;
    for (int rb = r0; rb < end; rb += NT) {
        float acc[NT][NP][VEC];
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int p = 0; p < NP; ++p) {
                if (rb + i < end) from_rows(rb + i, p, u[TAPS - 1 + i][p]);
                else
#pragma unroll
                    for (int e = 0; e < VEC; ++e) u[TAPS - 1 + i][p][e] = 0.f;
            }
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int p = 0; p < NP; ++p) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[i][p][e] = 0.f;
#pragma unroll
                for (int k = TAPS - 1; k >= 0; --k)          // the value k tokens back, the oldest first
#pragma unroll
                    for (int e = 0; e < VEC; ++e) acc[i][p][e] = fmaf(w[k][p][e], u[TAPS - 1 + i - k][p][e], acc[i][p][e]);
            }
        // the last taps - 1 rows move up
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
            for (int p = 0; p < NP; ++p)
#pragma unroll
                for (int e = 0; e < VEC; ++e) u[k][p][e] = u[k + NT][p][e];
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            const int r = rb + i, pos = past + r;
            if (r >= end) continue;
            float (&v)[NP][VEC] = acc[i];
            long long place = 0;
            int page_row = -1;
            if (!is_q && a.do_write) {
                if (r - r0 < HP_GROUP) { place = place_s[r - r0]; page_row = row_s[r - r0]; }
                else find_place(r, place, page_row);
                place += head_at;
            }
            if (is_v || (is_k && a.v_col < 0)) {             // the values: the row's own, or the keys as the convolution left them
                if (a.write_kv) put(out + (long long)r * a.out_stride + v_out, v0, v, -1, v_others);
                if (page_row >= 0) put((T*)a.v_cache + place, v0, v, page_row, v_others);
                if (is_v) continue;
            }
            float f = 1.f;
            if (is_q && a.q_factor) f = a.q_factor[pos];
            if (nw) {
                float ss = 0.f;
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) ss = fmaf(v[p][e], v[p][e], ss);
#pragma unroll
                for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
                const float mean = fmaf(ss, inv_dim, a.eps);
                const float inv = sizeof(T) == 2 ? rsqrtf(mean) : 1.0f / sqrtf(mean);
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) v[p][e] = v[p][e] * inv * wn[p][e];
            }
            if (a.rot_n > 0) {
                const int half = a.rot_n >> 1;
                const float* cs = a.cos_t + (long long)pos * half;
                const float* sn = a.sin_t + (long long)pos * half;
                if constexpr (WIDE) {                        // a value's partner lies in the same place of another lane's piece
#pragma unroll
                    for (int p = 0; p < NP; ++p) {
                        const int x = (p * LANES + lane) * VEC;
                        const bool lower = x < half, on = x < a.rot_n;
                        float c[VEC], sv[VEC];
                        if (on) {
                            hp_load<float, VEC>(cs + (lower ? x : x - half), c);
                            hp_load<float, VEC>(sn + (lower ? x : x - half), sv);
                        }
                        const int partner = (lower ? x + half : x - half) / VEC;      // the piece's number
#pragma unroll
                        for (int e = 0; e < VEC; ++e) {
                            float other = 0.f;
#pragma unroll
                            for (int q = 0; q < NP; ++q) {
                                const float got = __shfl_sync(mask, acc[i][q][e], partner % LANES, LANES);
                                if (partner / LANES == q) other = got;
                            }
                            // (u cos - v sin, v cos + u sin)
                            u[TAPS - 1 + i][p][e] = on ? fmaf(v[p][e], c[e], (lower ? -other : other) * sv[e]) : v[p][e];
                        }
                    }
#pragma unroll
                    for (int p = 0; p < NP; ++p)
#pragma unroll
                        for (int e = 0; e < VEC; ++e) v[p][e] = u[TAPS - 1 + i][p][e];
                } else {
                    __syncwarp(mask);
#pragma unroll
                    for (int p = 0; p < NP; ++p) turn[WIDE ? 0 : team][p * LANES + lane] = v[p][0];
                    __syncwarp(mask);
#pragma unroll
                    for (int p = 0; p < NP; ++p) {
                        const int x = p * LANES + lane;
                        if (x < a.rot_n) {
                            const bool lower = x < half;
                            const float other = turn[WIDE ? 0 : team][lower ? x + half : x - half];
                            const float c = cs[lower ? x : x - half], s = sn[lower ? x : x - half];
                            v[p][0] = fmaf(v[p][0], c, (lower ? -other : other) * s);
                        }
                    }
                }
            }
            if (is_q && a.q_factor) {
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) v[p][e] *= f;
            }
            if (is_q || a.write_kv) put(out + (long long)r * a.out_stride + o_col, at, v, -1, k_others);
            if (page_row >= 0) put((T*)a.k_cache + place, at, v, page_row, k_others);
        }
    }
    if (r0 == 0 && keep > 0) {
        // the sequence's last taps - 1 values of u, in rising order: an entry is read before it is written (row j takes an
        // older entry j + n > j, or a row of the step)
#pragma unroll
        for (int p = 0; p < NP; ++p) {
            const int e = (p * LANES + lane) * VEC;
            if (e >= width) continue;
            for (int j = 0; j < keep; ++j) {
                float f[VEC];
                if (n - keep + j >= 0) from_rows(n - keep + j, p, f);
                else from_state(n - keep + j, p, f);
                hp_store<float, VEC>(st + (long long)j * C + e, f);
            }
        }
    }
}

template <typename T, int VEC, int NP, int LANES, int TAPS>
cudaError_t launch_taps(const HeadPrepareArgs& a, cudaStream_t st) {
    constexpr int SPAN = LANES * VEC * NP, TEAMS = HP_WARPS * 32 / LANES;
    constexpr int NT = VEC * NP <= 4 ? 4 : 1;          // as many tokens as a lane's registers hold
    const int items = (a.n_heads + a.n_kv_heads) * a.maps + (a.v_col >= 0 ? a.n_kv_heads * ((a.vdim + SPAN - 1) / SPAN) : 0);
    const unsigned gy = (unsigned)((items + TEAMS - 1) / TEAMS);
    if (a.n_tokens <= a.n_seqs) return rdl_launch(head_prepare_kernel<T, VEC, NP, LANES, 1, TAPS, true>, dim3(a.n_seqs, gy), dim3(HP_WARPS * 32), 0, st, a);
    return rdl_launch(head_prepare_kernel<T, VEC, NP, LANES, NT, TAPS, false>, dim3(a.n_tokens / HP_GROUP + a.n_seqs, gy), dim3(HP_WARPS * 32), 0, st, a);
}

template <typename T, int VEC, int NP, int LANES>
cudaError_t launch_heads(const HeadPrepareArgs& a, cudaStream_t st) {
    const int taps = a.conv ? a.taps : 1;
    if (taps == 1) return launch_taps<T, VEC, NP, LANES, 1>(a, st);
    return taps <= 4 ? launch_taps<T, VEC, NP, LANES, 4>(a, st) : launch_taps<T, VEC, NP, LANES, HP_MAX_TAPS>(a, st);
}

template <typename T>
cudaError_t launch_heads_for(const HeadPrepareArgs& a, bool wide, cudaStream_t st) {
    constexpr int VEC = 16 / (int)sizeof(T);
    if (wide) {
        if (a.dim <= 8 * VEC) return launch_heads<T, VEC, 1, 8>(a, st);
        if (a.dim <= 16 * VEC) return launch_heads<T, VEC, 1, 16>(a, st);
        if (a.dim <= 32 * VEC) return launch_heads<T, VEC, 1, 32>(a, st);
        return launch_heads<T, VEC, HP_MAX_DIM / (32 * VEC), 32>(a, st);
    }
    return a.dim <= 128 ? launch_heads<T, 1, 4, 32>(a, st) : launch_heads<T, 1, 16, 32>(a, st);
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
    RDL_REQUIRE((long long)(a.n_heads + a.n_kv_heads) * a.maps + (long long)a.n_kv_heads * (a.vdim + 31) / 32 <= 65535, "head_prepare: too many heads for one grid");
    const int per = a.dtype == RDL_BF16 ? 8 : 4;             // values of a 16-byte piece; rotated halves are whole numbers of them
    const bool wide = a.dim % per == 0 && a.vdim % per == 0 && a.pad % per == 0 && a.row_stride % per == 0 && a.out_stride % per == 0 && a.q_col % per == 0 &&
                      a.k_col % per == 0 && (a.v_col < 0 || a.v_col % per == 0) && (a.rot_n / 2) % per == 0 &&
                      (((uintptr_t)a.rows | (uintptr_t)a.out | (uintptr_t)a.bias | (uintptr_t)a.conv | (uintptr_t)a.state | (uintptr_t)a.wq |
                        (uintptr_t)a.wk | (uintptr_t)a.cos_t | (uintptr_t)a.sin_t | (uintptr_t)a.k_cache | (uintptr_t)a.v_cache) & 15) == 0;
    cudaStream_t st = (cudaStream_t)stream;
    cudaError_t e = a.dtype == RDL_BF16 ? launch_heads_for<__nv_bfloat16>(a, wide, st) : launch_heads_for<float>(a, wide, st);
    RDL_CHECK_EX(e, "head_prepare");
    return 0;
}
