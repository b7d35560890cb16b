// The matrix memory of xLSTM: per sequence and head a float state S [dim][vdim], a normaliser n [dim] and a running
// maximum m, with a log input gate i and a log forget gate f per head and token,
//   i = cap tanh((x_i + b_i) / cap),   f = log sigmoid(cap tanh((x_f + b_f) / cap)),
//   m_t = max(f + m_(t-1), i),   S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T,   n_t by the same rule with k for k v^T,
//   o = S_t^T q / (max(|n_t . q|, e^(-m_t)) + den_eps),     S, n and m zero before the first token,
// where q is multiplied by q_scale first.  Everything but the projections (the rows) is float.  Logarithms are kept to base
// two (m in the state too), so that every exponential is a power of two.
//
// This file walks a sequence token by token: the 32-bit path, single-token steps, and the reference of the chunked form
// (matrix_memory_chunked.cu).  A block owns MM_COLS columns of one head's state of one sequence (a column j of S decides the
// numerator of o[j] alone): thread (column, slice) keeps RPT rows of its column in registers, and the slices' parts of a
// column's sum are added in the order of the slices.  Every block also carries n and m, which its quotients need, in a copy
// of its own (`norm` holds one for every MM_COLS columns): blocks never wait on one another.
// Nothing depends on how many tokens a step brings or on what else is in the batch.
#include "api.h"
#include "common.cuh"
#include "launch.cuh"
#include "matrix_memory.cuh"

namespace {

template <typename T, int RPT>
__global__ void __launch_bounds__(256) matrix_memory_scan_kernel(MatrixMemoryArgs a) {
    constexpr int NL = (RPT + 31) / 32;       // rows of n a lane keeps
    extern __shared__ float sm[];
    const int dim = a.dim, vdim = a.vdim;
    const int slices = blockDim.x >> 5;
    float* q_s = sm;                          // [2][dim]
    float* k_s = q_s + 2 * dim;               // [2][dim]
    float* part = k_s + 2 * dim;              // [2][slices][MM_COLS]
    float* part_n = part + 2 * slices * MM_COLS;      // [2][slices]
    const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * MM_COLS;
    const int row0 = a.seq_start[seq], n = a.seq_start[seq + 1] - row0;
    if (n <= 0) return;
    if (a.tok_pos[row0] < 0) return;          // a padding sequence of a fixed-size batch
    const int tid = threadIdx.x, j = tid & 31, r = tid >> 5, n_thr = blockDim.x;
    const int col = c0 + j, i0 = r * RPT;
    const bool col_ok = col < vdim;
    const long long head = (long long)a.slots[seq] * a.n_heads + h;
    float* S = a.state + head * dim * vdim;
    float* N = a.norm + (head * gridDim.z + blockIdx.z) * (dim + 1);
    // the state was left by an earlier step, the biases are the model's: fetched while the product before is still running
    float s_reg[RPT], n_reg[NL];
#pragma unroll
    for (int i = 0; i < RPT; ++i) s_reg[i] = (col_ok && i0 + i < dim) ? S[(long long)(i0 + i) * vdim + col] : 0.f;
#pragma unroll
    for (int u = 0; u < NL; ++u) {
        const int i = j + 32 * u;
        n_reg[u] = (i < RPT && i0 + i < dim) ? N[i0 + i] : 0.f;
    }
    float m = N[dim];
    const float bi = a.i_bias[h], bf = a.f_bias[h];
    rdl_grid_wait();
    rdl_grid_launch_dependents();

    const T* rows = (const T*)a.rows + (long long)row0 * a.row_stride;
    float pq[MM_MAX_PREFETCH], pk[MM_MAX_PREFETCH], pv = 0.f, pi = 0.f, pf = 0.f;
    auto fetch = [&](int t) {
        const T* row = rows + (long long)t * a.row_stride;
#pragma unroll
        for (int u = 0; u < MM_MAX_PREFETCH; ++u) {
            const int i = tid + u * n_thr;
            pq[u] = i < dim ? to_float(row[a.q_col + h * dim + i]) : 0.f;
            pk[u] = i < dim ? to_float(row[a.k_col + h * dim + i]) : 0.f;
        }
        pv = col_ok ? to_float(row[a.v_col + h * vdim + col]) : 0.f;
        pi = to_float(row[a.i_col + h]);
        pf = to_float(row[a.f_col + h]);
    };
    auto stage = [&](int b) {
#pragma unroll
        for (int u = 0; u < MM_MAX_PREFETCH; ++u) {
            const int i = tid + u * n_thr;
            if (i < dim) { q_s[b * dim + i] = pq[u] * a.q_scale; k_s[b * dim + i] = pk[u]; }
        }
    };
    fetch(0);
    stage(0);
    __syncthreads();
    for (int t = 0; t < n; ++t) {
        const int b = t & 1;
        const float v = pv;
        const float gi = mm_input_gate(pi, bi, a.cap), gf = mm_forget_gate(pf, bf, a.cap);
        if (t + 1 < n) fetch(t + 1);
        const float m_new = fmaxf(gf + m, gi);
        const float keep = exp2f(gf + m - m_new), take = exp2f(gi - m_new);
        m = m_new;
        const float* q = q_s + b * dim + i0;
        const float* k = k_s + b * dim + i0;
        const float tv = take * v;
        float acc = 0.f;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            if (i0 + i < dim) {
                s_reg[i] = fmaf(keep, s_reg[i], k[i] * tv);
                acc = fmaf(s_reg[i], q[i], acc);
            }
        }
        float nq = 0.f;
#pragma unroll
        for (int u = 0; u < NL; ++u) {
            const int i = j + 32 * u;
            if (i < RPT && i0 + i < dim) {
                n_reg[u] = fmaf(keep, n_reg[u], take * k[i]);
                nq = fmaf(n_reg[u], q[i], nq);
            }
        }
        nq = warp_sum(nq);
        part[(b * slices + r) * MM_COLS + j] = acc;
        if (j == 0) part_n[b * slices + r] = nq;
        if (t + 1 < n) stage(b ^ 1);
        __syncthreads();
        // what is read here is written again only after the next token's barrier, which these readers reach last
        if (r == 0 && col_ok) {
            float o = 0.f, d = 0.f;
            for (int s = 0; s < slices; ++s) { o += part[(b * slices + s) * MM_COLS + j]; d += part_n[b * slices + s]; }
            a.out[(long long)(row0 + t) * a.n_heads * vdim + (long long)h * vdim + col] = o / (fmaxf(fabsf(d), exp2f(-m)) + a.den_eps);
        }
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i)
        if (col_ok && i0 + i < dim) S[(long long)(i0 + i) * vdim + col] = s_reg[i];
#pragma unroll
    for (int u = 0; u < NL; ++u) {
        const int i = j + 32 * u;
        if (i < RPT && i0 + i < dim) N[i0 + i] = n_reg[u];
    }
    if (tid == 0) N[dim] = m;
}

template <typename T>
int launch_scan(const MatrixMemoryArgs* a, cudaStream_t st) {
    const int dim = a->dim;
    // rows a thread keeps: the fewest that let eight slices cover dim
    int rpt = 4;
    while (rpt < 64 && (dim + rpt - 1) / rpt > 8) rpt *= 2;
    const int slices = (dim + rpt - 1) / rpt;
    RDL_REQUIRE(slices <= 8, "matrix_memory_scan: dim %d exceeds 512", dim);
    const int threads = 32 * slices;
    RDL_REQUIRE(dim <= MM_MAX_PREFETCH * threads, "matrix_memory_scan: dim %d is too large for %d threads", dim, threads);
    const size_t smem = (size_t)(4 * dim + 2 * slices * MM_COLS + 2 * slices) * sizeof(float);
    const dim3 grid(a->n_seqs, a->n_heads, mm_copies(a->vdim)), block(threads);
    cudaError_t e;
    switch (rpt) {
        case 4: e = rdl_launch(matrix_memory_scan_kernel<T, 4>, grid, block, smem, st, *a); break;
        case 8: e = rdl_launch(matrix_memory_scan_kernel<T, 8>, grid, block, smem, st, *a); break;
        case 16: e = rdl_launch(matrix_memory_scan_kernel<T, 16>, grid, block, smem, st, *a); break;
        case 32: e = rdl_launch(matrix_memory_scan_kernel<T, 32>, grid, block, smem, st, *a); break;
        default: e = rdl_launch(matrix_memory_scan_kernel<T, 64>, grid, block, smem, st, *a); break;
    }
    RDL_CHECK_EX(e, "matrix_memory_scan");
    return 0;
}

}  // namespace

int rdl_check_matrix_memory_args(const MatrixMemoryArgs* a, const char* who) {
    RDL_REQUIRE(rdl_valid_dtype(a->dtype), "%s: bad dtype %d", who, a->dtype);
    RDL_REQUIRE(a->n_tokens >= 0 && a->n_seqs >= 0 && a->n_heads > 0 && a->dim > 0 && a->vdim > 0, "%s: bad sizes", who);
    RDL_REQUIRE(a->rows && a->i_bias && a->f_bias && a->tok_pos && a->seq_start && a->slots && a->state && a->norm && a->out,
                "%s: missing rows, gate biases, batch description, state or output", who);
    RDL_REQUIRE(a->cap > 0.f && a->den_eps >= 0.f, "%s: the gates' cap must be positive", who);
    RDL_REQUIRE(a->n_heads <= 65535 && mm_copies(a->vdim) <= 65535, "%s: too many heads or columns for one grid", who);
    return 0;
}

extern "C" int rdl_matrix_memory_scan(const MatrixMemoryArgs* a, void* stream) {
    if (int e = rdl_check_matrix_memory_args(a, "matrix_memory_scan")) return e;
    if (a->n_tokens == 0 || a->n_seqs == 0) return 0;
    return a->dtype == RDL_BF16 ? launch_scan<__nv_bfloat16>(a, (cudaStream_t)stream) : launch_scan<float>(a, (cudaStream_t)stream);
}

// copies of n and m a head keeps
extern "C" int rdl_matrix_memory_copies(int vdim) { return mm_copies(vdim); }
