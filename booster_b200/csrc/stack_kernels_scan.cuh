// stack_kernels_scan.cuh — CUDA kernels (sm_100a) of the layer-stack models' recurrences over time, on top of stack_kernels.cuh:
//   outer-product recurrence  S <- a S + b k v^T, o = S^T q per head, a matrix state with one decay a and one input scale b per
//                             token and head: constant (retention), from a step size (state-space duality, heads sharing the
//                             keys and queries of their group) or from a table (mLSTM, whose normaliser is one more column)
//   mLSTM gates               log gates, running maximum and the a, b they give
//   gated norm in parts       the read-out of the state-space mixer: skip term, silu gate, then the norm
//   selective scan            S[c][n] <- exp(dt_c A[c][n]) S[c][n] + dt_c x_c B[n], y_c = S[c] . C + D_c x_c, silu gate
// Every size and constant is a kernel argument. Everything here is float32: decays and their logarithms, step sizes, gates of a
// recurrence, the states.
#pragma once
#include "stack_kernels.cuh"

namespace b200 {
namespace stk {

// ---- outer-product recurrence -----------------------------------------------------------------------------------------------
// Row t of Q / K / V starts at Q + t ldq (K, V alike); head h reads query and key (h / share) of D entries each and value h of V
// entries. The state of a head is [D][V], followed by a vector n [D] when `norm` is set: n takes part as one more column of the
// state whose value is always 1; its read-out n . q goes to den[t][h].
// Where a and b come from (`kind`):
//   SCAN_CONST   a = decay[h], b = 1
//   SCAN_STEP    step size dt = softplus(ab[t ld_ab + h] + dt_bias[h]):  a = exp(-exp(A_log[h]) dt), b = dt (one-token steps)
//   SCAN_TABLE   a = ab[t ld_ab + h], b = ab[t ld_ab + H + h]
enum { SCAN_CONST = 0, SCAN_STEP = 1, SCAN_TABLE = 2 };
struct OuterScan {
    const float * Q; int ldq;
    const float * K; int ldk;
    const float * Vv; int ldv;
    int T, H, share, D, V;
    int kind;
    const float * decay;
    const float * ab; int ld_ab;
    const float * dt_bias; const float * A_log;
    float * S; long long head_stride;
    int norm;
    float * O;                  // [T][H][V]
    float * den;                // [T][H]
};
__device__ __forceinline__ float step_size(const float * raw, const float * dt_bias, int h) { return softplusf_(raw[h] + dt_bias[h]); }
__device__ __forceinline__ void outer_ab(const OuterScan & s, int t, int h, float & a, float & b) {
    if (s.kind == SCAN_CONST) { a = s.decay[h]; b = 1.0f; }
    else if (s.kind == SCAN_STEP) { b = step_size(s.ab + (size_t) t * s.ld_ab, s.dt_bias, h); a = expf(-expf(s.A_log[h]) * b); }
    else { a = s.ab[(size_t) t * s.ld_ab + h]; b = s.ab[(size_t) t * s.ld_ab + s.H + h]; }
}
// the table of a and b from step sizes, for portions of several tokens: AB[t] = [ a: H | b: H ]
__global__ void k_step_table(const float * __restrict__ raw, int ldr, const float * __restrict__ dt_bias, const float * __restrict__ A_log, int H, float * __restrict__ AB, int ld_ab) {
    const int t = blockIdx.x;
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
        const float dt = step_size(raw + (size_t) t * ldr, dt_bias, h);
        AB[(size_t) t * ld_ab + h] = expf(-expf(A_log[h]) * dt);
        AB[(size_t) t * ld_ab + H + h] = dt;
    }
}

// The token walk: S stays in registers for the whole portion; four neighbouring lanes share one column of S, each holding a quarter
// of its rows, and close the read-out with two shuffles. q, k, v (and the table's a, b) of a few tokens arrive in shared memory by
// asynchronous copies while the tokens before them are walked (two buffers); each quarter of the rows is padded apart so that the
// four lanes' reads fall into different banks. A head's columns are spread over gridDim.y blocks.
template <int DMAX>
__global__ void __launch_bounds__(512) k_outer_scan(const OuterScan a) {
    constexpr int TT = DMAX > 128 ? 4 : 8, DR = DMAX / GD_RG, ROW = GD_RG * (DR + GD_PAD);
    __shared__ __align__(16) float qs[2][TT][ROW], ks[2][TT][ROW], vs[2][TT][128], gs[2][TT][2];
    const int h = blockIdx.x, hq = h / a.share, tid = threadIdx.x, lane = tid & 31, rg = lane & 3, ncols = blockDim.x / GD_RG;
    const int D = a.D, V = a.V, cl = (tid >> 5) * 8 + (lane >> 2), col = blockIdx.y * ncols + cl;
    const bool live = col < V, is_n = a.norm && col == V;
    const auto stage = [&](int t0, int buf) {
        const int nt = min(TT, a.T - t0);
        for (int i = tid; i < nt * DMAX; i += blockDim.x) {
            const int tt = i / DMAX, d = i % DMAX, at = (d / DR) * (DR + GD_PAD) + d % DR;
            const bool in = d < D;
            const size_t off = (size_t) hq * D + (in ? d : 0);
            cp_async4(&qs[buf][tt][at], a.Q + (size_t) (t0 + tt) * a.ldq + off, in);
            cp_async4(&ks[buf][tt][at], a.K + (size_t) (t0 + tt) * a.ldk + off, in);
        }
        for (int i = tid; i < nt * ncols; i += blockDim.x) {
            const int tt = i / ncols, c = i % ncols;
            const bool in = blockIdx.y * ncols + c < V;
            cp_async4(&vs[buf][tt][c], a.Vv + (size_t) (t0 + tt) * a.ldv + (size_t) h * V + (in ? blockIdx.y * ncols + c : 0), in);
        }
        if (a.kind == SCAN_TABLE) {
            if (tid < 2 * nt) cp_async4(&gs[buf][tid >> 1][tid & 1], a.ab + (size_t) (t0 + (tid >> 1)) * a.ld_ab + (tid & 1) * a.H + h, true);
        } else if (tid < nt) outer_ab(a, t0 + tid, h, gs[buf][tid][0], gs[buf][tid][1]);
    };
    stage(0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    float s[DR];
    float * Sh = a.S + (size_t) h * a.head_stride;
    const size_t rstep = is_n ? 1 : V;                  // row d of this thread's column: S[d][col], or n[d] behind the matrix
    float * Sc = Sh + (is_n ? (size_t) D * V : (size_t) col);
    const bool held = live || is_n;
#pragma unroll
    for (int i = 0; i < DR; i++) { const int d = rg * DR + i; s[i] = (held && d < D) ? Sc[(size_t) d * rstep] : 0.f; }
    const int base = rg * (DR + GD_PAD);
    for (int t0 = 0, buf = 0; t0 < a.T; t0 += TT, buf ^= 1) {
        const int nt = min(TT, a.T - t0);
        if (t0 + TT < a.T) stage(t0 + TT, buf ^ 1);     // its last readers passed the barrier that closed the previous walk
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        for (int tt = 0; tt < nt; tt++) {               // every lane walks (the shuffles need the whole warp); dead columns hold zeros
            const float g = gs[buf][tt][0], v = (is_n ? 1.0f : vs[buf][tt][cl]) * gs[buf][tt][1];
            float op[4] = { 0.f, 0.f, 0.f, 0.f };
#pragma unroll
            for (int i = 0; i < DR; i++) {
                s[i] = fmaf(g, s[i], ks[buf][tt][base + i] * v);
                op[i & 3] = fmaf(s[i], qs[buf][tt][base + i], op[i & 3]);
            }
            float o = (op[0] + op[1]) + (op[2] + op[3]);
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (rg == 0) {
                if (live) a.O[(size_t) (t0 + tt) * a.H * V + (size_t) h * V + col] = o;
                else if (is_n) a.den[(size_t) (t0 + tt) * a.H + h] = o;
            }
        }
        __syncthreads();
    }
    if (held) {
#pragma unroll
        for (int i = 0; i < DR; i++) { const int d = rg * DR + i; if (d < D) Sc[(size_t) d * rstep] = s[i]; }
    }
}

// Long prompt portions run the same recurrence chunk by chunk (RC tokens), so that only the short walk over chunks is serial.
// With t, j local to chunk c of n_c tokens, S_c the state before it and w(j, t) = prod_(j < i <= t) a_i (w(-1, t): from the start):
//   U_c = sum_j w(j, n_c - 1) b_j k_j v_j^T,  A_c = w(-1, n_c - 1)      k_outer_chunk_kv     (all chunks at once)
//   S_(c+1) = A_c S_c + U_c                                            k_outer_chunk_state  (in place: U_c's slot then holds S_c)
//   o_t = w(-1, t) S_c^T q_t + sum_(j <= t) w(j, t) b_j (q_t . k_j) v_j  k_outer_chunk_out    (all chunks at once)
// Decays enter as products of at most RC factors, as in the walk; sums in another order. SB [H][chunks][head_stride] is a working
// buffer of the pass, AC [H][chunks] the chunks' decays. A tile of values is NC columns wide (128 or 64).
constexpr int RC = 32;
// rows [0, n_rows) x columns [0, n_cols) of a row-major source into a shared tile of `rows` x `cols` (row stride dst_ld), zeros
// elsewhere, by asynchronous copies that are all issued before any is awaited (16 bytes each when `vec`: every address a multiple of 16)
__device__ __forceinline__ void stage_tile_async(float * dst, int dst_ld, const float * src, size_t src_ld, int rows, int cols, int n_rows, int n_cols, bool vec, int tid, int nthreads) {
    if (vec) {
        const int c4 = cols >> 2;
        for (int i = tid; i < rows * c4; i += nthreads) {
            const int j = i / c4, x = (i - j * c4) << 2;
            const bool in = j < n_rows && x < n_cols;
            cp_async16((uint32_t) __cvta_generic_to_shared(dst + j * dst_ld + x), in ? (const void *) (src + (size_t) j * src_ld + x) : (const void *) src, in ? 16u : 0u);
        }
    } else {
        for (int i = tid; i < rows * cols; i += nthreads) {
            const int j = i / cols, x = i - j * cols;
            const bool in = j < n_rows && x < n_cols;
            cp_async4(dst + j * dst_ld + x, in ? src + (size_t) j * src_ld + x : src, in);
        }
    }
}
__device__ __forceinline__ void async_copies_done() {
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
}
// grid (H, chunks, ceil(V / NC)), 256 threads: thread (ty, tx) owns 8 x NC / 16 of a 128 x NC tile of U_c; keys and values of the
// chunk are staged in shared memory
template <int NC>
__global__ void __launch_bounds__(256, NC == 128 ? 2 : 1) k_outer_chunk_kv(const OuterScan a, int vec, float * __restrict__ SB, float * __restrict__ AC) {
    constexpr int CW = NC / 16;
    __shared__ __align__(16) float Ks[RC][128], Vs[RC][NC];
    __shared__ float pw[RC];
    const int h = blockIdx.x, hq = h / a.share, c = blockIdx.y, v0 = blockIdx.z * NC, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int D = a.D, V = a.V, t0 = c * RC, nt = min(RC, a.T - t0), nch = gridDim.y;
    stage_tile_async(&Vs[0][0], NC, a.Vv + (size_t) t0 * a.ldv + (size_t) h * V + v0, (size_t) a.ldv, RC, NC, nt, V - v0, vec, tid, 256);
    if (tid < RC) {                                     // the key's weight at the chunk's end: b_j times the decays after j
        float ga = 1.f, gb = 0.f;
        if (tid < nt) outer_ab(a, t0 + tid, h, ga, gb);
        float suf = ga;                                 // product of a_i, i >= lane
#pragma unroll
        for (int o = 1; o < RC; o <<= 1) { const float u = __shfl_down_sync(0xffffffffu, suf, o); if (tid + o < RC) suf *= u; }
        const float after = __shfl_down_sync(0xffffffffu, suf, 1);
        pw[tid] = tid < nt ? gb * (tid + 1 < RC ? after : 1.f) : 0.f;
        if (tid == 0 && blockIdx.z == 0) AC[(size_t) h * nch + c] = suf;
    }
    float * U = SB + ((size_t) h * nch + c) * a.head_stride;
    for (int d0 = 0; d0 < D; d0 += 128) {
        __syncthreads();
        stage_tile_async(&Ks[0][0], 128, a.K + (size_t) t0 * a.ldk + (size_t) hq * D + d0, (size_t) a.ldk, RC, 128, nt, D - d0, vec, tid, 256);
        async_copies_done();
        __syncthreads();
        float acc[8][CW];
#pragma unroll
        for (int i = 0; i < 8; i++)
#pragma unroll
            for (int b = 0; b < CW; b++) acc[i][b] = 0.f;
#pragma unroll 4
        for (int j = 0; j < RC; j++) {
            const float4 ka = *reinterpret_cast<const float4 *>(&Ks[j][ty * 8]), kb = *reinterpret_cast<const float4 *>(&Ks[j][ty * 8 + 4]);
            float vv[CW];
#pragma unroll
            for (int b = 0; b < CW; b += 4) { const float4 f4 = *reinterpret_cast<const float4 *>(&Vs[j][tx * CW + b]); vv[b] = f4.x; vv[b + 1] = f4.y; vv[b + 2] = f4.z; vv[b + 3] = f4.w; }
            const float f = pw[j];
            const float kk[8] = { ka.x * f, ka.y * f, ka.z * f, ka.w * f, kb.x * f, kb.y * f, kb.z * f, kb.w * f };
#pragma unroll
            for (int i = 0; i < 8; i++)
#pragma unroll
                for (int b = 0; b < CW; b++) acc[i][b] = fmaf(kk[i], vv[b], acc[i][b]);
        }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int d = d0 + ty * 8 + i;
            if (d >= D) continue;
#pragma unroll
            for (int b = 0; b < CW; b++) { const int v = v0 + tx * CW + b; if (v < V) U[(size_t) d * V + v] = acc[i][b]; }
        }
        if (a.norm && blockIdx.z == 0 && tid < 128 && d0 + tid < D) {       // the normaliser's column
            float n = 0.f;
#pragma unroll 8
            for (int j = 0; j < RC; j++) n = fmaf(pw[j], Ks[j][tid], n);
            U[(size_t) D * V + d0 + tid] = n;
        }
    }
}
// grid (H, ceil(entries / 256)): a thread owns one entry of the state (matrix and normaliser alike) and walks the chunks
__global__ void k_outer_chunk_state(int n, long long head_stride, int nch, const float * __restrict__ AC, float * __restrict__ S, float * __restrict__ SB) {
    const int h = blockIdx.x, e = blockIdx.y * blockDim.x + threadIdx.x;
    if (e >= n) return;
    const float * ac = AC + (size_t) h * nch;
    float s = S[(size_t) h * head_stride + e];
    float * sb = SB + (size_t) h * nch * head_stride + e;
    for (int c0 = 0; c0 < nch; c0 += 8) {
        float u[8], g[8];
#pragma unroll
        for (int i = 0; i < 8; i++) { u[i] = c0 + i < nch ? sb[(size_t) (c0 + i) * head_stride] : 0.f; g[i] = c0 + i < nch ? ac[c0 + i] : 0.f; }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            if (c0 + i < nch) {
                sb[(size_t) (c0 + i) * head_stride] = s;
                s = fmaf(g[i], s, u[i]);
            }
        }
    }
    S[(size_t) h * head_stride + e] = s;
}
// grid (H, chunks, ceil(V / NC)), 128 threads: warp w owns tokens 8 w .. 8 w + 7 of the chunk, a lane NC / 32 value channels.
// Dynamic shared memory: q and k of the chunk [RC][D + 4] each, the weighted scores [RC][RC + 4], the values [RC][NC].
template <int NC>
__global__ void __launch_bounds__(128) k_outer_chunk_out(const OuterScan a, int vec_all, const float * __restrict__ SB) {
    extern __shared__ __align__(16) float csm[];
    constexpr int CW = NC / 32, AP = RC + 4;            // score rows padded to whole 16-byte chunks
    const int D = a.D, V = a.V, Dp = D + 4;
    float * Qs = csm, * Ks = Qs + RC * Dp, * As = Ks + RC * Dp, * Vs = As + RC * AP;
    __shared__ float ga_s[RC], gb_s[RC], pw[RC];
    const int h = blockIdx.x, hq = h / a.share, c = blockIdx.y, v0 = blockIdx.z * NC, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int t0 = c * RC, nt = min(RC, a.T - t0), nch = gridDim.y;
    stage_tile_async(Qs, Dp, a.Q + (size_t) t0 * a.ldq + (size_t) hq * D, (size_t) a.ldq, RC, D, nt, D, vec_all, tid, 128);
    stage_tile_async(Ks, Dp, a.K + (size_t) t0 * a.ldk + (size_t) hq * D, (size_t) a.ldk, RC, D, nt, D, vec_all, tid, 128);
    stage_tile_async(Vs, NC, a.Vv + (size_t) t0 * a.ldv + (size_t) h * V + v0, (size_t) a.ldv, RC, NC, nt, V - v0, vec_all, tid, 128);
    if (tid < RC) {
        float ga = 1.f, gb = 0.f;
        if (tid < nt) outer_ab(a, t0 + tid, h, ga, gb);
        ga_s[tid] = ga; gb_s[tid] = gb;
        float pre = ga;                                 // product of a_i, i <= lane
#pragma unroll
        for (int o = 1; o < RC; o <<= 1) { const float u = __shfl_up_sync(0xffffffffu, pre, o); if (tid >= o) pre *= u; }
        pw[tid] = pre;
    }
    async_copies_done();
    __syncthreads();
    const int D4 = (D & 3) ? 0 : D;                     // 16-byte reads along d need whole chunks per row (D + 4 is then a multiple of 4 too)
    {   // scores of the chunk against itself: lane = key j, the warp's 8 tokens; 16-byte reads along d (a lane's own key row, the
        // tokens' query rows as broadcasts) when D is a multiple of 4, else entry by entry
        float sc[8] = { 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f };
        const float * kr = Ks + lane * Dp;
        for (int d = 0; d < D4; d += 4) {
            const float4 k4 = *reinterpret_cast<const float4 *>(kr + d);
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const float4 q4 = *reinterpret_cast<const float4 *>(Qs + (warp * 8 + i) * Dp + d);
                sc[i] = fmaf(q4.x, k4.x, fmaf(q4.y, k4.y, fmaf(q4.z, k4.z, fmaf(q4.w, k4.w, sc[i]))));
            }
        }
        for (int d = D4; d < D; d++)
#pragma unroll
            for (int i = 0; i < 8; i++) sc[i] = fmaf(Qs[(warp * 8 + i) * Dp + d], kr[d], sc[i]);
        // w(j, t) b_j: zero before the key, b at the key's own token, then one decay per token
        float w = 0.f;
        for (int t = 0; t < warp * 8; t++) w = t == lane ? gb_s[t] : w * ga_s[t];
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int t = warp * 8 + i;
            w = t == lane ? gb_s[t] : w * ga_s[t];
            As[t * AP + lane] = sc[i] * w;
        }
    }
    __syncthreads();
    float acc[8][CW];
#pragma unroll
    for (int i = 0; i < 8; i++)
#pragma unroll
        for (int b = 0; b < CW; b++) acc[i][b] = 0.f;
    const float * Sc = SB + ((size_t) h * nch + c) * a.head_stride;
    const int v = v0 + lane * CW;
    const bool vec = (V % CW) == 0 && (a.head_stride & 3) == 0 && v + CW - 1 < V;
    const auto srow = [&](int d, float (&sv)[CW]) {
        const float * p = Sc + (size_t) d * V + v;
        if (vec) {
            if constexpr (CW == 4) { const float4 f = __ldg(reinterpret_cast<const float4 *>(p)); sv[0] = f.x; sv[1] = f.y; sv[2] = f.z; sv[3] = f.w; }
            else { const float2 f = __ldg(reinterpret_cast<const float2 *>(p)); sv[0] = f.x; sv[1] = f.y; }
        } else {
#pragma unroll
            for (int b = 0; b < CW; b++) sv[b] = v + b < V ? __ldg(p + b) : 0.f;
        }
    };
#pragma unroll 2
    for (int d = 0; d < D4; d += 4) {                   // four rows of the chunk's entry state per step, the queries as 16-byte broadcasts
        float sv[4][CW];
#pragma unroll
        for (int r = 0; r < 4; r++) srow(d + r, sv[r]);
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const float4 q4 = *reinterpret_cast<const float4 *>(Qs + (warp * 8 + i) * Dp + d);
#pragma unroll
            for (int b = 0; b < CW; b++) acc[i][b] = fmaf(q4.x, sv[0][b], fmaf(q4.y, sv[1][b], fmaf(q4.z, sv[2][b], fmaf(q4.w, sv[3][b], acc[i][b]))));
        }
    }
    for (int d = D4; d < D; d++) {
        float sv[CW];
        srow(d, sv);
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const float qv = Qs[(warp * 8 + i) * Dp + d];
#pragma unroll
            for (int b = 0; b < CW; b++) acc[i][b] = fmaf(qv, sv[b], acc[i][b]);
        }
    }
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const float f = pw[warp * 8 + i];
#pragma unroll
        for (int b = 0; b < CW; b++) acc[i][b] *= f;
    }
    for (int j = 0; j < RC; j += 4) {
        float f[4][CW];
#pragma unroll
        for (int r = 0; r < 4; r++) {
            if constexpr (CW == 4) { const float4 x = *reinterpret_cast<const float4 *>(Vs + (j + r) * NC + lane * 4); f[r][0] = x.x; f[r][1] = x.y; f[r][2] = x.z; f[r][3] = x.w; }
            else { const float2 x = *reinterpret_cast<const float2 *>(Vs + (j + r) * NC + lane * 2); f[r][0] = x.x; f[r][1] = x.y; }
        }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const float4 w = *reinterpret_cast<const float4 *>(As + (warp * 8 + i) * AP + j);
#pragma unroll
            for (int b = 0; b < CW; b++) acc[i][b] = fmaf(w.x, f[0][b], fmaf(w.y, f[1][b], fmaf(w.z, f[2][b], fmaf(w.w, f[3][b], acc[i][b]))));
        }
    }
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const int tl = warp * 8 + i;
        if (tl >= nt) continue;
#pragma unroll
        for (int b = 0; b < CW; b++) if (v + b < V) a.O[(size_t) (t0 + tl) * a.H * V + (size_t) h * V + v + b] = acc[i][b];
    }
    if (a.norm && blockIdx.z == 0) {                    // n . q: the scores' weighted sum plus the entry state's share
        const float * nc = Sc + (size_t) D * V;
        float dq[8] = { 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f };
        for (int d = lane; d < D; d += 32) {
            const float n = __ldg(nc + d);
#pragma unroll
            for (int i = 0; i < 8; i++) dq[i] = fmaf(n, Qs[(warp * 8 + i) * Dp + d], dq[i]);
        }
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int tl = warp * 8 + i;
            const float r = warp_sum(fmaf(pw[tl], dq[i], As[tl * AP + lane]));
            if (lane == 0 && tl < nt) a.den[(size_t) (t0 + tl) * a.H + h] = r;
        }
    }
}

// ---- mLSTM ----------------------------------------------------------------------------------------------------------------------
// Gate pre-activations (biases included) become log gates i = cap tanh(. / cap) and f = log sigmoid(cap tanh(. / cap)); with the
// running maximum m_t = max(f + m_(t-1), i), m starting at 0, the recurrence is S_t = a S_(t-1) + b k v^T and n_t alike, with
// a = exp(f + m_(t-1) - m_t) and b = exp(i - m_t), both at most 1.
__device__ __forceinline__ float log_sigmoidf_(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float mlstm_log_in(float raw, float cap) { return cap * tanhf(raw / cap); }
__device__ __forceinline__ float mlstm_log_keep(float raw, float cap) { return log_sigmoidf_(cap * tanhf(raw / cap)); }
// the read-out's divisor, from n . q (scaled like the query) and m
__device__ __forceinline__ float mlstm_divisor(float nq, float m) { return fmaxf(fabsf(nq), expf(-m)) + 1e-6f; }
// portions of several tokens: AB[t] = [ a: H | b: H | m: H ]. One block per head: log gates of all tokens at once into shared memory
// (3 T floats, dynamic), the maximum from token to token in order by one warp (two dependent operations each), then a and b of
// all tokens at once. m_state [H] is part of the sequence's state.
__global__ void __launch_bounds__(256) k_mlstm_gates(const float * __restrict__ P, int ldp, int i_off, int f_off, float cap, int T, int H,
                                                     float * __restrict__ m_state, float * __restrict__ AB, int ld_ab) {
    extern __shared__ float msm[];
    float * li = msm, * lf = msm + T, * mx = msm + 2 * T;
    const int h = blockIdx.x;
    const float m0 = m_state[h];
    for (int t = threadIdx.x; t < T; t += blockDim.x) {
        li[t] = mlstm_log_in(P[(size_t) t * ldp + i_off + h], cap);
        lf[t] = mlstm_log_keep(P[(size_t) t * ldp + f_off + h], cap);
    }
    __syncthreads();
    if (threadIdx.x < 32) {
        float m = m0;
        int t = 0;
        for (; t + 8 <= T; t += 8) {
            float f[8], i[8];
#pragma unroll
            for (int k = 0; k < 8; k++) { f[k] = lf[t + k]; i[k] = li[t + k]; }
#pragma unroll
            for (int k = 0; k < 8; k++) { m = fmaxf(f[k] + m, i[k]); if (threadIdx.x == 0) mx[t + k] = m; }
        }
        for (; t < T; t++) { m = fmaxf(lf[t] + m, li[t]); if (threadIdx.x == 0) mx[t] = m; }
        if (threadIdx.x == 0) m_state[h] = m;
    }
    __syncthreads();
    for (int t = threadIdx.x; t < T; t += blockDim.x) {
        float * o = AB + (size_t) t * ld_ab;
        const float m = mx[t];
        o[h] = expf(lf[t] + (t ? mx[t - 1] : m0) - m);
        o[H + h] = expf(li[t] - m);
        o[2 * H + h] = m;
    }
}

// ---- one token, a whole mixer core in one launch: gates, state update, read-out, its norm and gate; one block per head -----------
// The same four-lanes-per-column layout as the walk, tile by tile of up to 128 columns; the head's read-out is kept in shared
// memory (V + 1 floats, dynamic) until its sum of squares is known (eps inside the root).
//   TOKEN_RETENTION  q and k rotated by the position on the way into shared memory, k scaled; a = decay[h], b = 1;
//                    A[h] = o / rms(o) * silu(gate)
//   TOKEN_MLSTM      a, b and the running maximum from the two gate pre-activations; q scaled; o over its divisor first;
//                    A[h] = o / rms(o) * w[h] * sigmoid(gate)
enum { TOKEN_RETENTION = 0, TOKEN_MLSTM = 1 };
struct OuterToken {
    const float * P; int q_off, k_off, v_off, g_off, i_off, f_off;
    const float * decay; RopeArgs rope; float k_scale, q_scale;
    const StepState * st;
    float cap; const float * w;
    int H, D, V; float eps;
    float * S; long long head_stride;           // [D][V], then n [D] (mLSTM)
    float * m_state;
    float * A;
};
template <int DMAX, int KIND>
__global__ void __launch_bounds__(512) k_outer_token(const OuterToken a) {
    constexpr int DR = DMAX / GD_RG, ROW = GD_RG * (DR + GD_PAD);
    extern __shared__ float o_s[];                      // [V] read-out, [V]: n . q
    __shared__ __align__(16) float qs[ROW], ks[ROW];
    __shared__ float red[16];
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rg = lane & 3, ncols = blockDim.x / GD_RG, D = a.D, V = a.V;
    const float * q = a.P + a.q_off + (size_t) h * D, * k = a.P + a.k_off + (size_t) h * D;
    float g, b = 1.f, m = 0.f;
    if constexpr (KIND == TOKEN_MLSTM) {
        const float li = mlstm_log_in(a.P[a.i_off + h], a.cap), lf = mlstm_log_keep(a.P[a.f_off + h], a.cap), m0 = a.m_state[h];
        m = fmaxf(lf + m0, li);
        g = expf(lf + m0 - m); b = expf(li - m);
    } else g = a.decay[h];
    float * Sh = a.S + (size_t) h * a.head_stride;
    constexpr int NL = (DMAX + 31) / 32;                // mLSTM: warp 0 keeps the normaliser, a lane every 32nd entry
    float nv[NL];
    if (KIND == TOKEN_MLSTM && warp == 0) {
#pragma unroll
        for (int i = 0; i < NL; i++) nv[i] = lane + 32 * i < D ? Sh[(size_t) D * V + lane + 32 * i] : 0.f;
    }
    for (int i = tid; i < 2 * DMAX; i += blockDim.x) {
        const bool is_k = i >= DMAX;
        const int d = is_k ? i - DMAX : i, at = (d / DR) * (DR + GD_PAD) + d % DR;
        float v = 0.f;
        if (d < D) {
            const float * x = is_k ? k : q;
            if constexpr (KIND == TOKEN_RETENTION) {
                const int pos = a.st->pos0, half = a.rope.dims / 2;
                if (d < half) { float u, w; rope_pair(a.rope, pos, d, x[d], x[d + half], u, w); v = u; }
                else if (d < a.rope.dims) { float u, w; rope_pair(a.rope, pos, d - half, x[d - half], x[d], u, w); v = w; }
                else v = x[d];
                if (is_k) v *= a.k_scale;
            } else v = is_k ? x[d] : x[d] * a.q_scale;
        }
        (is_k ? ks : qs)[at] = v;
    }
    __syncthreads();
    if (KIND == TOKEN_MLSTM && warp == 0) {
        if (lane == 0) a.m_state[h] = m;                // every thread has read the old one
        float nq = 0.f;
#pragma unroll
        for (int i = 0; i < NL; i++) {
            const int d = lane + 32 * i, at = (d / DR) * (DR + GD_PAD) + d % DR;
            if (d < D) {
                nv[i] = fmaf(g, nv[i], ks[at] * b);
                Sh[(size_t) D * V + d] = nv[i];
                nq = fmaf(nv[i], qs[at], nq);
            }
        }
        nq = warp_sum(nq);
        if (lane == 0) o_s[V] = nq;
    }
    const int base = rg * (DR + GD_PAD), cl = warp * 8 + (lane >> 2);
    float ss = 0.f;
    for (int c0 = 0; c0 < V; c0 += ncols) {
        const int col = c0 + cl;
        const bool live = col < V;
        const float v = live ? b * a.P[a.v_off + (size_t) h * V + col] : 0.f;
        float * Sc = Sh + col;
        float op[4] = { 0.f, 0.f, 0.f, 0.f };
        constexpr int CH = DR < 16 ? DR : 16;           // rows whose loads are in flight together (the stores would order them otherwise)
#pragma unroll 1
        for (int i0 = 0; i0 < DR; i0 += CH) {
            float sv[CH];
#pragma unroll
            for (int i = 0; i < CH; i++) { const int d = rg * DR + i0 + i; sv[i] = (live && d < D) ? Sc[(size_t) d * V] : 0.f; }
#pragma unroll
            for (int i = 0; i < CH; i++) {
                const int d = rg * DR + i0 + i;
                sv[i] = fmaf(g, sv[i], ks[base + i0 + i] * v);
                if (live && d < D) Sc[(size_t) d * V] = sv[i];
                op[i & 3] = fmaf(sv[i], qs[base + i0 + i], op[i & 3]);
            }
        }
        float o = (op[0] + op[1]) + (op[2] + op[3]);
        o += __shfl_xor_sync(0xffffffffu, o, 1);
        o += __shfl_xor_sync(0xffffffffu, o, 2);
        if (rg == 0 && live) { o_s[col] = o; ss = fmaf(o, o, ss); }
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < (int) (blockDim.x >> 5); w++) tot += red[w];
    if constexpr (KIND == TOKEN_MLSTM) {
        const float f = 1.0f / mlstm_divisor(o_s[V], m);
        const float r = f / sqrtf(tot * f * f / (float) V + a.eps);
        for (int i = tid; i < V; i += blockDim.x) a.A[(size_t) h * V + i] = o_s[i] * r * a.w[(size_t) h * V + i] * sigmoidf_(a.P[a.g_off + (size_t) h * V + i]);
    } else {
        const float r = 1.0f / sqrtf(tot / (float) V + a.eps);
        for (int i = tid; i < V; i += blockDim.x) a.A[(size_t) h * V + i] = o_s[i] * r * siluf_(a.P[a.g_off + (size_t) h * V + i]);
    }
}
// portions of several tokens, mLSTM's last step: each head's read-out (times the query's scale, over its divisor) over its root mean
// square, times a weight [H][V], times sigmoid(gate). m sits in the third part of a row of the gate table. One warp per (token, head).
__global__ void k_mlstm_out(const float * __restrict__ O, const float * __restrict__ den, const float * __restrict__ AB, int ld_ab, float q_scale, const float * __restrict__ P, int ldp, int gate_off,
                            int H, int V, const float * __restrict__ w, float eps, float * __restrict__ A) {
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int h = blockIdx.y * nw + warp; h < H; h += gridDim.y * nw) {
        const size_t at = (size_t) t * H * V + (size_t) h * V;
        const float * gp = P + (size_t) t * ldp + gate_off + (size_t) h * V;
        const float f = q_scale / mlstm_divisor(den[(size_t) t * H + h] * q_scale, AB[(size_t) t * ld_ab + 2 * H + h]);
        float ss = 0.f;
        for (int i = lane; i < V; i += 32) { const float o = O[at + i] * f; ss = fmaf(o, o, ss); }
        ss = warp_sum(ss);
        const float r = f / sqrtf(ss / (float) V + eps);
        for (int i = lane; i < V; i += 32) A[at + i] = O[at + i] * r * w[(size_t) h * V + i] * sigmoidf_(gp[i]);
    }
}

// ---- state-space mixer's read-out: y = (o + skip[h] x) silu(z), then each of `parts` equal parts of the row over its own root mean
// square (eps inside the root), times a weight. One block per (token, part).
__global__ void __launch_bounds__(1024) k_gated_part_norm(const float * __restrict__ O, const float * __restrict__ X, int ldx, const float * __restrict__ skip, const float * __restrict__ Z, int ldz,
                                                          int inner, int V, int parts, const float * __restrict__ w, float eps, float * __restrict__ A) {
    __shared__ float red[32];
    constexpr int OWN = 8;                              // entries a thread keeps in registers until the part's sum of squares is known
    const int t = blockIdx.x, n = inner / parts, i0 = blockIdx.y * n, nt = blockDim.x;
    const float * o = O + (size_t) t * inner + i0, * x = X + (size_t) t * ldx + i0, * z = Z + (size_t) t * ldz + i0;
    float * out = A + (size_t) t * inner + i0;
    float keep[OWN], ss = 0.f;
#pragma unroll
    for (int k = 0; k < OWN; k++) {
        const int i = threadIdx.x + k * nt;
        keep[k] = i < n ? fmaf(skip[(i0 + i) / V], x[i], o[i]) * siluf_(z[i]) : 0.f;
    }
#pragma unroll
    for (int k = 0; k < OWN; k++) ss = fmaf(keep[k], keep[k], ss);
    for (int i = threadIdx.x + OWN * nt; i < n; i += nt) {
        const float y = fmaf(skip[(i0 + i) / V], x[i], o[i]) * siluf_(z[i]);
        out[i] = y;
        ss = fmaf(y, y, ss);
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int k = 0; k < (nt >> 5); k++) tot += red[k];
    const float r = 1.0f / sqrtf(tot / (float) n + eps);
#pragma unroll
    for (int k = 0; k < OWN; k++) { const int i = threadIdx.x + k * nt; if (i < n) out[i] = keep[k] * r * w[i0 + i]; }
    for (int i = threadIdx.x + OWN * nt; i < n; i += nt) out[i] *= r * w[i0 + i];
}

// ---- selective scan -----------------------------------------------------------------------------------------------------------------
// Per channel c and state entry n: S <- exp(dt_c A[c][n]) S + dt_c x_c B[n], y_c = sum_n S C[n] + skip[c] x_c, A[t][c] = y_c silu(z_c),
// with dt_c = softplus(raw dt_c) (bias included) and A[c][n] = -exp(A_log[c][n]). The state [inner][N] stays in registers for the
// whole portion: LANES neighbouring lanes share a channel, each holding NS of its entries. The inputs of TT tokens arrive in shared
// memory by asynchronous copies while the tokens before them are walked (two buffers); step sizes and gates are taken there once per
// (token, channel).
// Long portions are cut into segments of `seg` tokens that run side by side. A segment takes the state before it to
// exp(A sum_t dt_t) S + L, with L what it leaves when it starts from zero, so:
//   SEL_FIRST   segments 0 .. n - 2: segment 0 is the walk itself from the sequence's state, the others start from zero and write
//               nothing but L; all leave L (segment 0: the state after it) and their sum of step sizes
//   SEL_REST    segments 1 .. n - 1: the entry state folded from what the segments before left, then the walk; the last one
//               leaves the sequence's state
// SEL_WHOLE is the walk over a short portion.
enum { SEL_WHOLE = 0, SEL_FIRST = 1, SEL_REST = 2 };
struct SelScan {
    const float * X; int ldx;               // convolved inputs [T][inner]
    const float * dt; int ldt;              // raw step sizes (bias included) [T][inner]
    const float * BC; int ldb; int b_off, c_off;
    const float * Z; int ldz;
    const float * A_log; const float * skip;
    float * S;
    int T, inner, N;
    float * A;                              // [T][inner]
    int seg;                                // tokens per segment
    float * L; float * sum;                 // [segments][inner][N], [segments][inner]
};
template <int LANES, int NS, int MODE>
__global__ void __launch_bounds__(256) k_selective_scan(const SelScan a) {
    constexpr int NCH = 256 / LANES, NM = LANES * NS, TT = NM > 64 ? 8 : 16;
    __shared__ __align__(16) float xs[2][TT][NCH], ds[2][TT][NCH], zs[2][TT][NCH], bs[2][TT][NM], cs[2][TT][NM];
    const int tid = threadIdx.x, rg = tid % LANES, cl = tid / LANES, c0 = blockIdx.x * NCH, c = c0 + cl, N = a.N;
    const bool live = c < a.inner;
    const int sg = MODE == SEL_WHOLE ? 0 : MODE == SEL_FIRST ? blockIdx.y : blockIdx.y + 1;
    const int T0 = MODE == SEL_WHOLE ? 0 : sg * a.seg, T1 = MODE == SEL_WHOLE ? a.T : min(a.T, T0 + a.seg);
    const bool emits = MODE != SEL_FIRST || sg == 0;
    const auto stage = [&](int t0, int buf) {
        const int nt = min(TT, T1 - t0);
        for (int i = tid; i < nt * NCH; i += 256) {
            const int tt = i / NCH, k = i % NCH;
            const bool in = c0 + k < a.inner;
            const size_t t = (size_t) (t0 + tt), ch = in ? c0 + k : 0;
            cp_async4(&xs[buf][tt][k], a.X + t * a.ldx + ch, in);
            cp_async4(&ds[buf][tt][k], a.dt + t * a.ldt + ch, in);
            if (emits) cp_async4(&zs[buf][tt][k], a.Z + t * a.ldz + ch, in);
        }
        for (int i = tid; i < nt * NM; i += 256) {
            const int tt = i / NM, n = i % NM;
            const bool in = n < N;
            const float * p = a.BC + (size_t) (t0 + tt) * a.ldb + (in ? n : 0);
            cp_async4(&bs[buf][tt][n], p + a.b_off, in);
            if (emits) cp_async4(&cs[buf][tt][n], p + a.c_off, in);
        }
    };
    stage(T0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    float s[NS], rate[NS];
    float * Sc = a.S + (size_t) (live ? c : 0) * N;
#pragma unroll
    for (int i = 0; i < NS; i++) {
        const int n = rg * NS + i;
        const bool in = live && n < N;
        s[i] = in && (MODE == SEL_WHOLE || (MODE == SEL_FIRST && sg == 0)) ? Sc[n] : 0.f;
        rate[i] = in ? -1.4426950408889634f * expf(a.A_log[(size_t) c * N + n]) : 0.f;      // in powers of two
    }
    if (MODE == SEL_REST) {
        for (int k = 0; k < sg; k++) {
            const size_t at = (size_t) k * a.inner + (live ? c : 0);
            const float sum = a.sum[at];
#pragma unroll
            for (int i = 0; i < NS; i++) { const int n = rg * NS + i; if (live && n < N) s[i] = fmaf(exp2f(sum * rate[i]), s[i], a.L[at * N + n]); }
        }
    }
    const float skip = live ? a.skip[c] : 0.f;
    float total = 0.f;
    for (int t0 = T0, buf = 0; t0 < T1; t0 += TT, buf ^= 1) {
        const int nt = min(TT, T1 - t0);
        if (t0 + TT < T1) stage(t0 + TT, buf ^ 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        for (int i = tid; i < nt * NCH; i += 256) {
            float & d = ds[buf][i / NCH][i % NCH], & z = zs[buf][i / NCH][i % NCH];
            d = softplusf_(d);
            if (emits) z = siluf_(z);
        }
        __syncthreads();
        if (!emits) {
#pragma unroll 4
            for (int tt = 0; tt < nt; tt++) {
                const float dt = ds[buf][tt][cl], dx = dt * xs[buf][tt][cl];
                total += dt;
#pragma unroll
                for (int i = 0; i < NS; i++) s[i] = fmaf(exp2f(dt * rate[i]), s[i], dx * bs[buf][tt][rg * NS + i]);
            }
            __syncthreads();
            continue;
        }
#pragma unroll 4
        for (int tt = 0; tt < nt; tt++) {
            const float dt = ds[buf][tt][cl], x = xs[buf][tt][cl], dx = dt * x;
            float y = 0.f;
            if (MODE == SEL_FIRST) total += dt;
#pragma unroll
            for (int i = 0; i < NS; i++) {
                s[i] = fmaf(exp2f(dt * rate[i]), s[i], dx * bs[buf][tt][rg * NS + i]);
                y = fmaf(s[i], cs[buf][tt][rg * NS + i], y);
            }
#pragma unroll
            for (int o = 1; o < LANES; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
            if (rg == 0 && live) a.A[(size_t) (t0 + tt) * a.inner + c] = fmaf(skip, x, y) * zs[buf][tt][cl];
        }
        __syncthreads();
    }
    if (MODE == SEL_REST && T1 < a.T) return;           // only the last segment's state is the sequence's
    if (live) {
        float * to = MODE == SEL_FIRST ? a.L + ((size_t) sg * a.inner + c) * N : Sc;
#pragma unroll
        for (int i = 0; i < NS; i++) { const int n = rg * NS + i; if (n < N) to[n] = s[i]; }
        if (MODE == SEL_FIRST && rg == 0) a.sum[(size_t) sg * a.inner + c] = total;
    }
}
// one token: the step size's low-rank product (Wdt [inner][R], bias) is part of the same launch; the lanes of a channel share it
template <typename WT, int LANES, int NS>
__global__ void __launch_bounds__(256) k_selective_token(const SelScan a, const WT * __restrict__ Wdt, const float * __restrict__ bdt, int R) {
    constexpr int NCH = 256 / LANES;
    extern __shared__ float low[];                      // [R] the step size's low-rank input
    const int tid = threadIdx.x, rg = tid % LANES, cl = tid / LANES, c = blockIdx.x * NCH + cl, N = a.N;
    const bool live = c < a.inner;
    float s[NS], rate[NS], bn[NS], cn[NS];
    float * Sc = a.S + (size_t) (live ? c : 0) * N;
#pragma unroll
    for (int i = 0; i < NS; i++) {                      // asked for before anything is waited on
        const int n = rg * NS + i;
        const bool in = live && n < N;
        s[i] = in ? Sc[n] : 0.f;
        rate[i] = in ? a.A_log[(size_t) c * N + n] : 0.f;
        bn[i] = in ? a.BC[a.b_off + n] : 0.f;
        cn[i] = in ? a.BC[a.c_off + n] : 0.f;
    }
    const float x = live ? a.X[c] : 0.f, z = live ? a.Z[c] : 0.f, skip = live ? a.skip[c] : 0.f, bias = live ? bdt[c] : 0.f;
    for (int i = tid; i < R; i += 256) low[i] = a.BC[i];
    __syncthreads();
    float d = 0.f;
    if (live) {
#pragma unroll 8
        for (int i = rg; i < R; i += LANES) d = fmaf(wf(Wdt, (size_t) c * R + i), low[i], d);
    }
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
    const float dt = softplusf_(d + bias), dx = dt * x;
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NS; i++) {
        s[i] = fmaf(exp2f(dt * (-1.4426950408889634f * expf(rate[i]))), s[i], dx * bn[i]);
        y = fmaf(s[i], cn[i], y);
        const int n = rg * NS + i;
        if (live && n < N) Sc[n] = s[i];
    }
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (rg == 0 && live) a.A[c] = fmaf(skip, x, y) * siluf_(z);
}

}  // namespace stk
}  // namespace b200
