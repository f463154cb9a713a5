// stack_kernels_side.cuh — CUDA kernels (sm_100a) of layer-stack blocks whose two sub-layers read one normed input and whose layers
// end with an input of the token's own, on top of stack_kernels.cuh and stack_kernels_hyper.cuh: an embedding that adds a row hashed
// from the token and the one before it, the sum that ends both sub-layers with the norm that follows, and the per-layer token input
// x += norm(W_p (gelu(W_g x) e)) with e a slice of a per-token table.
// Every size and constant is a kernel argument. Norms, the residual sum and what lies between the products are float32.
#pragma once
#include "stack_kernels.cuh"
#include "stack_kernels_hyper.cuh"

namespace b200 {
namespace stk {

// ---- embedding with a table of token pairs: X[t] = embed[tok] + pair[row], row = (prev mul_prev + tok mul_cur) mod buckets, or the extra
// row `buckets` for a sequence's first token (st->prev < 0 in front of the step's first); then Hn[t] = X / rms(X) * w, the first
// layer's input. One block per token (hc_threads threads).
struct PairTable { const void * w; unsigned long long mul_prev, mul_cur, buckets; };      // w == nullptr: no such table
template <typename WT>
__global__ void __launch_bounds__(1024) k_embed_pair(const WT * __restrict__ embed, PairTable pt, const StepState * __restrict__ st, const int32_t * __restrict__ tokens,
                                                    int E, int n_vocab, const float * __restrict__ w, float eps, float * __restrict__ X, float * __restrict__ Hn) {
    __shared__ float red[32];
    const int t = blockIdx.x, nt = blockDim.x;
    const auto id = [&](int i) { const int v = tokens[i]; return v < 0 ? 0 : v >= n_vocab ? n_vocab - 1 : v; };      // ids are validated on the host; never read outside the table
    const int tok = id(t), prev = t > 0 ? id(t - 1) : st->prev;
    const unsigned long long pr = prev < 0 ? pt.buckets : ((unsigned long long) prev * pt.mul_prev + (unsigned long long) tok * pt.mul_cur) % (pt.buckets ? pt.buckets : 1ull);
    const WT * a = embed + (size_t) tok * E, * b = reinterpret_cast<const WT *>(pt.w) + (size_t) pr * E;
    const size_t row = (size_t) t * E;
    float ss = 0.f;
    for (int i = threadIdx.x; i < E; i += nt) {
        const float x = pt.w ? wf(a, i) + wf(b, i) : wf(a, i);
        X[row + i] = x;
        ss = fmaf(x, x, ss);
    }
    ss = block_sum(ss, red);
    const float r = 1.0f / sqrtf(ss / (float) E + eps);
    for (int i = threadIdx.x; i < E; i += nt) Hn[row + i] = X[row + i] * r * w[i];        // what this thread wrote
}

// ---- end of two sub-layers that read the same input: X[t] += Ya[t] + Yb[t] + sum_k wt[t][k] Yk[slot(t, k)] (Yb, Yk may be absent; slot_of ==
// nullptr: slot t top + k), then, when nw is given, Hn[t] = X / rms(X) * nw. One block per token; VEC-entry chunks of the row are dealt
// over the threads, which keep SUM_OWN of them in registers.
struct SumArgs {
    float * X; int E; float eps;
    const float * Ya; const float * Yb;
    const float * Yk; const float * wt; const int32_t * slot_of; int top;
    const float * nw; float * Hn;
};
constexpr int SUM_OWN = 2;
template <int VEC> __device__ __forceinline__ void sum_chunk(const SumArgs & a, int t, int i, float (&x)[VEC]) {
    const size_t at = (size_t) t * a.E + i;
    float v[VEC];
    ld_chunk<VEC>(a.X + at, x);
    ld_chunk<VEC>(a.Ya + at, v);
#pragma unroll
    for (int e = 0; e < VEC; e++) x[e] += v[e];
    if (a.Yb) {
        ld_chunk<VEC>(a.Yb + at, v);
#pragma unroll
        for (int e = 0; e < VEC; e++) x[e] += v[e];
    }
    if (a.Yk) {
#pragma unroll 4
        for (int k = 0; k < a.top; k++) {
            const int s = t * a.top + k;
            const float w = a.wt[s];
            ld_chunk<VEC>(a.Yk + (size_t) (a.slot_of ? a.slot_of[s] : s) * a.E + i, v);
#pragma unroll
            for (int e = 0; e < VEC; e++) x[e] = fmaf(w, v[e], x[e]);
        }
    }
}
template <int VEC>
__global__ void __launch_bounds__(1024) k_sum_join(const SumArgs a) {
    __shared__ float red[32];
    const int t = blockIdx.x, nt = blockDim.x, nchunk = a.E / VEC;
    const size_t row = (size_t) t * a.E;
    float own[SUM_OWN][VEC], ss = 0.f;
#pragma unroll
    for (int k = 0; k < SUM_OWN; k++) {
        const int c = threadIdx.x + k * nt;
        if (c < nchunk) {
            sum_chunk<VEC>(a, t, c * VEC, own[k]);
            st_chunk<VEC>(a.X + row + c * VEC, own[k]);
#pragma unroll
            for (int e = 0; e < VEC; e++) ss = fmaf(own[k][e], own[k][e], ss);
        }
    }
    for (int c = threadIdx.x + SUM_OWN * nt; c < nchunk; c += nt) {
        float x[VEC];
        sum_chunk<VEC>(a, t, c * VEC, x);
        st_chunk<VEC>(a.X + row + c * VEC, x);
#pragma unroll
        for (int e = 0; e < VEC; e++) ss = fmaf(x[e], x[e], ss);
    }
    if (!a.nw) return;
    ss = block_sum(ss, red);
    const float r = 1.0f / sqrtf(ss / (float) a.E + a.eps);
    const auto finish = [&](int i, float (&x)[VEC]) {
        float w[VEC];
        ld_chunk<VEC>(a.nw + i, w);
#pragma unroll
        for (int e = 0; e < VEC; e++) x[e] = x[e] * r * w[e];
        st_chunk<VEC>(a.Hn + row + i, x);
    };
#pragma unroll
    for (int k = 0; k < SUM_OWN; k++) { const int c = threadIdx.x + k * nt; if (c < nchunk) finish(c * VEC, own[k]); }
    for (int c = threadIdx.x + SUM_OWN * nt; c < nchunk; c += nt) {
        float x[VEC];
        ld_chunk<VEC>(a.X + row + c * VEC, x);             // what this thread wrote
        finish(c * VEC, x);
    }
}

// ---- the token's own input of a layer: x += y / rms(y) * wn, y = W_p (gelu(W_g x) e), e = table[token][off .. off + dim) ------------------
struct SideW {
    const void * table; int ld, off, dim;       // [vocab][ld] in the model's storage type
    const void * Wg; const void * Wp;           // [dim][E], [E][dim]
    const float * wn;
};
// prompt portions, between the two products: Z[t][i] <- gelu(Z[t][i]) e_i. grid (T, slices of dim)
template <typename WT>
__global__ void k_side_gate(float * __restrict__ Z, SideW s, const int32_t * __restrict__ tokens, int n_vocab) {
    const int t = blockIdx.x, i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= s.dim) return;
    int tok = tokens[t];
    tok = tok < 0 ? 0 : tok >= n_vocab ? n_vocab - 1 : tok;
    float * z = Z + (size_t) t * s.dim + i;
    *z = gelu_tanhf_(*z) * wf(reinterpret_cast<const WT *>(s.table), (size_t) tok * s.ld + s.off + i);
}

// 16 bytes of a weight row against float32 entries in shared memory
__device__ __forceinline__ float dot16(const uint4 & raw, const float * x, const __nv_bfloat16 *) {
    const uint32_t u[4] = { raw.x, raw.y, raw.z, raw.w };
    const float4 p = *reinterpret_cast<const float4 *>(x), q = *reinterpret_cast<const float4 *>(x + 4);
    const float f[8] = { p.x, p.y, p.z, p.w, q.x, q.y, q.z, q.w };
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 4; i++) { s = fmaf(__uint_as_float(u[i] << 16), f[2 * i], s); s = fmaf(__uint_as_float(u[i] & 0xffff0000u), f[2 * i + 1], s); }
    return s;
}
__device__ __forceinline__ float dot16(const uint4 & raw, const float * x, const float *) {
    const float4 p = *reinterpret_cast<const float4 *>(x);
    return fmaf(__uint_as_float(raw.x), p.x, fmaf(__uint_as_float(raw.y), p.y, fmaf(__uint_as_float(raw.z), p.z, __uint_as_float(raw.w) * p.w)));
}

// Steps of few tokens: the whole end of a layer in one launch — the sum of both sub-layers, the token's own input and the norm that
// follows. A thread-block cluster of END_CTAS blocks per token: every block forms the summed row in its shared memory, takes a share of
// W_g's rows and writes the results into all blocks' shared memory; then a share of W_p's rows, the residual entries of that share, and
// their part of both sums of squares, exchanged the same way. No block rewrites X before all have read it. grid (END_CTAS, T).
constexpr int END_CTAS = 8, END_THREADS = 512;
inline int end_slice(int E) { return ((E + END_CTAS - 1) / END_CTAS + 3) / 4 * 4; }
inline size_t end_smem(int E, int dim) { return ((size_t) (E + 3) / 4 * 4 + (size_t) (dim + 3) / 4 * 4 + (size_t) end_slice(E)) * 4; }
template <typename WT>
__global__ void __cluster_dims__(END_CTAS, 1, 1) __launch_bounds__(END_THREADS)
k_layer_end(const SumArgs a, const SideW s, const int32_t * __restrict__ tokens, int n_vocab, int slice, int vec_g, int vec_p, int lpr) {
    namespace cg = cooperative_groups;
    cg::cluster_group cluster = cg::this_cluster();
    extern __shared__ __align__(16) float esm[];
    __shared__ float red[32], part[2][END_CTAS];
    constexpr int VEC = 16 / (int) sizeof(WT), NW = END_THREADS / 32;
    const int E = a.E, dim = s.dim, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rank = (int) cluster.block_rank(), t = blockIdx.y;
    float * xs = esm, * g = xs + (E + 3) / 4 * 4, * ys = g + (dim + 3) / 4 * 4;
    cluster.barrier_arrive();                              // waited for before the first store into another block's shared memory
    const int e0 = min(rank * slice, E), e1 = min(e0 + slice, E);
    const int dper = (dim + END_CTAS - 1) / END_CTAS, d0 = min(rank * dper, dim), d1 = min(d0 + dper, dim);
    const WT * Wg = reinterpret_cast<const WT *>(s.Wg), * Wp = reinterpret_cast<const WT *>(s.Wp);
    {   // both shares of weights are on their way to L2 while the row is summed
        const char * p = reinterpret_cast<const char *>(Wg + (size_t) d0 * E), * q = reinterpret_cast<const char *>(Wp + (size_t) e0 * dim);
        const size_t np = (size_t) (d1 - d0) * E * sizeof(WT), nq = (size_t) (e1 - e0) * dim * sizeof(WT);
        for (size_t b = (size_t) tid * 128; b < np; b += (size_t) END_THREADS * 128) asm volatile("prefetch.global.L2 [%0];" :: "l"(p + b));
        for (size_t b = (size_t) tid * 128; b < nq; b += (size_t) END_THREADS * 128) asm volatile("prefetch.global.L2 [%0];" :: "l"(q + b));
    }
    int tok = tokens[t];
    tok = tok < 0 ? 0 : tok >= n_vocab ? n_vocab - 1 : tok;
    const WT * e = reinterpret_cast<const WT *>(s.table) + (size_t) tok * s.ld + s.off;
    if ((E & 3) == 0) {
        for (int i = tid * 4; i < E; i += END_THREADS * 4) { float v[4]; sum_chunk<4>(a, t, i, v); st_chunk<4>(xs + i, v); }
    } else {
        for (int i = tid; i < E; i += END_THREADS) { float v[1]; sum_chunk<1>(a, t, i, v); xs[i] = v[0]; }
    }
    __syncthreads();
    cluster.barrier_wait();
    for (int r = d0 + warp; r < d1; r += NW) {             // a warp per row of W_g
        const WT * w = Wg + (size_t) r * E;
        const float er = wf(e, r);
        float acc = 0.f;
        if (vec_g) {
#pragma unroll 8
            for (int k = lane * VEC; k < E; k += 32 * VEC) acc += dot16(__ldg(reinterpret_cast<const uint4 *>(w + k)), xs + k, w);
        } else {
            for (int k = lane; k < E; k += 32) acc = fmaf(wf(w, k), xs[k], acc);
        }
        acc = warp_sum(acc);
        if (lane < END_CTAS) *cluster.map_shared_rank(g + r, lane) = gelu_tanhf_(acc) * er;
    }
    cluster.sync();
    float ss = 0.f;
    const int sub = tid % lpr, grp = tid / lpr, ngrp = END_THREADS / lpr;      // lpr lanes per row of W_p (a power of two)
#pragma unroll 4
    for (int base = e0; base < e1; base += ngrp) {
        const int row = base + grp;
        float acc = 0.f;
        if (row < e1) {
            const WT * w = Wp + (size_t) row * dim;
            if (vec_p) { for (int k = sub * VEC; k < dim; k += lpr * VEC) acc += dot16(__ldg(reinterpret_cast<const uint4 *>(w + k)), g + k, w); }
            else { for (int k = sub; k < dim; k += lpr) acc = fmaf(wf(w, k), g[k], acc); }
        }
        for (int o = lpr >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (sub == 0 && row < e1) { ys[row - e0] = acc; ss = fmaf(acc, acc, ss); }
    }
    ss = block_sum(ss, red);
    if (tid < END_CTAS) *cluster.map_shared_rank(&part[0][rank], tid) = ss;
    cluster.sync();
    float tot = 0.f;
#pragma unroll
    for (int r = 0; r < END_CTAS; r++) tot += part[0][r];  // the same order in every block
    const float ry = 1.0f / sqrtf(tot / (float) E + a.eps);
    ss = 0.f;
    for (int i = e0 + tid; i < e1; i += END_THREADS) {
        const float v = fmaf(ys[i - e0] * ry, s.wn[i], xs[i]);
        xs[i] = v;
        a.X[(size_t) t * E + i] = v;
        ss = fmaf(v, v, ss);
    }
    if (!a.nw) return;                                     // no block reads another's shared memory any more
    ss = block_sum(ss, red);
    if (tid < END_CTAS) *cluster.map_shared_rank(&part[1][rank], tid) = ss;
    cluster.sync();
    tot = 0.f;
#pragma unroll
    for (int r = 0; r < END_CTAS; r++) tot += part[1][r];
    const float rx = 1.0f / sqrtf(tot / (float) E + a.eps);
    for (int i = e0 + tid; i < e1; i += END_THREADS) a.Hn[(size_t) t * E + i] = xs[i] * rx * a.nw[i];
}

}  // namespace stk
}  // namespace b200
