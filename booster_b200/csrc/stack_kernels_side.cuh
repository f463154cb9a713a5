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

// Steps of few tokens: the end of a layer in two launches wide enough to fetch both matrices at full bandwidth. Weights are asked for
// before anything they wait for.
// First: every block sums the row (as k_sum_join does, but into Xs: X stays as it is while others read it) into shared memory and takes
// SIDE_ROWS rows of W_g: G[t][i] = gelu(W_g x) e_i. grid (ceil(dim / SIDE_ROWS), T), E floats of shared memory.
constexpr int SIDE_THREADS = 512, SIDE_ROWS = 2, SIDE_MOST = 10240;       // SIDE_MOST: the widest row these kernels take
__device__ __forceinline__ uint4 ld_now(const void * p) {                 // stays where it is written: ahead of the waits that follow
    uint4 v;
    asm volatile("ld.global.nc.v4.b32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
template <typename WT>
__global__ void __launch_bounds__(SIDE_THREADS) k_side_in(const SumArgs a, const SideW s, const int32_t * __restrict__ tokens, int n_vocab, int vec, float * __restrict__ Xs, float * __restrict__ G) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float ps[SIDE_THREADS / 32];
    constexpr int VEC = 16 / (int) sizeof(WT), GP = 4, WPR = SIDE_THREADS / 32 / SIDE_ROWS;      // chunks per lane asked for ahead; warps per row
    const int E = a.E, dim = s.dim, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, t = blockIdx.y;
    const int r = blockIdx.x * SIDE_ROWS + warp / WPR, first = (warp % WPR) * 32 + lane;
    const bool on = r < dim;
    const WT * w = reinterpret_cast<const WT *>(s.Wg) + (size_t) (on ? r : 0) * E;
    uint4 wg[GP];
    if (vec) {
#pragma unroll
        for (int j = 0; j < GP; j++) { const int k = (j * WPR * 32 + first) * VEC; wg[j] = on && k < E ? ld_now(w + k) : make_uint4(0u, 0u, 0u, 0u); }
    }
    int tok = tokens[t];
    tok = tok < 0 ? 0 : tok >= n_vocab ? n_vocab - 1 : tok;
    const float e = on ? wf(reinterpret_cast<const WT *>(s.table), (size_t) tok * s.ld + s.off + r) : 0.f;
    const auto sum = [&](int i, auto & v) {
        constexpr int N = sizeof(v) / sizeof(float);
        sum_chunk<N>(a, t, i, v);
        st_chunk<N>(xs + i, v);
        if (blockIdx.x == 0) st_chunk<N>(Xs + (size_t) t * E + i, v);
    };
    if ((E & 3) == 0) { for (int i = tid * 4; i < E; i += SIDE_THREADS * 4) { float v[4]; sum(i, v); } }
    else { for (int i = tid; i < E; i += SIDE_THREADS) { float v[1]; sum(i, v); } }
    __syncthreads();
    float acc = 0.f;
    if (vec) {
#pragma unroll
        for (int j = 0; j < GP; j++) { const int k = (j * WPR * 32 + first) * VEC; if (k < E) acc += dot16(wg[j], xs + k, w); }
        for (int k = (GP * WPR * 32 + first) * VEC; k < E; k += WPR * 32 * VEC) acc += dot16(ld_now(w + k), xs + k, w);
    } else {
        for (int k = first; k < E; k += WPR * 32) acc = fmaf(wf(w, k), xs[k], acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) ps[warp] = acc;
    __syncthreads();
    if (first == 0 && on) {                                // the row's warps in a fixed order
        acc = 0.f;
#pragma unroll
        for (int i = 0; i < WPR; i++) acc += ps[warp + i];
        G[(size_t) t * dim + r] = gelu_tanhf_(acc) * e;
    }
}
// Second: lpr lanes (a power of two) per row of W_p, SIDE_PER rows per group of lanes: Y[t] = W_p G[t]; the block of a token that finishes
// last (an atomic counter, no waiting) takes X[t] = Xs[t] + Y / rms(Y) wn and Hn[t] = X / rms(X) * nw, the row in registers in XV-entry
// chunks. grid (ceil(E / rows per block), T), dim floats of shared memory.
constexpr int SIDE_PER = 2;
inline int side_rows_per_block(int lpr) { return SIDE_THREADS / lpr * SIDE_PER; }
template <typename WT, int XV>
__global__ void __launch_bounds__(SIDE_THREADS) k_side_out(const SumArgs a, const SideW s, const float * __restrict__ Xs, const float * __restrict__ G, float * __restrict__ Y, int * __restrict__ counter, int vec, int lpr) {
    extern __shared__ __align__(16) float g[];
    __shared__ float red[32];
    __shared__ int last_s;
    constexpr int VEC = 16 / (int) sizeof(WT), OWN = SIDE_MOST / (SIDE_THREADS * XV);
    const int E = a.E, dim = s.dim, tid = threadIdx.x, t = blockIdx.y, sub = tid % lpr, grp = tid / lpr, ngrp = SIDE_THREADS / lpr, r0 = blockIdx.x * ngrp * SIDE_PER + grp;
    const WT * Wp = reinterpret_cast<const WT *>(s.Wp);
    uint4 wp[SIDE_PER];
    if (vec) {
#pragma unroll
        for (int j = 0; j < SIDE_PER; j++) { const int r = r0 + j * ngrp; wp[j] = r < E && sub * VEC < dim ? ld_now(Wp + (size_t) r * dim + sub * VEC) : make_uint4(0u, 0u, 0u, 0u); }
    }
    for (int i = tid; i < dim; i += SIDE_THREADS) g[i] = G[(size_t) t * dim + i];
    __syncthreads();
    const size_t row = (size_t) t * E;
#pragma unroll
    for (int j = 0; j < SIDE_PER; j++) {
        const int r = r0 + j * ngrp;
        float acc = 0.f;
        if (r < E) {
            const WT * w = Wp + (size_t) r * dim;
            if (vec) {
                if (sub * VEC < dim) acc = dot16(wp[j], g + sub * VEC, w);
                for (int k = (lpr + sub) * VEC; k < dim; k += lpr * VEC) acc += dot16(ld_now(w + k), g + k, w);
            } else {
                for (int k = sub; k < dim; k += lpr) acc = fmaf(wf(w, k), g[k], acc);
            }
        }
        for (int o = lpr >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (sub == 0 && r < E) Y[row + r] = acc;
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) last_s = atomicAdd(counter + t, 1) == (int) gridDim.x - 1;
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    if (tid == 0) counter[t] = 0;
    float y[OWN][XV], x[OWN][XV], w[OWN][XV], f[OWN][XV], ss = 0.f;
#pragma unroll
    for (int k = 0; k < OWN; k++) {
        const int i = (tid + k * SIDE_THREADS) * XV;
        if (i < E) {
            if constexpr (XV == 4) { const float4 v = __ldcg(reinterpret_cast<const float4 *>(Y + row + i)); y[k][0] = v.x; y[k][1] = v.y; y[k][2] = v.z; y[k][3] = v.w; }
            else y[k][0] = __ldcg(Y + row + i);
            ld_chunk<XV>(Xs + row + i, x[k]); ld_chunk<XV>(s.wn + i, w[k]); ld_chunk<XV>(a.nw + i, f[k]);
        }
    }
#pragma unroll
    for (int k = 0; k < OWN; k++) if ((tid + k * SIDE_THREADS) * XV < E) {
#pragma unroll
        for (int e = 0; e < XV; e++) ss = fmaf(y[k][e], y[k][e], ss);
    }
    ss = block_sum(ss, red);
    const float ry = 1.0f / sqrtf(ss / (float) E + a.eps);
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < OWN; k++) {
        const int i = (tid + k * SIDE_THREADS) * XV;
        if (i < E) {
#pragma unroll
            for (int e = 0; e < XV; e++) { x[k][e] = fmaf(y[k][e] * ry, w[k][e], x[k][e]); ss = fmaf(x[k][e], x[k][e], ss); }
            st_chunk<XV>(a.X + row + i, x[k]);
        }
    }
    ss = block_sum(ss, red);
    const float rx = 1.0f / sqrtf(ss / (float) E + a.eps);
#pragma unroll
    for (int k = 0; k < OWN; k++) {
        const int i = (tid + k * SIDE_THREADS) * XV;
        if (i < E) {
#pragma unroll
            for (int e = 0; e < XV; e++) x[k][e] = x[k][e] * rx * f[k][e];
            st_chunk<XV>(a.Hn + row + i, x[k]);
        }
    }
}

}  // namespace stk
}  // namespace b200
