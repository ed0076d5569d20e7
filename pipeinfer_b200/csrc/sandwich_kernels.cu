// sandwich_kernels.cu -- the sandwich frame of layer-list models (hybrid.cuh), all fp32: a LayerNorm in front of and one behind every sublayer.
//
//   x[t] += LN'(y[t]), y what the sublayer before left: its output rows, or a shared expert's rows plus the routed experts' weighted rows (the
//           mixture is summed here, it never exists in memory), LN' the norm behind it with layer scale and residual multiplier in its weight and bias
//   h[t]  = LN(x[t]), the norm in front of the sublayer that follows (or the model's last one)
//   small batches in front of a mixture: the router's logits of h[t] and the token's choice on the same launch; the last block to finish sorts the pairs
#include "hybrid.cuh"
#include "moe_route.cuh"

#include <algorithm>

#define CKL() do { cudaError_t e__ = cudaGetLastError(); if (e__ != cudaSuccess) { pib_set_error("%s:%d: launch failed: %s", __FILE__, __LINE__, cudaGetErrorString(e__)); return PIB_ERR_CUDA; } } while (0)

template <int VEC> struct sw_vec { float v[VEC]; };
template <int VEC> __device__ __forceinline__ sw_vec<VEC> sw_load(const float * p) {
    sw_vec<VEC> r;
    if (VEC == 4) { const float4 q = *reinterpret_cast<const float4 *>(p); r.v[0] = q.x; r.v[1 % VEC] = q.y; r.v[2 % VEC] = q.z; r.v[3 % VEC] = q.w; }
    else r.v[0] = *p;
    return r;
}
template <int VEC> __device__ __forceinline__ void sw_store(float * p, const sw_vec<VEC> & r) {
    if (VEC == 4) *reinterpret_cast<float4 *>(p) = make_float4(r.v[0], r.v[1 % VEC], r.v[2 % VEC], r.v[3 % VEC]);
    else *p = r.v[0];
}
__device__ __forceinline__ float sw_block_sum(float v, float * red) {
    v = warp_sum(v);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < nw; i++) t += red[i];
    return t;
}

struct sw_args {
    float * x;
    pib_sublayer_y o;
    const float * w, * b; float eps; int W;
    float * h;
    pib_norm_route route;
};
// mean and 1 / sqrt(variance + eps) of the block's row, held in registers as NV pieces of VEC channels per thread
template <int VEC, int NV> __device__ __forceinline__ float2 sw_moments(const sw_vec<VEC> (&r)[NV], int W, float eps, float * red) {
    float s = 0.f, q = 0.f;
#pragma unroll
    for (int n = 0; n < NV; n++) {
        const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
        if (c < W) {
#pragma unroll
            for (int i = 0; i < VEC; i++) s += r[n].v[i];
        }
    }
    const float mean = sw_block_sum(s, red) / W;
#pragma unroll
    for (int n = 0; n < NV; n++) {
        const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
        if (c < W) {
#pragma unroll
            for (int i = 0; i < VEC; i++) { const float d = r[n].v[i] - mean; q = fmaf(d, d, q); }
        }
    }
    return make_float2(mean, 1.0f / sqrtf(sw_block_sum(q, red) / W + eps));
}

// the router's logits of the row in shared memory (a warp per output in turn), the token's choice (one warp), and -- in the block that finishes last --
// the grouping of all pairs.  Shared memory: row (W) | logits (E) | scratch of the choice (E + groups) | pairs | counts (E)
__device__ __forceinline__ void sw_route(const sw_args & A, int t, float * row) {
    const pib_router & R = A.route.R;
    const int W = A.W, E = R.E, T = gridDim.x, P = T * R.top, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    float * logits = row + W, * cv = logits + E;
    int32_t * sid = reinterpret_cast<int32_t *>(cv + E + R.groups), * cnt = sid + P;
    __shared__ int last;
    __syncthreads();
    for (int n = warp; n < E; n += nw) {
        const float * w = A.route.rows + (size_t) n * W;
        float s = 0.f;
#pragma unroll 8
        for (int k = lane * 4; k < W; k += 128) {
            const float4 a = *reinterpret_cast<const float4 *>(row + k), b = *reinterpret_cast<const float4 *>(w + k);
            s = fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, s))));
        }
        s = warp_sum(s);
        if (lane == 0) logits[n] = s;
    }
    __syncthreads();
    if (warp == 0) {
        moe_route_token(logits, R, cv, lane, A.route.ids + (size_t) t * R.top, A.route.wts + (size_t) t * R.top);
        if (lane == 0) {
            __threadfence();
            last = atomicAdd(A.route.done, 1) == T - 1;
        }
    }
    __syncthreads();
    if (!last) return;
    __threadfence();
    for (int i = threadIdx.x; i < P; i += blockDim.x) sid[i] = __ldcg(A.route.ids + i);
    if (threadIdx.x == 0) *A.route.done = 0;
    __syncthreads();
    moe_sort_small(sid, P, E, R.n_real, cnt, A.route.offs, A.route.perm, A.route.inv, A.route.act);
}
// one block per token; every row crosses memory once
template <int VEC, int NV, bool ROUTE>
__global__ void __launch_bounds__(NV >= 4 ? 512 : 1024) sandwich_norm_kernel(sw_args A) {
    pib_pdl_wait();
    pib_pdl_trigger();
    __shared__ float red[32];
    extern __shared__ __align__(16) float sw_dyn[];
    const int    t = blockIdx.x, W = A.W;
    const size_t row = (size_t) t * W;
    const bool   any = A.o.y || A.o.top > 0;
    sw_vec<VEC> x[NV];
#pragma unroll
    for (int n = 0; n < NV; n++) {
        const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
        if (c < W) x[n] = sw_load<VEC>(A.x + row + c);
    }
    if (any) {
        sw_vec<VEC> y[NV];
#pragma unroll
        for (int n = 0; n < NV; n++) {
            const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
#pragma unroll
            for (int i = 0; i < VEC; i++) y[n].v[i] = 0.f;
            if (c < W && A.o.y) y[n] = sw_load<VEC>(A.o.y + row + c);
        }
        for (int k = 0; k < A.o.top; k++) {              // k in ascending order
            const size_t  pair = (size_t) t * A.o.top + k;
            const float   wk   = A.o.wts[pair];
            const float * src  = A.o.ids[pair] < A.o.n_real ? A.o.edn + (size_t) A.o.inv[pair] * W : A.o.hin + row;
#pragma unroll
            for (int n = 0; n < NV; n++) {
                const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
                if (c < W) {
                    const sw_vec<VEC> v = sw_load<VEC>(src + c);
#pragma unroll
                    for (int i = 0; i < VEC; i++) y[n].v[i] = fmaf(wk, v.v[i], y[n].v[i]);
                }
            }
        }
        const float2 my = sw_moments<VEC, NV>(y, W, A.eps, red);
#pragma unroll
        for (int n = 0; n < NV; n++) {
            const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
            if (c < W) {
                const sw_vec<VEC> w = sw_load<VEC>(A.o.w + c), b = sw_load<VEC>(A.o.b + c);
#pragma unroll
                for (int i = 0; i < VEC; i++) x[n].v[i] += fmaf((y[n].v[i] - my.x) * my.y, w.v[i], b.v[i]);
                sw_store<VEC>(A.x + row + c, x[n]);
            }
        }
    }
    if (!A.h) return;
    const float2 mx = sw_moments<VEC, NV>(x, W, A.eps, red);
#pragma unroll
    for (int n = 0; n < NV; n++) {
        const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
        if (c < W) {
            const sw_vec<VEC> w = sw_load<VEC>(A.w + c), b = sw_load<VEC>(A.b + c);
            sw_vec<VEC> h;
#pragma unroll
            for (int i = 0; i < VEC; i++) h.v[i] = fmaf((x[n].v[i] - mx.x) * mx.y, w.v[i], b.v[i]);
            sw_store<VEC>(A.h + row + c, h);             // a thread wrote and read only its own channels of this token: hin may be h
            if (ROUTE) sw_store<VEC>(sw_dyn + c, h);
        }
    }
    if (ROUTE) sw_route(A, t, sw_dyn);
}
static size_t sw_route_smem(int T, int W, const pib_router & R) { return (size_t) (W + 3 * R.E + R.groups + T * R.top) * 4; }
bool pib_norm_route_fits(int T, int W, const pib_router & R) {
    return W % 4 == 0 && T <= MOE_SMALL_T && T * R.top <= MOE_SMALL_PAIRS && R.E <= MOE_SMALL_E && sw_route_smem(T, W, R) <= 46 * 1024;
}
// o empty: only the norm of x; h null: only the sum; route: see pib_norm_route (the caller has asked pib_norm_route_fits)
int pib_sandwich_norm(float * x, const pib_sublayer_y & o, const float * w, const float * b, float eps, int T, int W, float * h, cudaStream_t st, const pib_norm_route * route) {
    sw_args A = { x, o, w, b, eps, W, h, pib_norm_route() };
    if (route) {
        const int rc = pib_moe_router_check(route->R);
        if (rc != PIB_OK) return rc;
        if (!h || !pib_norm_route_fits(T, W, route->R)) { pib_set_error("sandwich norm: no routing for %d tokens of width %d", T, W); return PIB_ERR_ARG; }
        A.route = *route;
    }
    const int vec = W % 4 == 0 ? 4 : 1, pieces = (W + vec - 1) / vec, want = T > 32 ? 256 : 1024;      // decode steps: one piece per thread, as many loads in flight as there are
    int nv = 1;
    while (nv < 8 && (pieces + nv - 1) / nv > want) nv *= 2;
    int threads = ((pieces + nv - 1) / nv + 31) & ~31;
    if (threads > (nv >= 4 ? 512 : 1024)) { pib_set_error("sandwich norm: width %d not supported", W); return PIB_ERR_UNSUPP; }
    if (route) threads = std::max(threads, 512);                       // 16 warps over the router's rows
#define SW_GO(VEC, NV) pib_launch(sandwich_norm_kernel<VEC, NV, false>, dim3((unsigned) T), dim3((unsigned) threads), (size_t) 0, st, A)
#define SW_GO_ROUTE(NV) pib_launch(sandwich_norm_kernel<4, NV, true>, dim3((unsigned) T), dim3((unsigned) threads), sw_route_smem(T, W, route->R), st, A)
    if (route)         { if (nv == 1) SW_GO_ROUTE(1); else if (nv == 2) SW_GO_ROUTE(2); else if (nv == 4) SW_GO_ROUTE(4); else SW_GO_ROUTE(8); }
    else if (vec == 4) { if (nv == 1) SW_GO(4, 1); else if (nv == 2) SW_GO(4, 2); else if (nv == 4) SW_GO(4, 4); else SW_GO(4, 8); }
    else               { if (nv == 1) SW_GO(1, 1); else if (nv == 2) SW_GO(1, 2); else if (nv == 4) SW_GO(1, 4); else SW_GO(1, 8); }
#undef SW_GO
#undef SW_GO_ROUTE
    CKL();
    return PIB_OK;
}
