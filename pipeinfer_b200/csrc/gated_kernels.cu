// gated_kernels.cu -- parts for layer-list models (hybrid.cuh) whose sublayers are gated on their way into the stream, all fp32:
//
//   the gated frame: what the sublayer before left (one output, or two outputs RMS-normed over the width and averaged), times the sigmoid
//       of its residual gate, joins the stream; the RMS norm of the new stream; in decode steps also the next input convolution
//   attention beside a matrix memory, per-token work: one RMS norm over all query rows and one over all key rows, rotation, cache write;
//       the memory's gates (running maximum, decays and write strengths) per segment and head
//   after both branches: head gates on the attention; the memory's normaliser, unit RMS per head, weight and sigmoid gates
#include "hybrid.cuh"

#define CKL() do { cudaError_t e__ = cudaGetLastError(); if (e__ != cudaSuccess) { pib_set_error("%s:%d: launch failed: %s", __FILE__, __LINE__, cudaGetErrorString(e__)); return PIB_ERR_CUDA; } } while (0)

__device__ __forceinline__ float gk_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
// two sums over the block at once; every thread gets both
__device__ __forceinline__ float2 gk_block_sum2(float a, float b, float2 * red) {
    a = warp_sum(a); b = warp_sum(b);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    __syncthreads();
    if (lane == 0) red[warp] = make_float2(a, b);
    __syncthreads();
    float2 t = make_float2(0.f, 0.f);
    for (int i = 0; i < nw; i++) { t.x += red[i].x; t.y += red[i].y; }
    return t;
}

// ---- the gated frame -------------------------------------------------------------------------------------------------------------------
// x[t] += y[t] sigmoid(gl[t] + gb), y = ya, or (wa given) mix (ya / rms(ya) wa + yb / rms(yb) wb); h[t] = x[t] / rms(x[t]) w.  With conv (batches of
// single tokens only: the block is the only reader of its slot's tail and moves it on itself) hc[t] = h[t] + sum_j conv[:, j] h(t - taps + 1 + j).
// One block per token; a thread owns NV pieces of VEC neighbouring channels, held in registers from the first load to the last store.
struct gf_args {
    float * x;
    pib_sublayer_out o;
    const float * w; float eps; int W;
    float * h;
    const float * conv; int taps;
    const int32_t * slot; float * state; size_t state_stride, tail_off;
    float * hc;
};
template <int VEC> struct gf_vec { float v[VEC]; };
template <int VEC> __device__ __forceinline__ gf_vec<VEC> gf_load(const float * p) {
    gf_vec<VEC> r;
    if (VEC == 4) { const float4 q = *reinterpret_cast<const float4 *>(p); r.v[0] = q.x; r.v[1 % VEC] = q.y; r.v[2 % VEC] = q.z; r.v[3 % VEC] = q.w; }
    else r.v[0] = *p;
    return r;
}
template <int VEC> __device__ __forceinline__ void gf_store(float * p, const gf_vec<VEC> & r) {
    if (VEC == 4) *reinterpret_cast<float4 *>(p) = make_float4(r.v[0], r.v[1 % VEC], r.v[2 % VEC], r.v[3 % VEC]);
    else *p = r.v[0];
}
template <int VEC, int NV>
__global__ void __launch_bounds__(NV >= 4 ? 512 : 1024) gated_norm_kernel(gf_args A) {
    pib_pdl_wait();
    pib_pdl_trigger();
    __shared__ float2 red[32];
    const int    t = blockIdx.x, W = A.W;
    const size_t row = (size_t) t * W;
    gf_vec<VEC> x[NV];
    float ss = 0.f;
    if (A.o.ya) {
        gf_vec<VEC> y[NV], yb[NV], g[NV];
        float sa = 0.f, sb = 0.f;
#pragma unroll
        for (int n = 0; n < NV; n++) {
            const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
            if (c < W) {
                x[n] = gf_load<VEC>(A.x + row + c);
                y[n] = gf_load<VEC>(A.o.ya + row + c);
                g[n] = gf_load<VEC>(A.o.gl + row + c);
                const gf_vec<VEC> b = gf_load<VEC>(A.o.gb + c);
                if (A.o.wa) yb[n] = gf_load<VEC>(A.o.yb + row + c);
#pragma unroll
                for (int i = 0; i < VEC; i++) {
                    g[n].v[i] = gk_sigmoid(g[n].v[i] + b.v[i]);
                    if (A.o.wa) { sa = fmaf(y[n].v[i], y[n].v[i], sa); sb = fmaf(yb[n].v[i], yb[n].v[i], sb); }
                }
            }
        }
        float ra = 1.f, rb = 0.f;
        if (A.o.wa) {
            const float2 s = gk_block_sum2(sa, sb, red);
            ra = A.o.mix / sqrtf(s.x / W + A.eps); rb = A.o.mix / sqrtf(s.y / W + A.eps);
        }
#pragma unroll
        for (int n = 0; n < NV; n++) {
            const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
            if (c < W) {
                if (A.o.wa) {
                    const gf_vec<VEC> wa = gf_load<VEC>(A.o.wa + c), wb = gf_load<VEC>(A.o.wb + c);
#pragma unroll
                    for (int i = 0; i < VEC; i++) y[n].v[i] = fmaf(y[n].v[i] * ra, wa.v[i], yb[n].v[i] * rb * wb.v[i]);
                }
#pragma unroll
                for (int i = 0; i < VEC; i++) { x[n].v[i] = fmaf(y[n].v[i], g[n].v[i], x[n].v[i]); ss = fmaf(x[n].v[i], x[n].v[i], ss); }
                gf_store<VEC>(A.x + row + c, x[n]);
            }
        }
    } else {
#pragma unroll
        for (int n = 0; n < NV; n++) {
            const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
            if (c < W) {
                x[n] = gf_load<VEC>(A.x + row + c);
#pragma unroll
                for (int i = 0; i < VEC; i++) ss = fmaf(x[n].v[i], x[n].v[i], ss);
            }
        }
    }
    if (!A.h) return;
    const float inv = 1.0f / sqrtf(gk_block_sum2(ss, 0.f, red).x / W + A.eps);
    float * tail = A.conv ? A.state + (size_t) A.slot[t] * A.state_stride + A.tail_off : nullptr;
#pragma unroll
    for (int n = 0; n < NV; n++) {
        const int c = (n * (int) blockDim.x + (int) threadIdx.x) * VEC;
        if (c < W) {
            const gf_vec<VEC> w = gf_load<VEC>(A.w + c);
#pragma unroll
            for (int i = 0; i < VEC; i++) x[n].v[i] = x[n].v[i] * inv * w.v[i];
            gf_store<VEC>(A.h + row + c, x[n]);
            if (A.conv) {
                gf_vec<VEC> acc = x[n];
                for (int j = 0; j < A.taps; j++) {
                    gf_vec<VEC> v = x[n];
                    if (j < A.taps - 1) {
#pragma unroll
                        for (int i = 0; i < VEC; i++) v.v[i] = tail[(size_t) j * W + c + i];
                    }
#pragma unroll
                    for (int i = 0; i < VEC; i++) {
                        acc.v[i] = fmaf(A.conv[(size_t) (c + i) * A.taps + j], v.v[i], acc.v[i]);
                        if (j > 0) tail[(size_t) (j - 1) * W + c + i] = v.v[i];      // row j - 1 was read in the trip before: every row moves up one place
                    }
                }
                gf_store<VEC>(A.hc + row + c, acc);
            }
        }
    }
}
// conv: null, or (only when every segment of the batch is one token) the input convolution of the sublayer that follows; h null: only the sum is done
int pib_gated_norm(float * x, const pib_sublayer_out & o, const float * w, float eps, int W, float * h, const float * conv, int taps, const pib_hbatch & b, float * state,
                   size_t state_stride, size_t tail_off, float * hc, cudaStream_t st) {
    if (conv && b.T != b.S) { pib_set_error("gated norm: the fused convolution takes batches of single tokens"); return PIB_ERR_ARG; }
    gf_args A = { x, o, w, eps, W, h, conv, taps, b.slot, state, state_stride, tail_off, hc };
    const int vec = W % 4 == 0 ? 4 : 1, pieces = (W + vec - 1) / vec, want = b.T > 32 ? 256 : 1024;      // decode steps: one piece per thread, as many loads in flight as there are
    int nv = 1;
    while (nv < 8 && (pieces + nv - 1) / nv > want) nv *= 2;
    const int threads = ((pieces + nv - 1) / nv + 31) & ~31;
    if (threads > (nv >= 4 ? 512 : 1024)) { pib_set_error("gated norm: width %d not supported", W); return PIB_ERR_UNSUPP; }
#define GF_GO(VEC, NV) pib_launch(gated_norm_kernel<VEC, NV>, dim3((unsigned) b.T), dim3((unsigned) threads), (size_t) 0, st, A)
    if (vec == 4) { if (nv == 1) GF_GO(4, 1); else if (nv == 2) GF_GO(4, 2); else if (nv == 4) GF_GO(4, 4); else GF_GO(4, 8); }
    else          { if (nv == 1) GF_GO(1, 1); else if (nv == 2) GF_GO(1, 2); else if (nv == 4) GF_GO(1, 4); else GF_GO(1, 8); }
#undef GF_GO
    CKL();
    return PIB_OK;
}

// ---- attention beside a matrix memory: what follows the projections -----------------------------------------------------------------------
// The last T blocks: one token each.  proj[t] = [q (nq = H*D) | k (nk = G*D) | v (nv = G*V) | ...]: q / rms(q) q_norm and k / rms(k) k_norm (one root mean
// square over ALL rows of q, one over all of k), then the first rot_dims coordinates of every D-wide row turn (pairs (i, i + rot_dims / 2)); q[t] gets
// the query rows, the token's cell [k | v].
// The blocks in front of them: the memory's gates of a few heads of one segment.  i = cap tanh((proj[i_off + h] + i_bias) / cap), f = log sigmoid(cap tanh((proj[f_off + h] +
// f_bias) / cap)); the running maximum m' = max(f + m, i) starts from the slot's and is left there.  It composes like a pair (F, M): m -> max(F + m, M),
// (F1, M1) then (F2, M2) = (F1 + F2, max(M1 + F2, M2)), so a warp takes 32 K tokens per trip: K in a row per lane, an inclusive scan over the lanes (and, with
// several warps per head, over the warps).
// dg[t] = [e^(i - m') (H2) | e^(f + m - m') (H2) | f + m - m' (H2) | e^-m' (H2)].  Every factor is formed from the maxima as stored, so their rounding cancels
// between the factors of neighbouring tokens.
struct amp_args {
    const float * proj; int ldp, gate_blocks, groups;
    int nq, nk, nv, D, rot_dims;
    const float * q_norm, * k_norm; float eps;
    const int32_t * pos, * cell; const float2 * rope;
    float * q, * cache; int cache_row;
    int H2, i_off, f_off; const float * i_bias, * f_bias; float cap;
    const int32_t * seg_start, * seg_len, * seg_slot;
    float * state; size_t state_stride, max_off;
    float * dg;
};
__device__ __forceinline__ float gk_capped(float z, float cap) { return cap > 0.f ? cap * tanhf(z / cap) : z; }
// one token: a warp per head row, VEC neighbouring coordinates per lane
template <int VEC>
__device__ __forceinline__ void amp_token(const amp_args & A, int t, float2 * red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5, D = A.D, half = A.rot_dims / 2, nqk = A.nq + A.nk;
    const float * p = A.proj + (size_t) t * A.ldp;
    float sq = 0.f, sk = 0.f;
    for (int e = threadIdx.x * VEC; e < nqk; e += blockDim.x * VEC) {
        const gf_vec<VEC> v = gf_load<VEC>(p + e);
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < VEC; i++) s = fmaf(v.v[i], v.v[i], s);
        if (e < A.nq) sq += s; else sk += s;
    }
    const float2 s = gk_block_sum2(sq, sk, red);
    const float rq = 1.0f / sqrtf(s.x / A.nq + A.eps), rk = 1.0f / sqrtf(s.y / A.nk + A.eps);
    const float2 * cs = A.rope + (size_t) A.pos[t] * half;
    float * row = A.cache + (size_t) A.cell[t] * A.cache_row;
    for (int e0 = warp * D; e0 < nqk; e0 += nw * D) {
        const bool    isq = e0 < A.nq;
        const float * w   = isq ? A.q_norm + e0 : A.k_norm + (e0 - A.nq), * src = p + e0;
        float *       dst = isq ? A.q + (size_t) t * A.nq + e0 : row + (e0 - A.nq);
        const float   r   = isq ? rq : rk;
        for (int i = lane * VEC; i < D; i += 32 * VEC) {
            gf_vec<VEC> v = gf_load<VEC>(src + i);
            const gf_vec<VEC> wv = gf_load<VEC>(w + i);
#pragma unroll
            for (int j = 0; j < VEC; j++) v.v[j] = v.v[j] * r * wv.v[j];
            if (i < A.rot_dims) {
                const bool first = i < half;
                const int  pi = first ? i + half : i - half, ci = first ? i : pi;
                const gf_vec<VEC> o = gf_load<VEC>(src + pi), wo = gf_load<VEC>(w + pi);
#pragma unroll
                for (int j = 0; j < VEC; j++) {
                    const float2 c = cs[ci + j];
                    const float  x = o.v[j] * r * wo.v[j];
                    v.v[j] = first ? v.v[j] * c.x - x * c.y : v.v[j] * c.x + x * c.y;
                }
            }
            gf_store<VEC>(dst + i, v);
        }
    }
    for (int e = threadIdx.x * VEC; e < A.nv; e += blockDim.x * VEC) gf_store<VEC>(row + A.nk + e, gf_load<VEC>(p + nqk + e));
}
// K == 1: batches of single tokens; K == 4: any batch
template <int K, int VEC>
__global__ void __launch_bounds__(K == 1 ? 1024 : 256, K == 1 ? 1 : 4) attn_mem_prep_kernel(amp_args A) {
    pib_pdl_wait();
    pib_pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if ((int) blockIdx.x >= A.gate_blocks) {
        __shared__ float2 red[32];
        amp_token<VEC>(A, blockIdx.x - A.gate_blocks, red);
        return;
    }
    // K == 1 (single tokens): a block takes 8 heads of one segment, a warp per head.  K == 4: a block takes two heads, four warps each on neighbouring runs of
    // 128 tokens; logits come in, and factors leave, through shared memory with neighbouring lanes on neighbouring heads
    static_assert(K == 1 || K == 4, "tokens per lane");
    constexpr int WPH = K == 1 ? 1 : 4, HPB = 8 / WPH, RUN = 32 * K, TT = WPH * RUN, PITCH = TT + TT / K + 1;      // token t sits at t + t / K: a lane's K tokens start K + 1 words behind its neighbour's
    __shared__ float buf[K == 1 ? 1 : 4 * HPB * PITCH];
    __shared__ float2 agg[8];
    if (warp >= 8) return;                                       // (only K == 1 has more threads, and no barrier below)
    const int sg = blockIdx.x / A.groups, h0 = (blockIdx.x % A.groups) * HPB, s0 = A.seg_start[sg], n = A.seg_len[sg], H = A.H2;
    const int hw = warp / WPH, part = warp % WPH, h = h0 + hw;   // this warp's head and its run of every tile
    if (K == 1 && h >= H) return;
    float * mslot = A.state + (size_t) A.seg_slot[sg] * A.state_stride + A.max_off + (h < H ? h : 0);
    float m0 = *mslot;
    const float ib = A.i_bias[h < H ? h : 0], fb = A.f_bias[h < H ? h : 0];
    const int hl = threadIdx.x % HPB, tl = threadIdx.x / HPB;    // staging: head, first token (steps of 256 / HPB tokens)
    constexpr int STEP = 256 / HPB, NS = K == 1 ? 1 : TT / STEP;
    float pi[NS], pf[NS];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int k = 0; k < NS; k++) {
            const int  t  = K == 1 ? t0 + lane : t0 + tl + STEP * k, hh = K == 1 ? h : h0 + hl;
            const bool ok = t < n && hh < H;
            const float * p = A.proj + (size_t) (s0 + t) * A.ldp + hh;
            pi[k] = ok ? p[A.i_off] : 0.f; pf[k] = ok ? p[A.f_off] : 0.f;
        }
    };
    fetch(0);
    for (int t0 = 0; t0 < n; t0 += TT) {
        float gi[K], gf[K];
        const int  base = part * RUN + lane * K;                 // this lane's first token of the tile
        const int  pos  = hw * PITCH + base + base / K;
        if (K > 1) {
            __syncthreads();                                     // the trip before has left the buffer
#pragma unroll
            for (int k = 0; k < NS; k++) {
                const int t = tl + STEP * k;
                buf[hl * PITCH + t + t / K] = pi[k]; buf[(HPB + hl) * PITCH + t + t / K] = pf[k];
            }
            __syncthreads();
        }
        float F = 0.f, M = -INFINITY;                            // tokens behind the end pass the maximum on unchanged
#pragma unroll
        for (int k = 0; k < K; k++) {
            const float zi = K == 1 ? pi[0] : buf[pos + k], zf = K == 1 ? pf[0] : buf[HPB * PITCH + pos + k];
            const float z = gk_capped(zf + fb, A.cap);
            gi[k] = gk_capped(zi + ib, A.cap);
            gf[k] = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
            if (t0 + base + k < n) { M = fmaxf(M + gf[k], gi[k]); F += gf[k]; }
        }
        if (t0 + TT < n) fetch(t0 + TT);                         // the next trip's logits are on their way while this one is scanned
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
            if (lane >= o) { M = fmaxf(Mp + F, M); F += Fp; }
        }
        float in = m0;                                           // the maximum in front of this warp's run
        if (K > 1) {
            if (lane == 31) agg[warp] = make_float2(F, M);
            __syncthreads();                                     // (and every warp has read its logits)
            float m = m0;
#pragma unroll
            for (int j = 0; j < WPH; j++) {
                if (j == part) in = m;
                const float2 r = agg[hw * WPH + j];
                m = fmaxf(r.x + m, r.y);
            }
            m0 = m;
        }
        const float last = fmaxf(F + in, M);
        float m = __shfl_up_sync(0xffffffffu, last, 1);          // the maximum in front of this lane's tokens
        if (lane == 0) m = in;
        if (K == 1) m0 = __shfl_sync(0xffffffffu, last, 31);
#pragma unroll
        for (int k = 0; k < K; k++) {
            // the lane's last token takes the scan's number, so that the next lane's first factor starts from the same one
            const float mn = k == K - 1 ? last : fmaxf(gf[k] + m, gi[k]), ld = (gf[k] + m) - mn, f0 = expf(gi[k] - mn), f1 = expf(ld), f3 = expf(-mn);
            if (K == 1) {
                if (t0 + base < n) { float * d = A.dg + (size_t) (s0 + t0 + base) * 4 * H + h; d[0] = f0; d[H] = f1; d[2 * H] = ld; d[3 * H] = f3; }
            } else {
                float * o = buf + pos + k;
                o[0] = f0; o[HPB * PITCH] = f1; o[2 * HPB * PITCH] = ld; o[3 * HPB * PITCH] = f3;
            }
            m = mn;
        }
        if (K > 1) {
            __syncthreads();
#pragma unroll
            for (int k = 0; k < NS; k++) {
                const int t = tl + STEP * k;
                if (t0 + t < n && h0 + hl < H) {
                    float * d = A.dg + (size_t) (s0 + t0 + t) * 4 * H + h0 + hl;
#pragma unroll
                    for (int j = 0; j < 4; j++) d[j * H] = buf[(HPB * j + hl) * PITCH + t + t / K];
                }
            }
        }
    }
    if (lane == 0 && part == 0 && h < H) *mslot = m0;
}
int pib_attn_mem_prep(const float * proj, int ldp, int i_off, int f_off, const pib_hlayer & L, float eps, const pib_hbatch & b, const float2 * rope, float * q, float * cache,
                      int cache_row, float * state, size_t state_stride, float * dg, cudaStream_t st) {
    const int nq = L.heads * L.dim, nk = L.kv_heads * L.dim, nv = L.kv_heads * L.vdim, n_all = nq + nk + nv, hpb = b.T == b.S ? 8 : 2, groups = (L.heads2 + hpb - 1) / hpb;
    amp_args A = { proj, ldp, b.S * groups, groups, nq, nk, nv, L.dim, L.rot_dims, L.q_norm, L.k_norm, eps, b.pos, b.cell, rope, q, cache, cache_row, L.heads2, i_off, f_off, L.i_bias, L.f_bias,
                   L.gate_cap, b.seg_start, b.seg_len, b.seg_slot, state, state_stride, L.max_off, dg };
    auto al = [](const void * p) { return ((uintptr_t) p & 15) == 0; };
    const bool vec = L.dim % 4 == 0 && (L.rot_dims / 2) % 4 == 0 && nv % 4 == 0 && ldp % 4 == 0 && cache_row % 4 == 0 && al(proj) && al(q) && al(cache);
    if (b.T == b.S) {
        const dim3 grid((unsigned) (b.T + b.S * groups)), threads(b.T > 32 ? 256u : n_all >= 2048 ? 1024u : n_all >= 1024 ? 512u : 256u);
        if (vec) pib_launch(attn_mem_prep_kernel<1, 4>, grid, threads, (size_t) 0, st, A);
        else     pib_launch(attn_mem_prep_kernel<1, 1>, grid, threads, (size_t) 0, st, A);
    } else {
        const dim3 grid((unsigned) (b.T + b.S * groups));
        if (vec) pib_launch(attn_mem_prep_kernel<4, 4>, grid, dim3(256), (size_t) 0, st, A);
        else     pib_launch(attn_mem_prep_kernel<4, 1>, grid, dim3(256), (size_t) 0, st, A);
    }
    CKL();
    return PIB_OK;
}

// out[t] = [ a[t][h][:] sigmoid(proj[t][hg_off + h]) (H*V) | gap | per head of the memory: u / rms(u) w sigmoid(proj[t][og_off + :]) (H2*V2) at mem_off ],
// u = s S^T q / (max(|s n . q|, e^-m) + 1e-6), s = dim^(-1/2); mem[t][h] = [S^T q | n . q].  One block per token, a warp per memory head.
__global__ void __launch_bounds__(1024) attn_mem_gate_kernel(const float * __restrict__ a, const float * __restrict__ mem, const float * __restrict__ dg, const float * __restrict__ proj, int ldp,
                                                             int hg_off, int og_off, int H, int V, int H2, int V2, float s, const float * __restrict__ w, float eps,
                                                             float * __restrict__ out, int ldo, int mem_off) {
    pib_pdl_wait();
    pib_pdl_trigger();
    const size_t  t = blockIdx.x;
    const int     lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const float * p = proj + t * ldp;
    float *       o = out + t * ldo;
    for (int h = warp; h < H2; h += nw) {
        const float * r = mem + (t * H2 + h) * (V2 + 1);
        const float   c = s / (fmaxf(fabsf(s * r[V2]), dg[t * 4 * H2 + 3 * H2 + h]) + 1e-6f);
        float ss = 0.f;
        for (int i = lane; i < V2; i += 32) { const float u = r[i] * c; ss = fmaf(u, u, ss); }
        const float inv = c / sqrtf(warp_sum(ss) / V2 + eps);
        for (int i = lane; i < V2; i += 32) o[mem_off + h * V2 + i] = r[i] * inv * w[h * V2 + i] * gk_sigmoid(p[og_off + h * V2 + i]);
    }
    for (int h = warp; h < H; h += nw) {
        const float g = gk_sigmoid(p[hg_off + h]);
        for (int i = lane; i < V; i += 32) o[h * V + i] = a[(t * H + h) * V + i] * g;
    }
}
int pib_attn_mem_gate(const float * a, const float * mem, const float * dg, const float * proj, int ldp, int hg_off, int og_off, const pib_hlayer & L, float eps, int T, float * out,
                      int ldo, int mem_off, cudaStream_t st) {
    const int most = L.heads > L.heads2 ? L.heads : L.heads2, threads = T > 32 || most <= 8 ? 256 : most <= 16 ? 512 : 1024;      // decode steps: a warp for every head
    pib_launch(attn_mem_gate_kernel, dim3((unsigned) T), dim3(threads), (size_t) 0, st, a, mem, dg, proj, ldp, hg_off, og_off, L.heads, L.vdim, L.heads2, L.vdim2,
               (float) (1.0 / sqrt((double) L.dim2)), (const float *) L.onorm, eps, out, ldo, mem_off);
    CKL();
    return PIB_OK;
}
