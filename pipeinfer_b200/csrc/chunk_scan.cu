// chunk_scan.cu -- linear recurrences with one decay per head and token as matmuls on the tensor cores (layer-list models, hybrid.cuh).
//
//   S_t = c_t S_(t-1) + w_t k_t v_t^T,   o_t = S_t^T q_t          (S [D][V] per head; with `ones` a last column whose value is always 1)
//
// A portion of n tokens is cut into chunks of CS_C.  With l_t the running sum of log c inside a chunk (l_C its last), S the matrix in front
// of the chunk and s over the chunk's tokens up to and with t:
//     o_t = sum_s e^(l_t - l_s) w_s (q_t . k_s) v_s + e^(l_t) S^T q_t,      S' = e^(l_C) S + sum_s e^(l_C - l_s) w_s k_s v_s^T
// so per (chunk, head) there are three matmuls -- scores q k^T; outputs [weighted scores | e^(l_t) q_t] x [v ; S]; the chunk's own addition
// to S -- and the only thing that walks along the sequence is S' over the chunks, one multiply-add per matrix element and chunk.
//
// Everything keeps (nearly) fp32 accuracy on bfloat16 tensor cores: a number enters as its bfloat16 part and the remainder of that rounding,
// one operand's rows as [hi | lo | hi], the other's as [hi | hi | lo] (three times as wide: hi.hi + lo.hi + hi.lo, fp32 accumulation).
// Decays, running sums, the weighting of the scores, the matrices between chunks and the whole `ones` column (its chunk's addition a weighted
// sum of keys, its output a sum over the weighted scores plus e^(l_t) n . q_t) are fp32.
#include "hybrid.cuh"

#include <algorithm>

#include <cuda_bf16.h>

#define CKL() do { cudaError_t e__ = cudaGetLastError(); if (e__ != cudaSuccess) { pib_set_error("%s:%d: launch failed: %s", __FILE__, __LINE__, cudaGetErrorString(e__)); return PIB_ERR_CUDA; } } while (0)

#define CS_C 128
typedef __nv_bfloat16 bf16;

struct cs_dev {
    pib_chunk_scan a;
    int NC, V1;                       // chunks; value columns with the one of ones
    bf16 * Qx, * Kw;                  // [z][CS_C][3 D]: queries hi | lo | hi, keys hi | hi | lo                 (z = chunk * H + head)
    bf16 * Kt;                        // [z][D][3 CS_C]: keys transposed, hi | hi | lo
    bf16 * Ux;                        // [z][V][3 CS_C]: e^(l_C - l_s) w_s v_s transposed, hi | lo | hi
    bf16 * Vw;                        // [z][V][3 CS_C + 3 D]: values transposed hi | hi | lo, then S transposed hi | hi | lo
    bf16 * Px;                        // [z][CS_C][3 CS_C + 3 D]: weighted scores hi | lo | hi, then e^(l_t) q_t hi | lo | hi
    float * Sc;                       // [z][CS_C][CS_C] scores
    float * Lo;                       // [z][V][D] what a chunk adds to S (transposed)
    float * Yo;                       // [z][CS_C][V] outputs
    float * lsum, * wts;              // [z][CS_C] running sums of log decays, write weights (0 behind the portion's end)
    float * nadd, * npv;              // [z][D] ones column: what a chunk adds to it; in front of the chunk
};
__device__ __forceinline__ void cs_split(float x, bf16 & hi, bf16 & lo) { hi = __float2bfloat16_rn(x); lo = __float2bfloat16_rn(x - __bfloat162float(hi)); }

// grid (z, 2, 32 columns): y = 0 queries and keys, y = 1 values, which go through shared memory to come out transposed.
__global__ void __launch_bounds__(256) cs_operands_kernel(cs_dev d) {
    pib_pdl_wait();
    pib_pdl_trigger();
    __shared__ float tile[32][CS_C + 1];
    __shared__ float ls[CS_C], us[CS_C], wsum[4];        // us: e^(l_C - l_s) w_s
    const pib_chunk_scan & a = d.a;
    const int z = blockIdx.x, c = z / a.H, h = z % a.H, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, D = a.D, V = a.V;
    const int c0 = blockIdx.z * 32, i = c0 + lane, first = c * CS_C, nt = min(CS_C, a.n - first);
    const size_t row0 = (size_t) (a.t0 + first);
    // running sums of the log decays: a warp's scan over 32 tokens, then the sums of the warps in front
    float l = 0.f, w = 0.f;
    if (threadIdx.x < CS_C) {
        const int t = threadIdx.x;
        const bool ok = t < nt;
        l = ok ? a.log_decay[(row0 + t) * a.ldg + h] : 0.f;
        w = ok ? a.weight[(row0 + t) * a.ldg + h] : 0.f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const float p = __shfl_up_sync(0xffffffffu, l, o); if (lane >= o) l += p; }
        if (lane == 31) wsum[warp] = l;
    }
    __syncthreads();
    if (threadIdx.x < CS_C) {
        for (int i = 0; i < warp; i++) l += wsum[i];
        ls[threadIdx.x] = l;
        if (blockIdx.y == 0 && blockIdx.z == 0) { d.lsum[(size_t) z * CS_C + threadIdx.x] = l; d.wts[(size_t) z * CS_C + threadIdx.x] = w; }
    }
    __syncthreads();
    if (threadIdx.x < CS_C) us[threadIdx.x] = expf(ls[CS_C - 1] - l) * w;
    __syncthreads();
    if (blockIdx.y == 0) {
        const int g = h / (a.H / a.G);
        const float * q = a.q + row0 * a.ldq + (size_t) g * D, * k = a.k + row0 * a.ldk + (size_t) g * D;
        bf16 * Qx = d.Qx + (size_t) z * CS_C * 3 * D, * Kw = d.Kw + (size_t) z * CS_C * 3 * D, * Kt = d.Kt + (size_t) z * D * 3 * CS_C;
        if (c0 >= D) return;
        float qv[CS_C / 8], kv[CS_C / 8];
#pragma unroll
        for (int r = 0; r < CS_C / 8; r++) {                  // all of a warp's rows in flight at once
            const int  t  = warp + 8 * r;
            const bool ok = i < D && t < nt;
            qv[r] = ok ? q[(size_t) t * a.ldq + i] : 0.f; kv[r] = ok ? k[(size_t) t * a.ldk + i] : 0.f;
        }
#pragma unroll
        for (int r = 0; r < CS_C / 8; r++) {
            const int t = warp + 8 * r;
            if (i < D) {
                bf16 hi, lo;
                cs_split(qv[r], hi, lo);
                bf16 * p = Qx + (size_t) t * 3 * D + i;
                p[0] = hi; p[D] = lo; p[2 * D] = hi;
                cs_split(kv[r], hi, lo);
                p = Kw + (size_t) t * 3 * D + i;
                p[0] = hi; p[D] = hi; p[2 * D] = lo;
            }
            tile[lane][t] = kv[r];
        }
        __syncthreads();
        for (int r = warp; r < 32 && c0 + r < D; r += 8) {
            float add = 0.f;
            bf16 * p = Kt + (size_t) (c0 + r) * 3 * CS_C;
#pragma unroll
            for (int j = 0; j < CS_C; j += 64) {
                const int t = j + 2 * lane;
                bf16 h0, l0, h1, l1;
                cs_split(tile[r][t], h0, l0); cs_split(tile[r][t + 1], h1, l1);
                const __nv_bfloat162 hh = __halves2bfloat162(h0, h1);
                *reinterpret_cast<__nv_bfloat162 *>(p + t) = hh; *reinterpret_cast<__nv_bfloat162 *>(p + CS_C + t) = hh;
                *reinterpret_cast<__nv_bfloat162 *>(p + 2 * CS_C + t) = __halves2bfloat162(l0, l1);
                add = fmaf(tile[r][t], us[t], fmaf(tile[r][t + 1], us[t + 1], add));
            }
            add = warp_sum(add);
            if (lane == 0) d.nadd[(size_t) z * D + c0 + r] = add;
        }
        return;
    }
    if (c0 >= V) return;
    const float * v = a.v + row0 * a.ldv + (size_t) h * V;
    const int KX = 3 * CS_C + 3 * D;
    bf16 * Ux = d.Ux + (size_t) z * V * 3 * CS_C, * Vw = d.Vw + (size_t) z * V * KX;
#pragma unroll
    for (int r = 0; r < CS_C / 8; r++) { const int t = warp + 8 * r; tile[lane][t] = i < V && t < nt ? v[(size_t) t * a.ldv + i] : 0.f; }
    __syncthreads();
    for (int r = warp; r < 32 && c0 + r < V; r += 8) {
        bf16 * u = Ux + (size_t) (c0 + r) * 3 * CS_C, * p = Vw + (size_t) (c0 + r) * KX;
#pragma unroll
        for (int j = 0; j < CS_C; j += 64) {
            const int t = j + 2 * lane;
            const float x0 = tile[r][t], x1 = tile[r][t + 1];
            bf16 h0, l0, h1, l1;
            cs_split(x0 * us[t], h0, l0); cs_split(x1 * us[t + 1], h1, l1);
            *reinterpret_cast<__nv_bfloat162 *>(u + t) = __halves2bfloat162(h0, h1); *reinterpret_cast<__nv_bfloat162 *>(u + CS_C + t) = __halves2bfloat162(l0, l1);
            *reinterpret_cast<__nv_bfloat162 *>(u + 2 * CS_C + t) = __halves2bfloat162(h0, h1);
            cs_split(x0, h0, l0); cs_split(x1, h1, l1);
            *reinterpret_cast<__nv_bfloat162 *>(p + t) = __halves2bfloat162(h0, h1); *reinterpret_cast<__nv_bfloat162 *>(p + CS_C + t) = __halves2bfloat162(h0, h1);
            *reinterpret_cast<__nv_bfloat162 *>(p + 2 * CS_C + t) = __halves2bfloat162(l0, l1);
        }
    }
}

// one thread per element (head, value column, row) of the matrices: the matrix in front of every chunk, and the slot's new one
__global__ void __launch_bounds__(256) cs_carry_kernel(cs_dev d) {
    pib_pdl_wait();
    pib_pdl_trigger();
    const pib_chunk_scan & a = d.a;
    const int D = a.D, V = a.V, V1 = d.V1, e = blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= a.H * V1 * D) return;
    const int i = e % D, v = (e / D) % V1, h = e / (D * V1), KX = 3 * CS_C + 3 * D;
    float * slot = a.state + (size_t) h * D * V1 + (size_t) i * V1 + v;
    float s = *slot;
    for (int c0 = 0; c0 < d.NC; c0 += 4) {
        float add[4], dec[4];
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const size_t z = (size_t) min(c0 + j, d.NC - 1) * a.H + h;
            add[j] = v < V ? d.Lo[(z * V + v) * D + i] : d.nadd[z * D + i];
            dec[j] = expf(d.lsum[z * CS_C + CS_C - 1]);
        }
#pragma unroll
        for (int j = 0; j < 4; j++) {
            if (c0 + j >= d.NC) break;
            const size_t z = (size_t) (c0 + j) * a.H + h;
            if (v < V) {
                bf16 hi, lo;
                cs_split(s, hi, lo);
                bf16 * p = d.Vw + (z * V + v) * KX + 3 * CS_C + i;
                p[0] = hi; p[D] = hi; p[2 * D] = lo;
            } else d.npv[z * D + i] = s;
            s = fmaf(dec[j], s, add[j]);
        }
    }
    *slot = s;
}

// grid (z, CS_C / 8), a warp per token: weights on the scores, the query for the matrix in front of the chunk, the ones column's output
__global__ void __launch_bounds__(256) cs_weight_kernel(cs_dev d) {
    pib_pdl_wait();
    pib_pdl_trigger();
    const pib_chunk_scan & a = d.a;
    const int z = blockIdx.x, c = z / a.H, h = z % a.H, lane = threadIdx.x & 31, t = blockIdx.y * 8 + (threadIdx.x >> 5), D = a.D, KX = 3 * CS_C + 3 * D;
    const bool live = c * CS_C + t < a.n;
    const float * ls = d.lsum + (size_t) z * CS_C, * ws = d.wts + (size_t) z * CS_C, * sc = d.Sc + ((size_t) z * CS_C + t) * CS_C;
    bf16 * p = d.Px + ((size_t) z * CS_C + t) * KX;
    const float lt = ls[t];
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < CS_C; j += 64) {
        const int s = j + 2 * lane;
        const float2 x = *reinterpret_cast<const float2 *>(sc + s), l2 = *reinterpret_cast<const float2 *>(ls + s), w2 = *reinterpret_cast<const float2 *>(ws + s);
        const float p0 = live && s <= t ? x.x * (expf(lt - l2.x) * w2.x) : 0.f, p1 = live && s + 1 <= t ? x.y * (expf(lt - l2.y) * w2.y) : 0.f;
        sum += p0 + p1;
        bf16 h0, l0, h1, l1;
        cs_split(p0, h0, l0); cs_split(p1, h1, l1);
        *reinterpret_cast<__nv_bfloat162 *>(p + s) = __halves2bfloat162(h0, h1); *reinterpret_cast<__nv_bfloat162 *>(p + CS_C + s) = __halves2bfloat162(l0, l1);
        *reinterpret_cast<__nv_bfloat162 *>(p + 2 * CS_C + s) = __halves2bfloat162(h0, h1);
    }
    const float et = expf(lt);
    const float * q = a.q + (size_t) (a.t0 + c * CS_C + (live ? t : 0)) * a.ldq + (size_t) (h / (a.H / a.G)) * D, * n = d.npv + (size_t) z * D;
    for (int i = lane; i < D; i += 32) {
        const float x = live ? et * q[i] : 0.f;
        if (a.ones) sum = fmaf(x, n[i], sum);
        bf16 hi, lo;
        cs_split(x, hi, lo);
        bf16 * r = p + 3 * CS_C + i;
        r[0] = hi; r[D] = lo; r[2 * D] = hi;
    }
    if (a.ones) {
        sum = warp_sum(sum);
        if (lane == 0 && live) a.out[((size_t) (a.t0 + c * CS_C + t) * a.H + h) * d.V1 + a.V] = sum;
    }
}

// the outputs back in token order, grid (token)
__global__ void __launch_bounds__(256) cs_order_kernel(cs_dev d) {
    pib_pdl_wait();
    pib_pdl_trigger();
    const pib_chunk_scan & a = d.a;
    const int tok = blockIdx.x, c = tok / CS_C, t = tok % CS_C, V = a.V;
    float * out = a.out + (size_t) (a.t0 + tok) * a.H * d.V1;
    for (int e = threadIdx.x; e < a.H * V; e += blockDim.x) {
        const int h = e / V, v = e % V;
        out[(size_t) h * d.V1 + v] = d.Yo[(((size_t) c * a.H + h) * CS_C + t) * V + v];
    }
}

// sizes of the work buffers: the same walk as pib_chunk_scan_run's
static size_t cs_layout(cs_dev & d, char * base) {
    const pib_chunk_scan & a = d.a;
    const size_t Z = (size_t) d.NC * a.H, D = (size_t) a.D, V = (size_t) a.V, C = CS_C, KX = 3 * C + 3 * D;
    size_t off = 0;
    auto take = [&](size_t bytes) { char * p = base + off; off = (off + bytes + 255) & ~(size_t) 255; return p; };
    d.Qx = (bf16 *) take(Z * C * 3 * D * 2); d.Kw = (bf16 *) take(Z * C * 3 * D * 2); d.Kt = (bf16 *) take(Z * D * 3 * C * 2); d.Ux = (bf16 *) take(Z * V * 3 * C * 2);
    d.Vw = (bf16 *) take(Z * V * KX * 2); d.Px = (bf16 *) take(Z * C * KX * 2); d.Sc = (float *) take(Z * C * C * 4); d.Lo = (float *) take(Z * V * D * 4);
    d.Yo = (float *) take(Z * C * V * 4); d.lsum = (float *) take(Z * C * 4); d.wts = (float *) take(Z * C * 4); d.npv = (float *) take(Z * D * 4); d.nadd = (float *) take(Z * D * 4);
    return off;
}
// head sizes that the tensor-core matmuls take (rows of multiples of 16 bytes, more than 16 rows)
bool pib_chunk_scan_fits(int D, int V) { return D % 8 == 0 && D >= 8 && V > 16; }
size_t pib_chunk_scan_bytes(const pib_chunk_scan & a) {
    cs_dev d;
    d.a = a; d.NC = (a.n + CS_C - 1) / CS_C; d.V1 = a.V + (a.ones ? 1 : 0);
    return cs_layout(d, nullptr);
}
int pib_chunk_scan_run(const pib_chunk_scan & a, void * buf, cudaStream_t st) {
    if (!pib_chunk_scan_fits(a.D, a.V) || a.n < 1 || a.H % a.G) { pib_set_error("recurrence as matmuls: sizes not supported"); return PIB_ERR_UNSUPP; }
    cs_dev d;
    d.a = a; d.NC = (a.n + CS_C - 1) / CS_C; d.V1 = a.V + (a.ones ? 1 : 0);
    cs_layout(d, (char *) buf);
    const int Z = d.NC * a.H, D = a.D, V = a.V, V1 = d.V1, KX = 3 * CS_C + 3 * D;
    int rc;
    pib_launch(cs_operands_kernel, dim3((unsigned) Z, 2, (unsigned) ((std::max(D, V) + 31) / 32)), dim3(256), (size_t) 0, st, d);
    CKL();
    auto mm = [&](const bf16 * X, int M, const bf16 * Wt, int N, int K, float * Y) {
        pib_mm m;
        m.W = Wt; m.wtype = PIB_TYPE_BF16; m.ldw = K; m.wz = (int64_t) N * K; m.X = (const float *) X; m.ldx = K; m.xz = (int64_t) M * K; m.x_bf16 = 1;
        m.Y = Y; m.ldy = N; m.yz = (int64_t) M * N; m.M = M; m.N = N; m.K = K; m.Z = Z;
        return pib_dense_mm(m, st);
    };
    if ((rc = mm(d.Ux, V, d.Kt, D, 3 * CS_C, d.Lo)) != PIB_OK) return rc;
    pib_launch(cs_carry_kernel, dim3((unsigned) ((a.H * V1 * D + 255) / 256)), dim3(256), (size_t) 0, st, d);
    CKL();
    if ((rc = mm(d.Qx, CS_C, d.Kw, CS_C, 3 * D, d.Sc)) != PIB_OK) return rc;
    pib_launch(cs_weight_kernel, dim3((unsigned) Z, CS_C / 8), dim3(256), (size_t) 0, st, d);
    CKL();
    if ((rc = mm(d.Px, CS_C, d.Vw, V, KX, d.Yo)) != PIB_OK) return rc;
    pib_launch(cs_order_kernel, dim3((unsigned) a.n), dim3(256), (size_t) 0, st, d);
    CKL();
    return PIB_OK;
}
