// flash_attn.cu -- attention of long portions over cached key / value heads (served mode) with scores and weights in tensor memory.
//
// One block takes 128 query rows of one problem (key / value head, map): rows are (token, head of the group), the `rep` heads that share the keys next to each other.
// It walks the key columns its tokens can see in tiles of 64 with one pass and running maxima:
//   warp 0       one lane brings the query rows once and every tile's keys and values by TMA (two stages each)
//   warp 1       an elected lane issues tcgen05.mma: scores S = Q K^T of a tile, then O += P V of the tile before the last
//   warps 2..9   two groups of 128 threads, one for the even and one for the odd tiles, a thread per query row: scores from tensor memory, cap, distance bias and
//                mask, running maximum, weights as two bfloat16 parts into shared memory (the operand of the second product).  Each group has its own accumulator
//                in tensor memory, rescaled only when a maximum has grown by more than 2^FA_LAZY; both are merged on the way out
// Scores keep fp32 accuracy on bfloat16 operands: queries and keys enter as their bfloat16 part and the remainder of that rounding, three products are summed
// (hi.hi + lo.hi + hi.lo); weights enter as two parts against the bfloat16 values.  The sink is the running state's start (maximum = sink, denominator = 1).
// The result leaves in token order, divided by the denominator and (optionally) gated.
// Key columns are laid out by kv_gather_kernel (mixer_kernels.cu): [kept first positions (n_front) | positions j0, j0 + 1, ...]; tiles nobody in the block sees are
// not visited.  Every wait is bounded (tc_common.cuh).
#include <cuda_bf16.h>

#include <algorithm>

#include "tc_common.cuh"

#define FA_ROWS    128
#define FA_KEYS    64
#define FA_THREADS 320
#define FA_LAZY    8.0f
#define FA_LOG2E   1.4426950408889634f

struct fa_args {
    int nq, rep, maps, H, V, VN, p0, t0;             // tokens, heads per problem, maps per head, query rows per token, value size (rounded up to 16: VN), first position, first batch row
    int j0, n_front, window, mask, keep;
    float softcap;
    const float * sink, * slopes, * rel; int n_rel;
    const float * gate; int ldg;
    float * out;
    int * err;
};
__device__ __forceinline__ float fa_exp2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ int fa_low(const fa_args & A, int p) { return A.mask == PIB_MASK_CHUNK ? p - p % A.window : max(0, p - A.window + 1); }

template <int NC> struct fa_cfg {                    // NC: 64-wide column chunks of a head (1 or 2)
    static constexpr int Q_TILE = FA_ROWS * 128, K_TILE = FA_KEYS * 128, V_TILE = 128 * 128, P_TILE = FA_ROWS * 128;
    static constexpr int Q_BYTES = 2 * NC * Q_TILE, K_BYTES = 2 * NC * K_TILE, STAGE = K_BYTES + V_TILE;
    static constexpr size_t SMEM = (size_t) Q_BYTES + 2 * STAGE + 4 * P_TILE + 16 * 8 + 32 + 1024;      // weights: two parts per group; the last tiles' shared memory also carries a group's maxima and denominators
};

template <int NC>
__global__ void __launch_bounds__(FA_THREADS)
flash_attn_kernel(const __grid_constant__ CUtensorMap qh, const __grid_constant__ CUtensorMap ql, const __grid_constant__ CUtensorMap kh, const __grid_constant__ CUtensorMap kl,
                  const __grid_constant__ CUtensorMap vm, fa_args A) {
    pib_pdl_wait();
    pib_pdl_trigger();
    using C = fa_cfg<NC>;
    extern __shared__ __align__(1024) uint8_t fa_dsm[];
    uint8_t *  sQ  = fa_dsm + ((1024u - (dt_smem(fa_dsm) & 1023u)) & 1023u);
    uint8_t *  sKV = sQ + C::Q_BYTES;
    uint8_t *  sP  = sKV + 2 * C::STAGE;
    uint64_t * bar = reinterpret_cast<uint64_t *>(sP + 4 * C::P_TILE);
    uint32_t * tmem_slot = reinterpret_cast<uint32_t *>(bar + 16);
    volatile int * abort_s = reinterpret_cast<volatile int *>(tmem_slot + 1);
    // barriers: queries; keys arrived / read, values arrived / read (per stage); scores ready, weights written, product done (per group)
    const uint32_t b0 = dt_smem(bar), bar_q = b0, bar_k = b0 + 8, bar_kf = b0 + 24, bar_v = b0 + 40, bar_vf = b0 + 56, bar_s = b0 + 72, bar_p = b0 + 88, bar_o = b0 + 104;
    // the longest rows' blocks (the portion's last tokens) start first
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, z = blockIdx.y, row0 = (gridDim.x - 1 - blockIdx.x) * FA_ROWS, n_rows = A.nq * A.rep;
    // the tiles this block's tokens see: [0, front) hold kept positions, [first, last] the window
    const int pa = A.p0 + row0 / A.rep, pb = A.p0 + min(n_rows - 1, row0 + FA_ROWS - 1) / A.rep;
    const int first = (A.n_front + fa_low(A, pa) - A.j0) / FA_KEYS, last = (A.n_front + pb - A.j0) / FA_KEYS;
    const int kept = A.n_front > 0 ? A.n_front : min(A.keep, pb + 1), front = (kept + FA_KEYS - 1) / FA_KEYS;
    const bool joined = front >= first;
    const int n_tiles = joined ? last + 1 : front + last - first + 1;
    auto tile_of = [&](int j) { return joined || j < front ? j : first + j - front; };

    if (threadIdx.x == 0) {
        dt_mbar_init(bar_q, 1);
        for (int k = 0; k < 2; k++) {
            for (uint32_t b : { bar_k, bar_kf, bar_v, bar_vf, bar_s, bar_o }) dt_mbar_init(b + 8 * k, 1);
            dt_mbar_init(bar_p + 8 * k, FA_ROWS);
        }
        *abort_s = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(dt_smem(tmem_slot)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    dt_fence_before();
    __syncthreads();
    dt_fence_after();
    const uint32_t tmem = *tmem_slot, tm_o = tmem + 128;          // columns: scores 0..63 and 64..127, outputs 128..255 and 256..383

    if (warp == 0) {
        if (lane == 0) {
            dt_mbar_expect_tx(bar_q, C::Q_BYTES);
            for (int c = 0; c < NC; c++) {
                dt_tma_3d(dt_smem(sQ + c * C::Q_TILE), &qh, bar_q, c * 64, row0, z);
                dt_tma_3d(dt_smem(sQ + (NC + c) * C::Q_TILE), &ql, bar_q, c * 64, row0, z);
            }
            auto keys = [&](int j) {
                const int k = 8 * (j & 1), col = tile_of(j) * FA_KEYS;
                uint8_t * st = sKV + (j & 1) * C::STAGE;
                if (j >= 2 && !dt_mbar_wait(bar_kf + k, ((j >> 1) - 1) & 1, abort_s)) return false;
                dt_mbar_expect_tx(bar_k + k, C::K_BYTES);
                for (int c = 0; c < NC; c++) {
                    dt_tma_3d(dt_smem(st + c * C::K_TILE), &kh, bar_k + k, c * 64, col, z);
                    dt_tma_3d(dt_smem(st + (NC + c) * C::K_TILE), &kl, bar_k + k, c * 64, col, z);
                }
                return true;
            };
            bool ok = keys(0);
            for (int j = 0; j < n_tiles && ok; j++) {               // the keys run one tile ahead: their place is free as soon as the scores before are formed
                const int k = 8 * (j & 1);
                if (j + 1 < n_tiles && !(ok = keys(j + 1))) break;
                if (j >= 2 && !dt_mbar_wait(bar_vf + k, ((j >> 1) - 1) & 1, abort_s)) break;
                dt_mbar_expect_tx(bar_v + k, A.VN * 128);
                dt_tma_3d(dt_smem(sKV + (j & 1) * C::STAGE + C::K_BYTES), &vm, bar_v + k, tile_of(j) * FA_KEYS, 0, z);
            }
        }
    } else if (warp == 1) {
        constexpr uint32_t id_s = dt_idesc(FA_ROWS, FA_KEYS);
        const uint32_t id_o = dt_idesc(FA_ROWS, A.VN);
        const uint64_t dq = dt_desc(dt_smem(sQ)), dp = dt_desc(dt_smem(sP));
        auto scores = [&](int j) {                             // S(j), once its keys are there: three products over the head's columns
            if (!__all_sync(0xffffffffu, dt_mbar_wait(bar_k + 8 * (j & 1), (j >> 1) & 1, abort_s))) return false;
            dt_fence_after();
            const uint64_t dk = dt_desc(dt_smem(sKV + (j & 1) * C::STAGE));
            bool acc = false;
#pragma unroll
            for (int part = 0; part < 3; part++) {
                const uint64_t a = dq + (part == 1 ? (uint64_t) (NC * C::Q_TILE >> 4) : 0), b = dk + (part == 2 ? (uint64_t) (NC * C::K_TILE >> 4) : 0);
#pragma unroll
                for (int c = 0; c < NC; c++)
#pragma unroll
                    for (int k = 0; k < 4; k++) { dt_mma(tmem + 64 * (j & 1), a + (c * C::Q_TILE >> 4) + 2 * k, b + (c * C::K_TILE >> 4) + 2 * k, id_s, acc); acc = true; }
            }
            dt_commit(bar_s + 8 * (j & 1));
            dt_commit(bar_kf + 8 * (j & 1));
            return true;
        };
        bool ok = __all_sync(0xffffffffu, dt_mbar_wait(bar_q, 0, abort_s)) && scores(0) && (n_tiles < 2 || scores(1));
        for (int j = 0; j < n_tiles && ok; j++) {
            ok = __all_sync(0xffffffffu, dt_mbar_wait(bar_p + 8 * (j & 1), (j >> 1) & 1, abort_s));       // the group has read its scores, too: their columns are free
            if (!ok) break;
            if (j + 2 < n_tiles && !(ok = scores(j + 2))) break;
            ok = __all_sync(0xffffffffu, dt_mbar_wait(bar_v + 8 * (j & 1), (j >> 1) & 1, abort_s));
            if (!ok) break;
            dt_fence_after();
            const uint64_t dv = dt_desc(dt_smem(sKV + (j & 1) * C::STAGE + C::K_BYTES)), dw = dp + ((j & 1) * 2 * C::P_TILE >> 4);
#pragma unroll
            for (int part = 0; part < 2; part++)
#pragma unroll
                for (int k = 0; k < 4; k++) dt_mma(tm_o + 128 * (j & 1), dw + (part * C::P_TILE >> 4) + 2 * k, dv + 2 * k, id_o, (j > 1) | ((part | k) != 0));
            dt_commit(bar_o + 8 * (j & 1));
            dt_commit(bar_vf + 8 * (j & 1));
        }
    } else {
        const int w = (warp - 2) >> 2, q4 = warp & 3, rt = q4 * 32 + lane, R = row0 + rt, Rc = min(R, n_rows - 1);
        const int p = A.p0 + Rc / A.rep, h = (z / A.maps * A.rep + Rc % A.rep) * A.maps + z % A.maps;
        const int pmin = A.p0 + min(n_rows - 1, row0 + q4 * 32) / A.rep, pmax = A.p0 + min(n_rows - 1, row0 + q4 * 32 + 31) / A.rep;      // of this warp's rows
        const uint32_t lane_off = (uint32_t) (q4 * 32) << 16;
        const float slope2 = A.slopes ? A.slopes[h] * FA_LOG2E : 0.f;
        const float * rel = A.rel ? A.rel + (size_t) h * A.n_rel : nullptr;
        const bool sunk = A.sink && w == 0;                                                                                              // the sink counts once
        float m = sunk ? A.sink[h] * FA_LOG2E : -INFINITY, l = sunk ? 1.f : 0.f;                                                         // maximum in units of log2
        const uint32_t tm_s = tmem + lane_off + 64 * w, tm_w = tm_o + lane_off + 128 * w;
        uint8_t * prow = sP + w * 2 * C::P_TILE + (rt >> 3) * 1024 + (rt & 7) * 128;
        bool ok = true;
        for (int j = w; j < n_tiles; j += 2) {
            const int c0 = tile_of(j) * FA_KEYS, xb = A.j0 + c0 - A.n_front;       // column c0 + i holds position xb + i (i when it is a kept column in front)
            ok = dt_mbar_wait(bar_s + 8 * w, (j >> 1) & 1, abort_s);
            if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
            dt_fence_after();
            float t[FA_KEYS];
            dt_ld32(tm_s, reinterpret_cast<uint32_t *>(t));
            dt_ld32(tm_s + 32, reinterpret_cast<uint32_t *>(t) + 32);
            dt_wait_ld();
            if (A.softcap > 0.f) {
                const float ic = 1.0f / A.softcap;
#pragma unroll
                for (int i = 0; i < FA_KEYS; i++) t[i] = A.softcap * tanhf(t[i] * ic);
            }
#pragma unroll
            for (int i = 0; i < FA_KEYS; i++) t[i] *= FA_LOG2E;
            if (c0 >= A.n_front) {                                   // no kept column in this tile
                const int d0 = p - xb;
                if (A.slopes) {
                    const float f0 = (float) d0;
#pragma unroll
                    for (int i = 0; i < FA_KEYS; i++) t[i] = fmaf(-slope2, f0 - (float) i, t[i]);
                }
                if (rel) {
                    if (pmin - xb - (FA_KEYS - 1) >= A.n_rel - 1) {  // the whole tile lies where the table has come to its end
                        const float e = rel[A.n_rel - 1];
#pragma unroll
                        for (int i = 0; i < FA_KEYS; i++) t[i] = fmaf(e, FA_LOG2E, t[i]);
                    } else {
#pragma unroll
                        for (int i = 0; i < FA_KEYS; i++) t[i] = fmaf(rel[min(max(d0 - i, 0), A.n_rel - 1)], FA_LOG2E, t[i]);
                    }
                }
                const bool all_seen = xb + FA_KEYS - 1 <= pmin && xb >= fa_low(A, pmax);
                if (!all_seen) {
                    const int lo = fa_low(A, p) - xb;                // columns lo .. d0, and those of kept positions
                    const int ka = A.keep - xb;
#pragma unroll
                    for (int i = 0; i < FA_KEYS; i++) t[i] = i <= d0 && (i >= lo || i < ka) ? t[i] : -INFINITY;
                }
            } else {
                const int lo = fa_low(A, p);
#pragma unroll
                for (int i = 0; i < FA_KEYS; i++) {
                    const int x = c0 + i < A.n_front ? c0 + i : xb + i, d = p - x;
                    if (A.slopes) t[i] = fmaf(-slope2, (float) d, t[i]);
                    if (rel) t[i] = fmaf(rel[min(max(d, 0), A.n_rel - 1)], FA_LOG2E, t[i]);
                    t[i] = d >= 0 && (x >= lo || x < A.keep) ? t[i] : -INFINITY;
                }
            }
            float mt = t[0];
#pragma unroll
            for (int i = 1; i < FA_KEYS; i++) mt = fmaxf(mt, t[i]);
            const bool grow = mt > m + FA_LAZY;                      // also the first key of a row without a sink (m -inf)
            const bool rescale = __any_sync(0xffffffffu, grow);
            float f = 1.f;
            if (grow) { f = fa_exp2(m - mt); m = mt; l *= f; }
            const float ms = m == -INFINITY ? 0.f : m;
            if (j > 1) {                                             // the group's product before has read its weights and left the accumulator
                ok = dt_mbar_wait(bar_o + 8 * w, ((j >> 1) - 1) & 1, abort_s);
                if (!__all_sync(0xffffffffu, ok)) { ok = false; break; }
                if (rescale) {
                    dt_fence_after();
                    for (int c = 0; c < A.VN; c += 32) {
                        uint32_t v[32];
                        dt_ld32(tm_w + c, v);
                        dt_wait_ld();
#pragma unroll
                        for (int i = 0; i < 32; i++) v[i] = __float_as_uint(__uint_as_float(v[i]) * f);
                        dt_st32(tm_w + c, v);
                    }
                    dt_wait_st();
                }
            }
            float l2 = 0.f;
#pragma unroll
            for (int c = 0; c < 8; c++) {                            // 16-byte pieces, swizzled as the descriptor expects them
                uint32_t hi[4], lo4[4];
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const float a = fa_exp2(t[8 * c + 2 * i] - ms), b = fa_exp2(t[8 * c + 2 * i + 1] - ms);
                    l += a; l2 += b;
                    const __nv_bfloat162 h2 = __floats2bfloat162_rn(a, b);
                    hi[i] = *reinterpret_cast<const uint32_t *>(&h2);
                    const __nv_bfloat162 r2 = __floats2bfloat162_rn(a - __uint_as_float(hi[i] << 16), b - __uint_as_float(hi[i] & 0xffff0000u));
                    lo4[i] = *reinterpret_cast<const uint32_t *>(&r2);
                }
                const int off = (c ^ (rt & 7)) * 16;
                *reinterpret_cast<uint4 *>(prow + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *reinterpret_cast<uint4 *>(prow + C::P_TILE + off) = make_uint4(lo4[0], lo4[1], lo4[2], lo4[3]);
            }
            l += l2;
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            dt_fence_before();
            dt_arrive(bar_p + 8 * w);
        }
        // both groups' products are done; maxima and denominators cross through shared memory (the weights' place), then each group writes half of the columns
        const int mine = (n_tiles - 1 - w) >> 1;                     // index of the group's last tile among its own (none: -1)
        if (ok && n_tiles > w) ok = dt_mbar_wait(bar_o + 8 * w, mine & 1, abort_s);
        ok = __all_sync(0xffffffffu, ok);
        asm volatile("bar.sync 1, 256;" ::: "memory");
        float2 * ml = reinterpret_cast<float2 *>(sP);
        ml[w * FA_ROWS + rt] = make_float2(m, l);
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (ok && !*abort_s) {
            dt_fence_after();
            const float2 o = ml[(1 - w) * FA_ROWS + rt];
            const float  M = fmaxf(m, o.x), fm = m == -INFINITY ? 0.f : fa_exp2(m - M), fo = o.x == -INFINITY ? 0.f : fa_exp2(o.x - M), inv = 1.0f / (l * fm + o.y * fo);
            const float  f0 = (w == 0 ? fm : fo) * inv, f1 = (w == 0 ? fo : fm) * inv;
            const size_t t_row = (size_t) (A.t0 + Rc / A.rep);
            float * op = A.out + (t_row * A.H + h) * A.V;
            const float * gp = A.gate ? A.gate + t_row * A.ldg + (size_t) h * A.V : nullptr;
            for (int c = 32 * w; c < A.VN; c += 64) {
                float v[32];
                dt_ld32(tm_o + lane_off + c, reinterpret_cast<uint32_t *>(v));
                dt_wait_ld();
#pragma unroll
                for (int i = 0; i < 32; i++) v[i] *= f0;
                if (n_tiles > 1) {
                    float u[32];
                    dt_ld32(tm_o + lane_off + 128 + c, reinterpret_cast<uint32_t *>(u));
                    dt_wait_ld();
#pragma unroll
                    for (int i = 0; i < 32; i++) v[i] = fmaf(u[i], f1, v[i]);
                }
                if (R >= n_rows) continue;
                if (gp) {
#pragma unroll
                    for (int i = 0; i < 32; i++) if (c + i < A.V) v[i] *= 1.0f / (1.0f + __expf(-gp[c + i]));
                }
                if (A.V % 4 == 0) {
#pragma unroll
                    for (int i = 0; i < 32; i += 4) if (c + i < A.V) *reinterpret_cast<float4 *>(op + c + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
                } else {
#pragma unroll
                    for (int i = 0; i < 32; i++) if (c + i < A.V) op[c + i] = v[i];
                }
            }
        }
    }
    dt_fence_before();
    __syncthreads();
    if (*abort_s) {
        // a wait ran out: say so, give copies and MMAs still in flight time to land (bounded), then free the tensor memory
        if (threadIdx.x == 0) atomicExch(A.err, 1 + (int) blockIdx.x);
        for (int i = 0; i < 2000; i++) __nanosleep(1000);
        __syncthreads();
    }
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
}

bool pib_flash_attention_fits(const pib_hlayer & L) {
    static const int on = getenv("PIB_FLASH_ATTN") ? atoi(getenv("PIB_FLASH_ATTN")) : 1;
    return on != 0 && L.dim % 8 == 0 && L.dim >= 8 && L.dim <= 128 && L.vdim >= 1 && L.vdim <= 128 && !(L.maps > 1 && L.sink);
}

// nq consecutive tokens of one segment (batch rows t0 .., positions p0 ..) over NK gathered key columns: Kb [G * maps][NKp][3 D] = [hi | hi | lo], Vt [G * maps][V][2 NKp] (the first
// half is read), Qc [G * maps][nq * rep][3 D] = [hi | lo | hi], all bfloat16 (kv_gather_kernel, kv_query_rows_kernel)
int pib_flash_attention(const pib_kv_query & q, const pib_hlayer & L, int t0, int nq, int p0, int j0, int n_front, int NK, const void * Kb, const void * Vt, const void * Qc, float * out, cudaStream_t st) {
    const int D = L.dim, V = L.vdim, maps = L.maps, rep = L.heads / L.kv_heads, Z = L.kv_heads * maps, NKp = (NK + 7) & ~7, M = nq * rep;
    const __nv_bfloat16 * kb = (const __nv_bfloat16 *) Kb, * qc = (const __nv_bfloat16 *) Qc;
    CUtensorMap qh, ql, kh, kl, vm;
    const int VN = (V + 15) & ~15;
    int rc = pib_tma_map3(&qh, qc, D, M, Z, 6 * (uint64_t) D, 6 * (uint64_t) D * M, FA_ROWS);
    if (rc == PIB_OK) rc = pib_tma_map3(&ql, qc + D, D, M, Z, 6 * (uint64_t) D, 6 * (uint64_t) D * M, FA_ROWS);
    if (rc == PIB_OK) rc = pib_tma_map3(&kh, kb, D, NKp, Z, 6 * (uint64_t) D, 6 * (uint64_t) D * NKp, FA_KEYS);
    if (rc == PIB_OK) rc = pib_tma_map3(&kl, kb + 2 * D, D, NKp, Z, 6 * (uint64_t) D, 6 * (uint64_t) D * NKp, FA_KEYS);
    if (rc == PIB_OK) rc = pib_tma_map3(&vm, Vt, NKp, V, Z, 4 * (uint64_t) NKp, 4 * (uint64_t) NKp * V, (uint32_t) VN);
    if (rc != PIB_OK) return rc;
    int * err = pib_tc_error_word(st);
    if (!err) { pib_set_error("attention: no error word"); return PIB_ERR_NOMEM; }
    const fa_args A = { nq, rep, maps, L.heads * maps, V, VN, p0, t0, j0, n_front, L.window, L.mask, L.keep, L.softcap, L.sink, L.slopes, L.rel, L.n_rel, q.gate, q.ldg, out, err };
    const dim3 grid((unsigned) ((M + FA_ROWS - 1) / FA_ROWS), (unsigned) Z);
#define FA_GO(NC) do {                                                                                                                             \
        static bool configured = false;                                                                                                            \
        if (!configured) { PIB_CHECK(cudaFuncSetAttribute(flash_attn_kernel<NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int) fa_cfg<NC>::SMEM)); configured = true; } \
        pib_launch(flash_attn_kernel<NC>, grid, dim3(FA_THREADS), fa_cfg<NC>::SMEM, st, qh, ql, kh, kl, vm, A);                                     \
    } while (0)
    if (D <= 64) FA_GO(1); else FA_GO(2);
#undef FA_GO
    PIB_CHECK(cudaGetLastError());
    return PIB_OK;
}
