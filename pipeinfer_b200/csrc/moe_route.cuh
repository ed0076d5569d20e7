// moe_route.cuh -- device code of a mixture's routing, shared by the kernels that route (hybrid_kernels.cu, sandwich_kernels.cu).
#pragma once

#include "hybrid.cuh"

#define MOE_SMALL_T     16
#define MOE_SMALL_PAIRS 256
#define MOE_SMALL_E     512

// One warp per token: the `top` outputs of the router with the largest choice value (ties: the lower index).
//   PIB_ROUTE_SOFTMAX_RENORM:  scores = softmax over the E logits, weights = score / (sum of the chosen + 1e-20); chosen by the logits
//   PIB_ROUTE_SIGMOID:         weights = sigmoid(logit) of the chosen, as they are (the order of the logits is the order of their sigmoids)
//   PIB_ROUTE_SOFTMAX_GROUPS:  scores = softmax over the E logits; the choice values are score + correction; the outputs form equal groups of neighbours, a group
//                              stands for its largest choice value, and only members of the keep_groups best groups are chosen; weights = score * scale
// cv: the warp's scratch in shared memory, E + groups floats.  Output k of the token goes to ids[k], wts[k].
#define MOE_MAX_TOP 16
__device__ __forceinline__ void moe_route_token(const float * __restrict__ z, const pib_router & R, float * cv, int lane, int32_t * ids, float * wts) {
    const int E = R.E;
    float mx = -INFINITY;
    for (int i = lane; i < E; i += 32) mx = fmaxf(mx, z[i]);
    mx = warp_max(mx);
    float sum = 0.f;
    for (int i = lane; i < E; i += 32) sum += expf(z[i] - mx);
    sum = warp_sum(sum);
    const bool grouped = R.mode == PIB_ROUTE_SOFTMAX_GROUPS;
    for (int i = lane; i < E; i += 32) cv[i] = grouped ? expf(z[i] - mx) / sum + (R.correction ? R.correction[i] : 0.f) : z[i];
    if (grouped && R.keep_groups < R.groups) {
        float *   gv  = cv + E;
        const int per = E / R.groups;
        __syncwarp();
        for (int g = lane; g < R.groups; g += 32) {
            float best = -INFINITY;
            for (int i = g * per; i < (g + 1) * per; i++) best = fmaxf(best, cv[i]);
            gv[g] = best;
        }
        __syncwarp();
        for (int i = lane; i < E; i += 32) {
            const int g = i / per;
            int better = 0;
            for (int o = 0; o < R.groups; o++) better += gv[o] > gv[g] || (gv[o] == gv[g] && o < g);
            if (better >= R.keep_groups) cv[i] = -INFINITY;
        }
    }
    float tot = 0.f, score[MOE_MAX_TOP];
    int   chosen[MOE_MAX_TOP];
    for (int k = 0; k < R.top; k++) {
        float bv = -INFINITY;
        int   bi = 0x7fffffff;
        for (int i = lane; i < E; i += 32) { const float v = cv[i]; if (v > bv || (v == bv && v > -INFINITY && i < bi)) { bv = v; bi = i; } }      // a lane reads back only what it wrote
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int   oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
        }
        if (bi >= E) bi = k;                                // nothing comparable is left (logits that are no numbers): stay inside the arrays
        if ((bi & 31) == lane) cv[bi] = -INFINITY;
        chosen[k] = bi;
        score[k]  = R.mode == PIB_ROUTE_SIGMOID ? 1.0f / (1.0f + expf(-z[bi])) : expf(z[bi] - mx) / sum;
        tot += score[k];
    }
    if (lane == 0)
        for (int k = 0; k < R.top; k++) {
            ids[k] = chosen[k];
            wts[k] = R.mode == PIB_ROUTE_SIGMOID ? score[k] : grouped ? score[k] * R.scale : score[k] / (tot + 1e-20f);
        }
}

// The pairs of a small batch grouped by router output, inside an output in pair order, by one whole block: offs[e] = first sorted position of output e; perm[sorted
// position] = pair; inv[pair] = sorted position; act = [how many of the outputs below n_real have pairs | those outputs].  cnt: E words of shared memory.
__device__ __forceinline__ void moe_sort_small(const int32_t * sid, int P, int E, int n_real, int32_t * cnt, int32_t * __restrict__ offs, int32_t * __restrict__ perm,
                                               int32_t * __restrict__ inv, int32_t * __restrict__ act) {
    for (int e = threadIdx.x; e < E; e += blockDim.x) {
        int n = 0;
        for (int i = 0; i < P; i++) n += sid[i] == e;
        cnt[e] = n;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += blockDim.x) {
        const int n = cnt[e];
        int o = 0, a = 0;
        for (int i = 0; i < e; i++) { o += cnt[i]; a += i < n_real && cnt[i] > 0; }
        offs[e] = o;
        if (e == E - 1) { offs[E] = o + n; act[0] = a + (e < n_real && n > 0); }
        if (n > 0 && e < n_real) act[1 + a] = e;
        if (n > 0) for (int i = 0; i < P; i++) if (sid[i] == e) { perm[o] = i; inv[i] = o; o++; }
    }
}
