// hybrid.cuh -- layer-list models: every layer names its own mixer and its own feed-forward.
//   mixers:        windowed latent attention with a sink; the gated linear recurrence HGRN2; windowed softmax attention over cached
//                  key / value heads (grouped queries, short convolutions on q / k / v, per-head query / key norms, value mixing with
//                  an earlier layer); RWKV-style time mixing (token shift, per-channel decay, bonus for the current token); the gated
//                  delta rule; the selective state-space scan (Mamba); a two-branch mixer -- softmax attention over chunks with a sink,
//                  rotated and unit-normed queries / keys, values that are the unrotated keys and a gate per head, beside a linear
//                  attention with a constant decay per head ("lightning attention") -- whose outputs are summed with two constants
//   feed-forwards: dense with a PolyNorm or an xIELU activation; routed mixtures of experts with a shared expert (softmax or sigmoid router,
//                  weights renormalised or not, on the experts' outputs or inputs, relu^2 or clamped gated experts)
//   layer forms:   sequential with LayerNorm on the sublayers' outputs; parallel with two RMS norms of the same input; sequential
//                  pre-norm (RMS norm with ONE number as its weight) with a token shift in front of every mixer
//                  hyper-connections: several residual streams; a sublayer reads a weighted sum of them through a LayerNorm with weight
//                  and bias, and every stream becomes a mix of the old streams plus its own multiple of the sublayer's output
//   layer runs:    a run of layers may be walked several times with the same weights, each walk with a cache and state of its own and
//                  (optionally) opened by a projection of [stream ; embedding] plus a learned vector per walk
//   more mixers:   Mamba-2 (state-space duality: one decay per head and token, keys / queries shared by groups of heads, gate before a
//                  grouped RMS norm); differential attention (two softmax maps per head over the same values, subtracted, per-head unit
//                  RMS; biases, partial rotation with YaRN-scaled frequencies); latent attention without a query latent or sink, rotated
//                  in adjacent pairs
//   more feed-forwards: dense clamped gated (the experts' activation of the mixtures above as one dense block); dense gated with a gelu
//   one more frame: sequential pre-norm with an input convolution in front of BOTH sublayers and a sigmoid gate per channel on what a
//                  sublayer adds to the stream
//   one more mixer: windowed softmax attention that also keeps the sequence's first tokens (one RMS norm over all query rows and one over
//                  all key rows, capped scores, a sink of score 0, a gate per head) beside a matrix memory with exponential gates (mLSTM);
//                  each branch has an output matrix of its own, their outputs are RMS-normed over the width and averaged
//   plain attention: queries, keys and values straight from one projection, which writes the cache cells itself; scores with a distance bias --
//                  a slope per head (ALiBi), or a learned number per head and distance bucket (T5) --, a learned sink or kept first tokens, an
//                  optional sigmoid gate on every value of the heads' outputs; a layer may read another layer's cells (kv_from)
//   and a frame for it: a LayerNorm before and one after every sublayer, the result scaled per channel and by one number (sandwich)
//   more mixtures: softmax scores without renormalisation, chosen by score + correction inside the best groups of neighbours, with identity
//                  outputs that pass the input on; silu-gated experts.  A dense squared-relu feed-forward
// Designs built from these parts: "Rapisun", "Fabivik", "Lulenex", "Putazen", "Bobunex", "Gusedra".  The parts take their sizes and constants as parameters so that another
// layer-list design can name them too.
//
// What such a model adds to the runtime, beside what llama / falcon graphs use:
//   * dense weights (bfloat16 or float32 rows, pib_weight with type PIB_TYPE_BF16 / PIB_TYPE_F32) and the matmul for them (dense_mm.cu);
//   * a per-sequence STATE SLOT (SeqSlots, kv_meta.cuh): the recurrent matrices, the tails of the short convolutions and the
//     position -> cell table of the sequence.  A slot is taken at a sequence's first token and given back by llama_kv_cache_seq_rm of the
//     whole sequence (or _clear / _seq_keep);
//   * KV cells that hold one latent row per caching layer instead of K and V rows; cells are handed out one by one (scattered), so
//     a batch needs no contiguous run of free cells.
#pragma once

#include "engine.cuh"

enum { PIB_MIXER_LATENT = 1, PIB_MIXER_HGRN2 = 2, PIB_MIXER_SWA = 3, PIB_MIXER_WKV = 4, PIB_MIXER_DELTA = 5, PIB_MIXER_SSM = 6, PIB_MIXER_DUAL = 7,
       PIB_MIXER_MAMBA2 = 8, PIB_MIXER_DIFF = 9, PIB_MIXER_ATTN_MEM = 10, PIB_MIXER_KV = 11 };
enum { PIB_MLP_NONE = 0, PIB_MLP_POLYNORM = 1, PIB_MLP_MOE = 2, PIB_MLP_XIELU = 3, PIB_MLP_GLU = 4, PIB_MLP_GEGLU = 5, PIB_MLP_RELU2 = 6 };
// which earlier positions j a token at p may read: the last `window` ones (p - window < j <= p), or those of its own chunk (j / window == p / window)
enum { PIB_MASK_WINDOW = 0, PIB_MASK_CHUNK = 1 };
// what a matmul does to an output on its way out: nothing; max(y, 0)^2; xIELU (y > 0: e0 y^2 + y/2, else e1 (exp(y) - 1 - y) + y/2)
//   PIB_EPI_GLU_PAIR: outputs come in pairs (2 i: gate g, 2 i + 1: linear part u; the weight rows are stored interleaved); output i of a row with pitch ldy is
//   a sigmoid(1.702 a) (b + 1), a = min(g, e0), b = clamp(u, -e0, e0).  N counts the weight rows (twice the outputs).
//   PIB_EPI_GEGLU_PAIR: pairs as above; output i is gelu(g) u, gelu in its tanh form.   PIB_EPI_SWIGLU_PAIR: g sigmoid(g) u.
enum { PIB_EPI_NONE = 0, PIB_EPI_RELU2 = 1, PIB_EPI_XIELU = 2, PIB_EPI_GLU_PAIR = 3, PIB_EPI_GEGLU_PAIR = 4, PIB_EPI_SWIGLU_PAIR = 5 };
// layer forms: x += LN(mixer(conv(x))), x += LN(ff(x))   |   x += mixer(N1(x)) + ff(N2(x)), N = RMS norm with weight (1 + w)
//              x += mixer(shift(N(x))), x += ff(N(x)), N = RMS norm times one number, shift(h)_t = h_t + (h_{t-1} - h_t) * mu
//              hyper-connections over S streams X_s: u = sum_s in_s X_s, y = sublayer(LN(u)) (LayerNorm with weight and bias),
//              X_t <- sum_s mix[s][t] X_s + out_t y, for the mixer and then for the feed-forward; the model's output reads sum_s X_s
//              gated: h = N(x), x += sublayer(h + conv(h)) * sigmoid(R h + r), for the mixer and then for the feed-forward
//              sandwich: x += m ls * LN'(sublayer(LN(x))), both LayerNorms with weight and bias, m one number, ls per channel
enum { PIB_FORM_POSTNORM = 0, PIB_FORM_PARALLEL = 1, PIB_FORM_PRENORM = 2, PIB_FORM_HYPER = 3, PIB_FORM_GATED = 4, PIB_FORM_SANDWICH = 5 };
// how a rotation pairs coordinates: (i, i + dims / 2) or (2 i, 2 i + 1)
enum { PIB_PAIR_HALF = 0, PIB_PAIR_ADJACENT = 1 };
// how a rotation's frequencies are scaled (see pib_hybrid::Rope)
enum { PIB_ROPE_PLAIN = 0, PIB_ROPE_YARN = 1, PIB_ROPE_BANDS = 2 };
// mixture of experts: how the router's logits become weights, where a weight multiplies, what an expert computes
enum { PIB_ROUTE_SOFTMAX_RENORM = 0, PIB_ROUTE_SIGMOID = 1, PIB_ROUTE_SOFTMAX_GROUPS = 2 };
enum { PIB_EXPERT_RELU2 = 0, PIB_EXPERT_GLU_CLAMP = 1, PIB_EXPERT_SWIGLU = 2 };

struct pib_hlayer {
    int     mixer = 0, mlp = 0;
    float * norm1 = nullptr, * norm2 = nullptr;      // LayerNorm weights applied to the sublayers' OUTPUTS
    float * canon = nullptr;                          // [width][taps] causal convolution in front of the mixer (null: none)
    // ---- latent attention ----
    int   heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0, q_rank = 0, window = 0, rot_dims = 0;
    float rot_base = 10000.f, scale = 1.f;
    int   kv_from = -1;                               // layer whose cache rows this layer reads (-1: its own)
    int   cache_id = -1;                              // index among the layers that own cache rows
    int   rope_id = -1;                               // index of the rotation table (distinct base / dims)
    pib_weight * dqkv = nullptr;                      // rows: W_dq (q_rank) | W_dkv (kv_rank + rot_dim, absent when kv_from >= 0)
    pib_weight * uq = nullptr, * ukT = nullptr, * uv = nullptr, * wo = nullptr;   // ukT: per head [kv_rank][dim] (W_uk transposed)
    float * dq_norm = nullptr, * dkv_norm = nullptr, * sink = nullptr;
    // ---- HGRN2 ----
    pib_weight * qfv = nullptr;                       // rows: W_q (heads*dim) | W_f (heads*dim) | W_v (heads*vdim)
    float * f_bias = nullptr, * lower = nullptr, * onorm = nullptr;
    size_t  state_off = 0;                            // floats into a slot's state: the recurrent matrices [heads][dim][vdim]
    size_t  tail_off = 0;                             // floats into a slot's state: the convolution's last taps-1 inputs [taps-1][width]
    // ---- windowed attention over cached key / value heads (PIB_MIXER_SWA): heads query heads share kv_heads key / value heads ----
    int   kv_heads = 0, taps = 0, v_mix = 0;          // taps: of the convolution on q | k | v (0: none); v_mix 1: the first mixing layer (its values are kept for the step), 2: a later one
    pib_weight * qkv = nullptr;                       // rows: W_q (heads*dim) | W_k (kv_heads*dim) | W_v (kv_heads*vdim); delta rule: ... | W_g (heads*vdim) | W_b (heads) | W_a (heads)
    float * conv = nullptr;                           // [channels of q | k | v][taps]
    float * q_norm = nullptr, * k_norm = nullptr;     // [dim], shared by the heads
    float   lambda = 0.f;                             // v <- (1 - lambda) v + lambda v_first
    // ---- RWKV-style time mixing (PIB_MIXER_WKV) ----
    float * mu = nullptr;                             // [5][width]: r, k, v, g, w
    pib_weight * rkvg = nullptr;                      // 4 problems [heads*dim][width]: r, k, v, g
    pib_weight * w1 = nullptr, * w2 = nullptr;        // decay: W_w2 tanh(W_w1 .)
    int   w_rank = 0;
    float * w0 = nullptr, * bonus = nullptr;          // [heads*dim] each
    size_t  shift_off = 0;                            // floats into a slot's state: the previous token's mixer input [width]
    // ---- gated delta rule (PIB_MIXER_DELTA) ----
    float * a_log = nullptr, * dt_bias = nullptr;     // [heads]
    // ---- a layer of a run that is walked several times: the tensors belong to the first walk's entry (the others point at them) ----
    int     weights_of = -1;                          // index of the entry that owns this one's tensors (-1: itself)
    pib_weight * loop_in = nullptr;                   // set on the first layer of a walk: x <- loop_in [x ; embedding] + loop_step
    float * loop_step = nullptr;                      // [width], this walk's row
    // ---- pre-norm form: the norms' single weights, the token shift in front of the mixer ----
    float   g1 = 1.f, g2 = 1.f;
    float * shift = nullptr;                          // [width]; the previous token's normed row lives at shift_off
    // ---- selective state-space scan (PIB_MIXER_SSM): S[c][n] <- exp(dt_c A[c][n]) S[c][n] + dt_c u_c B_n, y_c = sum_n S[c][n] C_n + D_c u_c ----
    int   inner = 0, n_state = 0, dt_rank = 0;        // taps: of the convolution on u
    pib_weight * ssm_in = nullptr, * ssm_x = nullptr, * ssm_dt = nullptr;   // [2 inner][width]: u | z;  [dt_rank + 2 n_state][inner];  [inner][dt_rank]
    float * conv_b = nullptr, * ssm_a = nullptr, * ssm_d = nullptr;         // [inner]; A = -exp(A_log) [inner][n_state]; [inner]   (dt_bias: [inner])
    // ---- two-branch mixer (PIB_MIXER_DUAL) ----
    // softmax branch: heads / kv_heads / dim (= vdim: the values are the unrotated keys) / rot_dims / rot_base / scale / window + mask / sink;
    // linear branch: heads2 x (dim2 -> vdim2), decay per head.  qkv holds the rows of every projection of the mixer's input:
    // q (heads*dim) | k (kv_heads*dim) | head gates (heads) | q2 (heads2*dim2) | k2 (heads2*dim2) | v2 (heads2*vdim2) | gates2 (heads2*vdim2);
    // wo the columns [softmax branch (heads*dim) | linear branch (heads2*vdim2)]
    int   mask = PIB_MASK_WINDOW;
    int   heads2 = 0, dim2 = 0, vdim2 = 0;
    float * proj_bias = nullptr;                      // [rows of qkv], zeros where a projection has none
    float * o_bias = nullptr;                         // [width], already times mix_a
    float * decay = nullptr;                          // [heads2]
    float   mix_a = 1.f, mix_b = 1.f;                 // mixer = mix_a * softmax branch + mix_b * linear branch
                                                      // (state_off: the linear branch's matrices [heads2][dim2][vdim2])
    // ---- hyper-connections (PIB_FORM_HYPER): per sublayer [in (S) | out (S) | mix (S x S, indexed [from][to])]; LayerNorm biases ----
    float * hc1 = nullptr, * hc2 = nullptr;
    float * norm1_b = nullptr, * norm2_b = nullptr;
    // ---- Mamba-2 (PIB_MIXER_MAMBA2): heads x vdim channels, n_state states, kv_heads groups of heads share B and C.  ssm_in rows
    // [z (I) | x (I) | B (G N) | C (G N) | dt (H)], I = heads * vdim; conv / conv_b over x | B | C (taps); dt_bias, a_log, ssm_d per head;
    // per head S [n_state][vdim] <- exp(-exp(a_log) dt) S + dt B x^T, y = S^T C + D x; (y silu(z)) RMS-normed in norm_groups parts, times onorm
    // (state_off: the matrices [heads][n_state][vdim]; tail_off: the convolution's last taps - 1 inputs) ----
    int   norm_groups = 1;
    // ---- differential attention (PIB_MIXER_DIFF): `maps` softmax maps per head over the same values; qkv rows
    // [q (heads * maps * dim) | k (kv_heads * maps * dim) | v (kv_heads * vdim)], head by head [map 1 | map 2], proj_bias over all rows;
    // a cell holds [k (kv_heads * maps * dim) | v (kv_heads * vdim)]; o = a1 - diff_lambda a2, o / rms(o) * diff_out ----
    int   maps = 1;                                   // attention rows per head that share its values (1: ordinary attention)
    float diff_lambda = 0.f, diff_out = 1.f;
    int   rot_pairs = PIB_PAIR_HALF;
    // ---- gated frame (PIB_FORM_GATED): residual gates' matrices and biases, the feed-forward's input convolution (the mixer's: canon, tail_off) ----
    pib_weight * rg1 = nullptr, * rg2 = nullptr;      // [width][width]
    float * rg1_b = nullptr, * rg2_b = nullptr, * canon2 = nullptr;
    size_t  tail2_off = 0;
    // ---- attention beside a matrix memory (PIB_MIXER_ATTN_MEM) ----
    // attention: heads / kv_heads / dim / vdim / rot_dims / scale / window; q_norm [heads*dim] and k_norm [kv_heads*dim] are weights of ONE norm over all
    // rows each; sink: zeros.  memory: heads2 x (dim2 -> vdim2), per head S [dim2][vdim2 + 1], whose last column is the normaliser n (its
    // value is always 1), and the running maximum m: S <- e^(f + m - m') S + e^(i - m') k [v | 1]^T, m' = max(f + m, i).
    // qkv rows: q (heads*dim) | k (kv_heads*dim) | v (kv_heads*vdim) | q2 (heads2*dim2) | k2 (heads2*dim2) | v2 (heads2*vdim2) | output gates (heads2*vdim2) |
    // head gates (heads) | input gates (heads2) | forget gates (heads2); wo [width][heads*vdim], wo2 [width][heads2*vdim2]
    int   keep = 0;                                   // the first `keep` positions are read from everywhere
    float softcap = 0.f;                              // score <- softcap tanh(score / softcap) (0: none)
    float gate_cap = 0.f;                             // the memory's gate logits, the same way
    pib_weight * wo2 = nullptr;
    float * i_bias = nullptr;                         // [heads2]  (forget gates: f_bias)
    float * out_a = nullptr, * out_b = nullptr;       // [width]: weights of the branches' output norms
    size_t  max_off = 0;                              // floats into a slot's state: m [heads2]   (state_off: the matrices)
    // ---- plain attention (PIB_MIXER_KV): qkv rows q (heads*dim) | output gates (heads*vdim, with out_gate) | k (kv_heads*dim) | v (kv_heads*vdim), the last two
    // absent with kv_from; any attention over cached key / value heads can name the distance biases ----
    float * slopes = nullptr;                         // [heads]: score - slope * distance
    float * rel = nullptr;                            // [heads][n_rel]: score + rel[head][min(distance, n_rel - 1)]
    int     n_rel = 0, out_gate = 0;
    // ---- sandwich frame: weights and biases of the norms behind the sublayers, times the layer scale and the residual multiplier ----
    float * post1 = nullptr, * post1_b = nullptr, * post2 = nullptr, * post2_b = nullptr;
    // ---- feed-forward ----
    int   ff = 0;
    pib_weight * up = nullptr, * down = nullptr;
    float act[4] = { 0, 0, 0, 0 };
    int   n_experts = 0, top = 0, ff_e = 0, ff_s = 0;
    pib_weight * e_up = nullptr, * e_down = nullptr;  // experts stacked: [E * ff_e][width], [E * width][ff_e]
    pib_weight * router = nullptr;                    // always float32
    pib_weight * s_up = nullptr, * s_down = nullptr;
    int   route = PIB_ROUTE_SOFTMAX_RENORM, expert = PIB_EXPERT_RELU2;
    float limit_e = 0.f, limit_s = 0.f;               // clamped gated experts: e_up / s_up hold rows gate | up (s_up one more row: the shared expert's gate logit)
    int   s_gate = 0;
    // PIB_ROUTE_SOFTMAX_GROUPS: the router has n_experts + identity outputs in `groups` equal groups of neighbours, of which the `keep_groups` with the
    // largest choice score (score + correction) take part; the chosen ones' softmax scores times route_scale are the weights
    int   identity = 0, groups = 1, keep_groups = 1;
    float route_scale = 1.f;
    float * correction = nullptr;
};

struct pib_hybrid {
    int     dtype = PIB_TYPE_BF16;                    // PIB_TYPE_BF16: matmul operands rounded to bfloat16, fp32 accumulation; PIB_TYPE_F32: all fp32
    int     form = PIB_FORM_POSTNORM;
    int     taps = 1;
    float   eps = 1e-5f;
    float   embd_scale = 1.f, logit_scale = 1.f;      // parallel form: x = embedding * embd_scale, logits = head(norm(x)) * logit_scale
    float * embd_norm = nullptr;
    int     streams = 1;                              // hyper-connections: residual streams per token
    float * final_b = nullptr;                        // hyper-connections: the last LayerNorm's bias (its weight is the model's output_norm)
    std::vector<pib_hlayer> layers;
    size_t  state_floats = 0;                         // per state slot
    float   final_g = 1.f;                            // pre-norm form: the last norm's weight
    int     loops = 0;                                // 1: some layers open a walk (the embedding rows are kept for the step)
    pib_weight * loop_in = nullptr;                   // [width][2 width]
    float * loop_steps = nullptr;                     // [walks][width]
    int     n_cache = 0;
    std::vector<int> cache_row;                       // floats per cell of caching layer i
    // YaRN scaling (factor > 0).  d(n) = dims ln(original / (2 pi n)) / (2 ln base) is the pair index whose wave turns n times over the original
    // context; pairs below a = max(floor(d(fast)), 0) keep their frequency, pairs above b = min(ceil(d(slow)), dims - 1) have it divided by
    // the factor, and between them the blend r_i = clamp((i - a) / max(b - a, 0.001), 0, 1) gives f_i (r_i / factor + 1 - r_i).  The table's
    // cos and sin carry the magnitude 0.1 ln(factor) + 1.
    // Bands (Llama 3.1): waves that turn more than `fast` times over the original context keep their frequency, those that turn less than
    // `slow` times have it divided by the factor, and a wave that turns n times in between gets f ((1 - s) / factor + s), s = (n - slow) / (fast - slow).
    struct Rope {
        float base; int dims; double factor = 0, original = 0, fast = 0, slow = 0; int scaling = PIB_ROPE_PLAIN;
        bool operator==(const Rope & o) const { return base == o.base && dims == o.dims && factor == o.factor && original == o.original && fast == o.fast && slow == o.slow && scaling == o.scaling; }
    };
    std::vector<Rope> ropes;
    // widest per-token scratch rows over all layers
    int     w_proj = 0, w_cq = 0, w_q = 0, w_lat = 0, w_att = 0, w_pairs = 0, w_eup = 0, w_router = 0;
    int     w_conv = 0, w_vfirst = 0, w_shift = 0;    // convolved q | k | v rows, the first mixing layer's values, the five token-shift mixes
    int     w_cat = 0;                                // [stream ; embedding] rows of a walk's opening
    int     w_gate = 0, w_y2 = 0;                     // residual gates' logits, a second branch's output
};

struct pib_hybrid_ctx;
pib_model * pib_model_load_dir(const char * dir, int dtype);          // model_dir.cu: config.json + model.safetensors
pib_model * pib_hybrid_synthetic(const char * config_json, uint64_t seed, int dtype);   // random weights for a configuration (bench)
void        pib_hybrid_model_free(pib_model * m);
int         pib_hybrid_ctx_init(pib_context * c, int n_slots);
void        pib_hybrid_ctx_free(pib_context * c);
int         pib_hybrid_set_slots(pib_context * c, int n_slots);
int         pib_hybrid_slots_free(const pib_context * c);
const char * pib_hybrid_kind_name(int kind);
int         pib_hybrid_profile_read(pib_context * c, int32_t * kind, float * ms, double * flops, double * bytes, int cap);
void        pib_hybrid_on_kv_ops(pib_context * c, const std::vector<KvOp> & ops);
int         pib_hybrid_decode_start(pib_context * c, int n_tokens, const int32_t * token, const int32_t * pos, const int32_t * n_seq_id,
                                    const int32_t * const * seq_id, int batch_id);
pib_run *   pib_take_run(pib_context * c, int n_tokens);               // engine.cu

// dense_mm.cu -- Y[z][m][n] (op)= sum_k X[z][row(m)][k] * W[z][n][k]
struct pib_mm {
    const void *    W = nullptr; int wtype = PIB_TYPE_BF16; int64_t ldw = 0, wz = 0;
    const float *   X = nullptr; int64_t ldx = 0, xz = 0;
    const int32_t * xrows = nullptr; int xdiv = 1;       // row m reads X row xrows[m] / xdiv (null: m)
    float *         Y = nullptr; int64_t ldy = 0, yz = 0;
    int             M = 0, N = 0, K = 0, Z = 1;
    const int32_t * zlist = nullptr;                     // device [1 + Z], with zrange: [how many z have rows | which], so that a few-row launch need not look at the others (at most M of them)
    const int32_t * zrange = nullptr;                    // device [Z + 1]: z owns rows [zrange[z], zrange[z + 1]); null: all M rows, every z
    int             epi = PIB_EPI_NONE;
    float           e0 = 0.f, e1 = 0.f;                  // the epilogue's constants (xIELU: softplus(p), 1/2 + softplus(q))
    int             exact = 0;                           // 1: operands stay fp32 (no bfloat16 rounding of X); W must be float32
    // outputs n >= n2 of row m go to Y2[rows2[m] * ld2 + n - n2] (keys and values straight into their cache cells); Z 1, no paired epilogue
    float *         Y2 = nullptr; int64_t ld2 = 0; int n2 = 0x7fffffff; const int32_t * rows2 = nullptr;
    int             x_bf16 = 0;                          // 1: X already holds bfloat16 rows (ldx in elements, a multiple of 8): tensor-core path only, no staging copy
};
#ifdef __CUDACC__
// FAST (served mode, where the result is rounded to bfloat16 as the next matmul's operand): the exponential through ex2.approx, no branch
template <int EPI, bool FAST> __device__ __forceinline__ float pib_epilogue(float v, float e0, float e1) {
    if (EPI == PIB_EPI_RELU2) { v = fmaxf(v, 0.f); return v * v; }
    if (EPI == PIB_EPI_XIELU) {
        if (FAST) { const float n = fminf(v, 0.f), neg = fmaf(e1, (__expf(n) - 1.0f) - n, 0.5f * v), pos = fmaf(e0 * v, v, 0.5f * v); return v > 0.f ? pos : neg; }
        return v > 0.f ? fmaf(e0 * v, v, 0.5f * v) : fmaf(e1, expm1f(v) - v, 0.5f * v);
    }
    return v;
}
__host__ __device__ constexpr bool pib_epi_pairs(int epi) { return epi == PIB_EPI_GLU_PAIR || epi == PIB_EPI_GEGLU_PAIR || epi == PIB_EPI_SWIGLU_PAIR; }
template <int EPI, bool FAST> __device__ __forceinline__ float pib_glu_pair(float g, float u, float limit) {
    if (EPI == PIB_EPI_GEGLU_PAIR) {      // 0.5 g (1 + tanh z) = g sigmoid(2 z)
        const float z = 0.7978845608028654f * fmaf(0.044715f * g * g, g, g);
        return (FAST ? g / (1.0f + __expf(-2.0f * z)) : 0.5f * g * (1.0f + tanhf(z))) * u;
    }
    if (EPI == PIB_EPI_SWIGLU_PAIR) return g / (1.0f + (FAST ? __expf(-g) : expf(-g))) * u;
    const float a = fminf(g, limit), b = fminf(fmaxf(u, -limit), limit);
    return a / (1.0f + (FAST ? __expf(-1.702f * a) : expf(-1.702f * a))) * (b + 1.0f);
}
#endif
int pib_dense_mm(const pib_mm & a, cudaStream_t st);
int pib_dense_mm_pair(const pib_mm & a, const pib_mm & b, cudaStream_t st);   // two independent matmuls; in decode steps one launch
int pib_dense_mm_experts(const pib_mm & routed, const pib_mm & shared, cudaStream_t st);   // a grouped matmul and a plain one with the same epilogue; in decode steps one launch
int pib_dense_mm_check(cudaStream_t st, int enqueue);   // dense_mma.cu: the error word of the bounded waits (1: copy it in stream order, 0: read the copy)
pib_weight * pib_dense_upload(int type, const void * host, int64_t N, int64_t K);   // type: PIB_TYPE_BF16 / PIB_TYPE_F32, row-major [N][K]

// hybrid_kernels.cu
struct pib_hbatch {                  // device view of one batch's bookkeeping
    const int32_t * tok, * pos, * cell, * slot, * seg;       // [T]
    const int32_t * mmflag;                                   // [T] 1: the token's attention runs in the matmul form (long portions, served mode)
    const int32_t * seg_start, * seg_len, * seg_slot;         // [S]
    int T, S;
};
int pib_embed_ln(const pib_weight * embd, const int32_t * tok, const float * w, float eps, int T, int W, float * x, cudaStream_t st);
int pib_layer_norm(const float * in, const float * w, float eps, int T, int W, float * out, int accumulate, cudaStream_t st);
void pib_rope_table(std::vector<float2> & tab, int n_pos, const pib_hybrid::Rope & r);
int pib_canon_conv(const float * x, const float * w, int taps, const pib_hbatch & b, float * state, size_t state_stride, size_t tail_off, int W, float * h,
                   cudaStream_t st);
int pib_chan_conv(const float * u, int ldu, const float * w, int taps, const pib_hbatch & b, float * state, size_t state_stride, size_t tail_off, int C, float * out, int ldo,
                  int add_input, int silu, cudaStream_t st, const float * bias = nullptr);
// kv_off: where W_dkv's rows start in a projection row (the query latent's rank, or the width of the query rows when the layer has no
// query latent: q_rank 0); ldq: pitch of the query rows [heads][dim + rot_dim]
int pib_latent_prep(const float * proj, int ldp, int kv_off, const pib_hlayer & L, const float * dq_norm, const float * dkv_norm, float eps, const pib_hbatch & b,
                    const float2 * rope, int rope_n_pos, float * cq, float * cache, int cache_row, cudaStream_t st);
int pib_latent_attention(const float * q, int ldq, const float * qlat, const pib_hlayer & L, const pib_hbatch & b, const float2 * rope, int rope_n_pos,
                         const float * cache, int cache_row, const int32_t * cellmap, int n_ctx, float * ctx, const int32_t * skip, cudaStream_t st);
int pib_latent_attention_mm(const float * q, int ldq, const float * qlat, const pib_hlayer & L, const pib_hbatch & b, const float2 * rope, const float * cache, int cache_row,
                            const int32_t * map, int t0, int nq, int j0, int NK, void * Kb, void * Vt, float * Qc, float * S, void * P, float * ctx, cudaStream_t st);
int pib_window_softmax(float * S, void * P, int NKp, int NK, int j0, int window, const int32_t * pos, int t0, int n_rows, int rows_per_z, int rep, const float * sink,
                       cudaStream_t st, int mask = PIB_MASK_WINDOW, int keep = 0, int n_front = 0, float softcap = 0.f, const float * slopes = nullptr, const float * rel = nullptr,
                       int n_rel = 0);
int pib_hgrn2_gates(float * qfv, int ld, const float * f_bias, const float * lower, int T, int HD, cudaStream_t st);
int pib_hgrn2_scan(const float * qfv, int ld, const pib_hlayer & L, const pib_hbatch & b, float * state, size_t state_stride, const float * onorm, float eps,
                   float * out, cudaStream_t st);
int pib_polynorm(float * z, int T, int F, const float * act4, float eps, cudaStream_t st);
struct pib_router { int E = 0, n_real = 0, top = 0, mode = PIB_ROUTE_SOFTMAX_RENORM, groups = 1, keep_groups = 1; float scale = 1.f; const float * correction = nullptr; };   // E outputs, the first n_real of them experts
int pib_moe_router_check(const pib_router & r);
int pib_moe_route(const float * logits, int T, const pib_router & r, int32_t * ids, float * wts, cudaStream_t st);
bool pib_moe_route_sort_fits(int T, const pib_router & r);
int pib_moe_route_sort(const float * logits, int T, const pib_router & r, int32_t * ids, float * wts, int32_t * offs, int32_t * perm, int32_t * inv, int32_t * act,
                       cudaStream_t st);   // both steps of a small batch in one launch; act = [how many experts have pairs | which]
int pib_moe_sort(const int32_t * ids, int n_pairs, int E, int32_t * counts, int32_t * offs, int32_t * perm, int32_t * inv, cudaStream_t st);
int pib_moe_combine(const float * shared, const float * edn, const float * wts, const int32_t * inv, int T, int top, int W, float * y, cudaStream_t st);
int pib_cellmap_set(int32_t * cellmap, int n_ctx, const pib_hbatch & b, cudaStream_t st);

// mixer_kernels.cu
int pib_embed_scale(const pib_weight * embd, const int32_t * tok, float scale, int T, int W, float * x, cudaStream_t st, int copies = 1);
int pib_rms_norm2(const float * x, const float * w1, const float * w2, float eps, float out_scale, int T, int W, float * h1, float * h2, cudaStream_t st);
int pib_swa_prep(const float * cv, int ldc, const pib_hlayer & L, float eps, const pib_hbatch & b, float * q, float * cache, int cache_row, float * vfirst, cudaStream_t st);
struct pib_kv_query {                // query rows [heads * maps][dim] of token t at q + t * ldq; gate (optional): the heads' outputs are multiplied by sigmoid(gate[t * ldg + i])
    const float * q; int ldq; const float * gate = nullptr; int ldg = 0;
};
int pib_kv_attention(const pib_kv_query & q, const pib_hlayer & L, const pib_hbatch & b, const float * cache, int cache_row, const int32_t * cellmap, int n_ctx, float * out,
                     const int32_t * skip, cudaStream_t st);
int pib_kv_attention_mm(const pib_kv_query & q, const pib_hlayer & L, const pib_hbatch & b, const float * cache, int cache_row, const int32_t * map, int t0, int nq, int p0, int j0, int n_front, int NK,
                        void * Kb, void * Vt, float * Qc, float * S, void * P, float * out, cudaStream_t st);
// flash_attn.cu: the same for heads of up to 128 coordinates, scores and weights in tensor memory
bool pib_flash_attention_fits(const pib_hlayer & L);
int pib_flash_attention(const pib_kv_query & q, const pib_hlayer & L, int t0, int nq, int p0, int j0, int n_front, int NK, const void * Kb, const void * Vt, const void * Qc, float * out, cudaStream_t st);
int pib_token_shift(const float * h, const float * mu, int n_mix, const pib_hbatch & b, float * state, size_t state_stride, size_t shift_off, int W, float * mixes, cudaStream_t st);
int pib_rows_act(float * z, int ld, int n, int T, int op, const float * bias, cudaStream_t st);           // op 0: tanh; 1: exp(-exp(z + bias))
int pib_delta_prep(float * cv, int ldc, const pib_hlayer & L, const float * proj, int ldp, int b_off, int a_off, float * bg, int T, cudaStream_t st);
int pib_wkv_scan(const float * rkvg, int ld, const float * wdec, int ldw, const pib_hlayer & L, const pib_hbatch & b, float * state, size_t state_stride, float * out, cudaStream_t st);
int pib_delta_scan(const float * cv, int ldc, const float * bg, const pib_hlayer & L, const pib_hbatch & b, float * state, size_t state_stride, float * out, cudaStream_t st);
int pib_gated_head_norm(float * o, int T, int H, int V, const float * w, int w_hs, const float * gate, int ldg, float eps, cudaStream_t st);
int pib_glu_clamp(float * gu, int ld, int F, float limit, const float * scale, const int32_t * scale_of, int n_rows, cudaStream_t st);
// scan_kernels.cu
int pib_prenorm_shift(const float * xin, const float * y, const float * bias, float * xout, float g, float eps, const float * mu, const pib_hbatch & b, float * state,
                      size_t state_stride, size_t shift_off, int W, float * h, cudaStream_t st);
int pib_embed_pair(const pib_weight * embd, const int32_t * tok, int T, int W, float * x, float * cat, cudaStream_t st);
int pib_concat_stream(const float * xin, const float * y, const float * bias, int T, int W, float * cat, cudaStream_t st);
int pib_ssm_scan(const float * u, int ldu, const float * dtr, int lddt, const float * bc, int ldbc, const float * z, int ldz, const pib_hlayer & L, const pib_hbatch & b,
                 float * state, size_t state_stride, float * out, cudaStream_t st);
int pib_dual_prep(float * proj, int ldp, const pib_hlayer & L, float eps, const pib_hbatch & b, const float2 * rope, float * q, float * cache, int cache_row, cudaStream_t st);
int pib_decay_scan(const float * proj, int ldp, int q_off, int k_off, int v_off, const pib_hlayer & L, const pib_hbatch & b, float * state, size_t state_stride, float * out,
                   cudaStream_t st, float * split_buf = nullptr, int parts = 0, int per = 0);
size_t pib_decay_split_bytes(const pib_hlayer & L, int parts);
int pib_dual_gate(const float * a, const float * bo, const float * proj, int ldp, int ga_off, int gb_off, const pib_hlayer & L, float eps, int T, float * out, cudaStream_t st);
int pib_mamba2_scan(const float * xbc, int ldc, float * dg, const pib_hlayer & L, const pib_hbatch & b, float * state, size_t state_stride, float * out, cudaStream_t st,
                    float * split_buf = nullptr, int parts = 0, int per = 0);
size_t pib_scan_split_bytes(int H, int D, int V, int parts);
int pib_parallel_sum(float * x, const float * mixer, const float * shared, const float * sgl, int ldsg, const float * edn, const int32_t * inv, int top, int T, int W, cudaStream_t st);
// stream_kernels.cu
int pib_hyper_norm(float * X, int S, const float * y, const float * hc_prev, const float * hc_in, const float * w, const float * bias, float eps, int T, int W, float * h,
                   cudaStream_t st);
int pib_mamba2_prep(const float * proj, int ldp, int dt_off, const pib_hlayer & L, int T, float * dg, cudaStream_t st);
int pib_gated_group_norm(float * y, const float * z, int ldz, int T, int C, int groups, const float * w, float eps, cudaStream_t st);
int pib_qkv_rope(const float * proj, int ldp, const pib_hlayer & L, const pib_hbatch & b, const float2 * rope, float * q, float * cache, int cache_row, cudaStream_t st);
// gated_kernels.cu
struct pib_sublayer_out {            // what the sublayer before left for the stream: y = ya, or mix (RMS(ya) wa + RMS(yb) wb); x += y sigmoid(gl + gb)
    const float * ya = nullptr, * wa = nullptr, * yb = nullptr, * wb = nullptr;
    float mix = 1.f;
    const float * gl = nullptr, * gb = nullptr;
};
int pib_gated_norm(float * x, const pib_sublayer_out & o, const float * w, float eps, int W, float * h, const float * conv, int taps, const pib_hbatch & b, float * state,
                   size_t state_stride, size_t tail_off, float * hc, cudaStream_t st);
int pib_attn_mem_prep(const float * proj, int ldp, int i_off, int f_off, const pib_hlayer & L, float eps, const pib_hbatch & b, const float2 * rope, float * q, float * cache,
                      int cache_row, float * state, size_t state_stride, float * dg, cudaStream_t st);
int pib_attn_mem_gate(const float * a, const float * mem, const float * dg, const float * proj, int ldp, int hg_off, int og_off, const pib_hlayer & L, float eps, int T, float * out,
                      int ldo, int mem_off, cudaStream_t st);
int pib_memory_scan(const float * proj, int ldp, int q_off, int k_off, int v_off, float * dg, const pib_hlayer & L, const pib_hbatch & b, float * state, size_t state_stride, float * out,
                    cudaStream_t st, float * split_buf = nullptr, int parts = 0, int per = 0, const int32_t * skip = nullptr);   // mixer_kernels.cu
// sandwich_kernels.cu
struct pib_sublayer_y {              // a sublayer's output: y, plus (top > 0) the routed experts: sum_k w_k edn[inv_k], or w_k hin for ids >= n_real (identity outputs)
    const float * y = nullptr, * edn = nullptr, * wts = nullptr, * hin = nullptr;
    const int32_t * ids = nullptr, * inv = nullptr;
    int top = 0, n_real = 0;
    const float * w = nullptr, * b = nullptr;       // the norm behind it (times layer scale and residual multiplier)
};
struct pib_norm_route {              // the router of the mixture that reads h, on the same launch (small batches): float32 rows [E][W]
    const float * rows = nullptr; pib_router R;
    int32_t * ids = nullptr, * offs = nullptr, * perm = nullptr, * inv = nullptr, * act = nullptr, * done = nullptr;   // done: a word that is 0 between launches
    float * wts = nullptr;
};
bool pib_norm_route_fits(int T, int W, const pib_router & R);
int pib_sandwich_norm(float * x, const pib_sublayer_y & o, const float * w, const float * b, float eps, int T, int W, float * h, cudaStream_t st, const pib_norm_route * route = nullptr);
// chunk_scan.cu: n tokens of one segment (batch rows t0 ..) of a recurrence with one decay per head and token, as matmuls (served mode)
struct pib_chunk_scan {
    const float * q = nullptr, * k = nullptr, * v = nullptr; int ldq = 0, ldk = 0, ldv = 0;   // rows [G][D], [G][D], [H][V] per token
    const float * weight = nullptr, * log_decay = nullptr; int ldg = 0;                       // [T][..H..] each
    int H = 0, G = 0, D = 0, V = 0, ones = 0, t0 = 0, n = 0;                                  // ones: one more value column, always 1
    float * state = nullptr;                                                                  // the segment's matrices [H][D][V (+ 1)]
    float * out = nullptr;                                                                    // [T][H][V (+ 1)]
};
bool   pib_chunk_scan_fits(int D, int V);
size_t pib_chunk_scan_bytes(const pib_chunk_scan & a);
int    pib_chunk_scan_run(const pib_chunk_scan & a, void * buf, cudaStream_t st);
int pib_diff_combine(const float * a, const pib_hlayer & L, float eps, int T, float * out, cudaStream_t st);
