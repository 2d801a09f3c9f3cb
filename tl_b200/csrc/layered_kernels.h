// Launchers of the kernels a layered model is made of: linear layers on bf16 weights, norms, activations, mixers.  All on
// ctx()->stream.  `f32` selects 32-bit operands (activations, caches) instead of the 16-bit ones.
#pragma once
#include <cuda_bf16.h>

#include "tlb_internal.h"

namespace tlb {

// ---------------------------------------------------------------- dense_linear.cu
// [n, k] bf16 weights, row pitch ld (a multiple of 8, columns past k are zero)
struct DenseW {
    const __nv_bfloat16 *w = nullptr;
    int n = 0, k = 0, ld = 0;
    const float *bias = nullptr;
    bool f16 = false;                     // w holds f16 instead of bf16 (GEMM over f16 rows only)
    // The first `glu` rows (a multiple of 4) are gate and up rows of a gated activation: rows 4 i, 4 i + 1 gates and 4 i + 2, 4 i + 3
    // ups of units 2 i, 2 i + 1.  They yield act(gate) * up of glu / 2 units to act_out; `out` holds the other rows, from 0.
    int glu = 0, glu_act = 0;
};
inline int act_ld(int k) { return (k + 7) / 8 * 8; }   // pitch of an activation row that feeds a [.., k] weight

// What the rows of a linear layer's input are made from.
enum DensePro {
    DPRO_PLAIN = 0,
    DPRO_NORM = 1,      // x / rms * weight
    DPRO_POLY = 2,      // PolyNorm
    DPRO_GNORM = 3,     // residual step of the sublayer before, then the norm in groups
    DPRO_EXPERT = 4,    // plain x; the weight is the expert the router gave this launch's blockIdx.y
    DPRO_EXPERTS = 5,   // activations of the chosen experts and the shared one, each times its weight, side by side
};
enum GluAct { GLU_SILU = 0, GLU_GELU_TANH = 1 };
// Router of a mixture of experts: the `top` best of the experts of the `keep` best groups; weights are scores over their sum * scale.
struct RouteDesc { int experts = 0, groups = 1, keep = 1, top = 0; float scale = 1.f; };
constexpr int kMaxTop = 64, kMaxExperts = 1024;
// One row through one weight (f32 activation, f32 accumulation): out = W pro(x) [+ bias], or with resid_scale
// out[i] += resid_scale[i] * (W pro(x))[i].
struct DenseMatvecJob {
    DenseW w;
    int pro = DPRO_PLAIN;
    const float *x = nullptr;             // [k]
    const __nv_bfloat16 *emb = nullptr;   // NORM: x is row *token of this table [.., k]; CTA 0 also stores it to x_out
    const int *token = nullptr;
    float *x_out = nullptr;
    const float *norm_w = nullptr;        // NORM: x / rms * (norm_w + norm_offset)
    float norm_offset = 0.f, eps = 0.f;
    const float *poly = nullptr;          // POLY: four numbers
    float *out = nullptr;
    const float *resid_scale = nullptr;
    float softcap = 0.f;                  // > 0: out = softcap * tanh(. / softcap)
    // GNORM: the norms are taken over `groups` equal parts.  With y the residual moves on first: x + norm(y * sigmoid(y_gate)) *
    // (post_w + norm_offset); CTA 0 stores it to x_out (not x itself) and, if asked, the normed row to h_out.
    int groups = 1;
    const float *y = nullptr, *y_gate = nullptr, *post_w = nullptr;
    float *h_out = nullptr;
    float *act_out = nullptr;             // w.glu
    // EXPERT: w.n rows per expert (all of them gated activations), experts stacked; slot s of the choice goes to act_out + s * w.n / 2.
    // The choice is stored to sel / weight.
    // EXPERTS: w [experts * w.n, ff]; x [top] rows of pitch ldx; the shared expert (shared.w may be null) has its activations at
    // shared_x and the logit of its weight at shared_gate (null: one)
    int ldx = 0;
    RouteDesc route;
    const float *logits = nullptr;
    int *sel = nullptr;
    float *weight = nullptr;
    DenseW shared;
    const float *shared_x = nullptr, *shared_gate = nullptr;
    bool pdl = true;
};
tlb_status launch_dense_matvec(const DenseMatvecJob &j);
bool dense_matvec_supported(int k);
bool experts_matvec_supported(const RouteDesc &r, int ff, int shared_ff);

// T rows: x [T, ldx] in the model's activation type (bf16 or f32)
struct DenseGemmJob {
    DenseW w;
    const void *x = nullptr;
    int ldx = 0, T = 0;
    float *out = nullptr;                 // [T, ldo]
    int ldo = 0;
    const float *resid_scale = nullptr;   // out[t][i] += resid_scale[i] * y instead of out = y + bias
    float softcap = 0.f;
    // columns in blocks of `per` (0: all), block b at out + b * block_stride; out_h: f16 output at the same places; out_t: f16 output
    // transposed, column c of block b at out_t + b * block_stride + c * ldo, zeros behind the last row up to a multiple of 128
    int per = 0;
    size_t block_stride = 0;
    __half *out_h = nullptr, *out_t = nullptr;
    void *act_out = nullptr;              // w.glu: rows in the activation type, pitch ld_act
    int ld_act = 0;
    // several weights [.., k] of w.n rows each, stacked: tile i covers rows y .. y + z - 1 of x and multiplies them with weight x
    const int4 *tiles = nullptr;
    int n_tiles = 0, tile_rows = 0, n_weights = 1;
};
tlb_status launch_dense_gemm(const DenseGemmJob &j, bool f32);
constexpr int kF32GemmRows = 64;          // rows of a tile of the 32-bit GEMM

// rows in the activation type, pitch ld; x: the first `width` of every ldx numbers, 16-byte aligned
tlb_status launch_norm_rows(const float *x, int T, int width, int ldx, const float *w, float offset, float eps, void *out, int ld, bool f32);
tlb_status launch_poly_rows(const float *z, int T, int ff, int ldz, const float *coef, float eps, void *out, int ld, bool f32);
tlb_status launch_embed_bf16(const int *tokens, const __nv_bfloat16 *table, int width, int ld, float *x, int T);
tlb_status launch_gather_rows(const float *x, int width, const int *idx, int n, float *out);
tlb_status launch_pack_rows(const __nv_bfloat16 *src, int n, int k, __nv_bfloat16 *dst, int ld, int col0);
// rows of a gated activation's gate (up: false) or up matrix to their places among the pairs (DenseW::glu)
tlb_status launch_pack_glu_rows(const __nv_bfloat16 *src, int ff, int k, __nv_bfloat16 *dst, int ld, bool up);
tlb_status launch_pack_rows_f16(const __nv_bfloat16 *src, int n, int k, void *dst, int ld);      // values as f16

// ---------------------------------------------------------------- resid_rows.cu
// What a mixture of experts leaves per token: y = sum over the choice of weight * part[slot] + sigmoid(shared_gate) * shared.
struct MoeRows {
    int top = 0;
    const int *slot = nullptr;            // [T][top] rows of part
    const float *weight = nullptr, *part = nullptr, *shared = nullptr, *shared_gate = nullptr;
    int ld_shared_gate = 0;
};
// Rows of the residual: x += norm(y * sigmoid(gate)) * (post_w + offset), both norms over `groups` parts; then, if norm_w is given,
// out = norm(x) * (norm_w + offset) in the activation type.  y null and moe null: the second step alone.
struct ResidNormJob {
    float *x = nullptr;
    int T = 0, width = 0, groups = 1;
    float offset = 0.f, eps = 0.f;
    const float *y = nullptr;             // [T, width]
    const MoeRows *moe = nullptr;
    const float *gate = nullptr;          // row 0; null: none
    int ld_gate = 0;
    const float *post_w = nullptr, *norm_w = nullptr;
    void *out = nullptr;
    int ldo = 0;
};
tlb_status launch_resid_norm_rows(const ResidNormJob &j, bool f32);

// ---------------------------------------------------------------- moe.cu
// The choice of T tokens and the order their rows take behind one another, expert by expert.
struct MoePlan {
    int *sel = nullptr, *place = nullptr;   // [T][top]: expert; row within the expert's part, then the row over all experts
    float *weight = nullptr;                // [T][top]
    int *count = nullptr;                   // [2 * experts]: rows per expert, first row
    int4 *tiles = nullptr;                  // (expert, first row, rows, 0), moe_max_tiles of them; rows 0: nothing to do
};
int moe_tile_rows(const RouteDesc &r, int T, bool f32);
int moe_max_tiles(const RouteDesc &r, int T, bool f32);
tlb_status launch_moe_plan(const RouteDesc &r, const float *logits, int ldl, int T, const MoePlan &p, bool f32);
// rows of act (pitch ld, activation type) to the places of their choices
tlb_status launch_moe_gather(const RouteDesc &r, const MoePlan &p, const void *act, int T, int ld, void *out, bool f32);

// ---------------------------------------------------------------- mix_attention.cu
// Softmax attention with optional window, per-head bias by distance and sink.
struct MixAttn {
    int H, KVH, D, DV, ldk, ldv;          // cache row pitches in elements (multiples of 8, padding zero)
    int max_seq, window;                  // window: keys a query sees (max_seq: all)
    float scale;
    const float *bias;                    // [H][bias_n] taken off the score at distance i, or null; bias_n >= min(window, max_seq)
    int bias_n;
    const float *sink;                    // [H] or null
    void *kcache, *vcache;                // [seq][KVH][max_seq][ld], f32 or f16
    size_t seq_stride_k, seq_stride_v;    // elements
    // rows of projections: q at column 0, k at H * D, v at H * D + KVH * D
    const float *proj;
    int ldp;
    const float *gate;                    // prompts: [T, ld_gate] logits of a gate on every output element, or null
    int ld_gate;
    // tcgen05 prompt kernel, instead of proj and vcache: queries [T][H * mix_attn_tc5_qd(D)] padded with zeros, V^T [KVH][128][vt_ld]
    const __half *q16, *vt;
    int vt_ld;
};
// One new token per sequence (rows of proj), at *pos: append and attend.  out: rows of H * DV in the activation type (out_f32: f32), pitch ldo.
struct MixAttnDecode {
    MixAttn a;
    int batch;
    const int *pos;                       // [batch]
    float *partial;                       // attn_decode_partial_floats
    int *counters;                        // [batch * KVH], zero
    void *out;
    int ldo;
    bool out_f32, cache_f32, pdl;
};
size_t mix_attn_decode_partial_floats(const MixAttn &a, int batch);
tlb_status launch_mix_attn_decode(const MixAttnDecode &j);
// T tokens of sequence seq at rows pos0 ..: append, then attend.
tlb_status launch_mix_attn_prefill(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo, bool f32);
tlb_status launch_mix_attn_prompt(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo, bool f32);      // rows already appended
bool mix_attn_supported(int D, int DV);
tlb_status launch_mix_attn_prefill_tc(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo);   // mix_attention_tc.cu: f16 cache
bool mix_attn_prefill_tc_supported(int D, int DV);
tlb_status launch_mix_attn_prefill_tc5(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo);  // prefill_attn_tc.cu: f16 cache, tcgen05
bool mix_attn_prefill_tc5_supported(int D, int DV, int T);
inline int mix_attn_tc5_qd(int D) { return D > 128 ? 192 : 128; }

// ---------------------------------------------------------------- mix_recurrent.cu
// Linear recurrences with a matrix state per head, S[value channel][key channel] (key channels padded to ld), f32.
struct MixRecur {
    int H, D, DV, ld;
    float *state;                         // [seq][H][DV][ld]
    size_t seq_stride;
    float eps;
    const float *decay;                   // retention: [H]
    const float *rot_cos, *rot_sin;       // retention: [max position][rot / 2] or null
    int rot;
    const float *norm_w;                  // general delta: [H * DV]
    // general delta: second half of the decay's projection and its constant
    DenseW w2;
    const float *w0;
    int rank;
    float *proj;                          // retention rows: q | k | v | g; general delta rows: r | k | v | g | a | w1   (f32, pitch ldp)
    int ldp;
};
struct MixRecurDecode {
    MixRecur m;
    int batch;
    const int *pos, *rope_pos;            // [batch]; position 0 starts from a zero state
    void *out;                            // gated rows [H * DV]
    int ldo;
    bool out_f32, pdl;
};
bool mix_recur_supported(int D, int DV);
int mix_recur_ld(int D);                  // pitch of the state's key channels
tlb_status launch_retention_decode(const MixRecurDecode &j);
tlb_status launch_delta_decode(const MixRecurDecode &j);
// T tokens of one sequence; `o` is scratch [T, H * DV] f32; out in the activation type
tlb_status launch_retention_prefill(const MixRecur &m, int seq, int T, int pos0, int rope0, int rope_step, float *o, void *out, int ldo, bool f32);
// decay: scratch [T, H * D] f32 that holds W_w2 tanh(W_w1 h) on entry; look: scratch [H, scan_look_ld(T)]
int scan_look_ld(int T);
tlb_status launch_delta_prefill(const MixRecur &m, int seq, int T, int pos0, float *decay, float2 *look, float *o, void *out, int ldo, bool f32);
// tanh of the first step of the decay's projection as two activation-type terms (value and remainder): out [T, 2 * ldh]
tlb_status launch_tanh_split(const float *x, int T, int rank, int ldx, void *out, int ldh, bool f32);

// ---------------------------------------------------------------- mix_latent.cu
// Latent attention: the cache holds, per token, a normed latent of R values and one rotated key part of RD values that all heads
// share (row pitch ld).  Keys and values of a head are W_uk c and W_uv c.  Rows of queries are attended in the latent space: W_uk goes
// to the query, W_uv to the weighted sum of latents; long portions of a prompt expand the visible keys and values instead.
struct MixLatent {
    int H, D, RD, DV, R, ld;              // D: unrotated dimensions of a head's query, which is [D | RD]
    int max_seq, window;
    float scale, eps;
    int rot;                              // leading dimensions of the RD that turn, in pairs of neighbours
    const float *rot_cos, *rot_sin;       // [position][rot / 2]
    const float *c_norm;                  // [R]
    DenseW uk, uv;                        // [H * D, R], [H * DV, R] bf16
    DenseW uk16, uv16;                    // the same as f16 (16-bit sessions)
    void *cache;                          // [seq][max_seq][ld], f32 or f16
    size_t seq_stride;
    float *q;                             // rows of queries [H][D + RD], pitch ldq
    int ldq;
    const float *kv;                      // rows of W_dkv h [R + RD], pitch ldkv
    int ldkv;
    const float *gate;                    // rows of H * DV logits, pitch ld_gate, or null
    int ld_gate;
};
// `rows` queries, each the newest token of its sequence or of those before it in a portion: row i of sequence seq0 + i * seq_step at
// position pos[i] (or pos0 + i), angles of rope_pos[i] (or rope0 + i * rope_step).  Appends, attends, writes gated rows [H * DV].
struct MixLatentRows {
    MixLatent m;
    int rows, seq0, seq_step;
    const int *pos, *rope_pos;
    int pos0, rope0, rope_step;
    void *qa;                             // scratch: rows * H * ld activations of the cache type
    float *partial;                       // scratch: latent_partial_floats
    void *out;
    int ldo;
    bool f32, out_f32, pdl;               // f32: cache and scores' operands
};
size_t latent_partial_floats(const MixLatent &m, int rows);
tlb_status launch_latent_rows(const MixLatentRows &j);
bool latent_supported(const MixLatent &m, bool f32);
int latent_ld(int R, int RD);
// portions with at least this many tokens expand keys and values
bool latent_expands(const MixLatent &m, int T);
tlb_status launch_latent_prompt(const MixLatent &m, int seq, int T, int pos0, int rope0, int rope_step, void *out, int ldo, bool f32);

// ---------------------------------------------------------------- mix_gru.cu
// Gated recurrence per channel, S <- (1 - z) S + z candidate(u); rows z | u | gate logits, each `width` wide; out = S * silu(gate).
struct MixGru {
    int width;
    float *state;                         // [seq][width]
    const float *proj;
    int ldp;
};
tlb_status launch_gru_rows(const MixGru &m, int batch, const int *pos, void *out, int ldo, bool out_f32, bool pdl);
tlb_status launch_gru_prefill(const MixGru &m, int seq, int T, int pos0, void *out, int ldo, bool f32);

// launch with programmatic dependent launch (the kernel calls griddepcontrol.wait before it touches what precedes it)
template <typename... KArgs, typename... Args>
inline cudaError_t launch_chained(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, bool pdl, Args... args)
{
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx()->stream;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = pdl ? 1 : 0;
    cfg.attrs = at;
    cfg.numAttrs = 1;
    return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

}  // namespace tlb
