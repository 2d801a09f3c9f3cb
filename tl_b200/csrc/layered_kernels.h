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
};
inline int act_ld(int k) { return (k + 7) / 8 * 8; }   // pitch of an activation row that feeds a [.., k] weight

// What the rows of a linear layer's input are made from.
enum DensePro { DPRO_PLAIN = 0, DPRO_NORM = 1, DPRO_POLY = 2 };
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
    bool pdl = true;
};
tlb_status launch_dense_matvec(const DenseMatvecJob &j);
bool dense_matvec_supported(int k);

// T rows: x [T, ldx] in the model's activation type (bf16 or f32)
struct DenseGemmJob {
    DenseW w;
    const void *x = nullptr;
    int ldx = 0, T = 0;
    float *out = nullptr;                 // [T, ldo]
    int ldo = 0;
    const float *resid_scale = nullptr;   // out[t][i] += resid_scale[i] * y instead of out = y + bias
};
tlb_status launch_dense_gemm(const DenseGemmJob &j, bool f32);

// rows in the activation type, pitch ld
tlb_status launch_norm_rows(const float *x, int T, int width, const float *w, float offset, float eps, void *out, int ld, bool f32);
tlb_status launch_poly_rows(const float *z, int T, int ff, int ldz, const float *coef, float eps, void *out, int ld, bool f32);
tlb_status launch_embed_bf16(const int *tokens, const __nv_bfloat16 *table, int width, int ld, float *x, int T);
tlb_status launch_gather_rows(const float *x, int width, const int *idx, int n, float *out);
tlb_status launch_pack_rows(const __nv_bfloat16 *src, int n, int k, __nv_bfloat16 *dst, int ld, int col0);

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
bool mix_attn_supported(int D, int DV);
tlb_status launch_mix_attn_prefill_tc(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo);   // mix_attention_tc.cu: f16 cache
bool mix_attn_prefill_tc_supported(int D, int DV);
tlb_status launch_mix_attn_prefill_tc5(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo);  // prefill_attn_tc.cu: f16 cache, tcgen05
bool mix_attn_prefill_tc5_supported(int D, int DV, int T);

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
