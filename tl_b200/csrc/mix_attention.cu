// Softmax attention with a sliding window, a per-head bias by distance and a sink, over a KV cache per sequence: the kernels
// that take any head size and either cache type.
//   mix_attn_decode_kernel   one new token per sequence: append, then 64 keys per CTA (16-byte loads, f32 arithmetic), merged by
//                            the last CTA of a (sequence, KV head)
//   mix_attn_rows_kernel     many tokens, one warp per (token, head): f32 caches, and head sizes the tensor-core kernel does
//                            not take (mix_attention_tc.cu)
// score(i, j) = q_i . k_j * scale - bias[i - j];   weights = exp(score) / (sum exp(score) + exp(sink)).
#include <algorithm>

#include "act.cuh"
#include "layered_kernels.h"
#include "qmv_common.cuh"

namespace tlb {

namespace {

constexpr int kDecThreads = 256, kDecKeys = 64;
constexpr int kMaxHeadDim = 256;

__device__ __forceinline__ void store_act(float *p, float v) { *p = v; }
__device__ __forceinline__ void store_act(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_cache(float *p, float v) { *p = v; }
__device__ __forceinline__ void store_cache(__half *p, float v) { *p = __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }

// 16 bytes of a cache row as floats
template <typename CT> struct Vec;
template <> struct Vec<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void unpack(const uint4 &a, float (&v)[4])
    {
        v[0] = __uint_as_float(a.x); v[1] = __uint_as_float(a.y); v[2] = __uint_as_float(a.z); v[3] = __uint_as_float(a.w);
    }
    static __device__ __forceinline__ void load(const float *p, float (&v)[4]) { unpack(*reinterpret_cast<const uint4 *>(p), v); }
};
template <> struct Vec<__half> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(const __half *p, float (&v)[8]) { unpack(*reinterpret_cast<const uint4 *>(p), v); }
    static __device__ __forceinline__ void unpack(const uint4 &a, float (&v)[8])
    {
        const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const float2 f = h2_to_f2(w[i]);
            v[2 * i] = f.x; v[2 * i + 1] = f.y;
        }
    }
};

// shared floats of the decode kernel: q rows, weights, max / sum per head, per-slice sums of 4 heads
template <typename CT> __host__ __device__ inline int dec_red_floats() { return kDecThreads * 4 * Vec<CT>::N; }

template <typename CT, typename TO>
__global__ void __launch_bounds__(kDecThreads) mix_attn_decode_kernel(const MixAttnDecode j)
{
    constexpr int VE = Vec<CT>::N;
    extern __shared__ __align__(16) float dec_smem[];
    __shared__ int last_cta;
    const MixAttn &a = j.a;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int sp = blockIdx.x, g = blockIdx.y, b = blockIdx.z;
    const int rep = a.H / a.KVH, h0 = g * rep;
    float *sq = dec_smem, *sp_w = sq + rep * a.ldk, *s_b = sp_w + rep * kDecKeys, *s_m = s_b + rep * kDecKeys, *s_l = s_m + rep, *s_red = s_l + rep + (-2 * rep & 3);        // 16-byte aligned
    // The position, and every cache row but the new one, were complete before the launch in front of this one started (they are
    // an earlier step's): they may be touched before the wait.
    const int pos = __ldcg(j.pos + b);
    const int first = max(0, pos - a.window + 1), n = pos - first + 1, nsplit = (n + kDecKeys - 1) / kDecKeys;
    if (sp >= nsplit) { pdl_wait(); pdl_launch_dependents(); return; }
    const int key0 = first + sp * kDecKeys, nk = min(kDecKeys, pos + 1 - key0);
    const float *row = a.proj + (size_t)b * a.ldp;
    CT *kc = reinterpret_cast<CT *>(a.kcache) + (size_t)b * a.seq_stride_k + (size_t)g * a.max_seq * a.ldk;
    CT *vc = reinterpret_cast<CT *>(a.vcache) + (size_t)b * a.seq_stride_v + (size_t)g * a.max_seq * a.ldv;
    for (int i = tid * 128; i < nk * a.ldk * (int)sizeof(CT); i += kDecThreads * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"((const char *)(kc + (size_t)key0 * a.ldk) + i));
    for (int i = tid * 128; i < nk * a.ldv * (int)sizeof(CT); i += kDecThreads * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"((const char *)(vc + (size_t)key0 * a.ldv) + i));
    pdl_wait();
    pdl_launch_dependents();
    for (int r = warp; r < rep; r += kDecThreads / 32)
        for (int d = lane; d < a.ldk; d += 32) sq[r * a.ldk + d] = d < a.D ? __ldcg(row + (size_t)(h0 + r) * a.D + d) : 0.f;
    for (int i = tid; i < rep * kDecKeys; i += kDecThreads) {
        const int r = i / kDecKeys, key = i - r * kDecKeys;
        s_b[i] = a.bias && key < nk ? a.bias[(size_t)(h0 + r) * a.bias_n + (pos - key0 - key)] : 0.f;
    }
    if (sp == nsplit - 1) {          // the new token's rows: this CTA writes them and reads them back like any other
        const float *kn = row + (size_t)a.H * a.D + (size_t)g * a.D, *vn = row + (size_t)(a.H + a.KVH) * a.D + (size_t)g * a.DV;
        for (int d = tid; d < a.D; d += kDecThreads) store_cache(kc + (size_t)pos * a.ldk + d, __ldcg(kn + d));
        for (int d = tid; d < a.DV; d += kDecThreads) store_cache(vc + (size_t)pos * a.ldv + d, __ldcg(vn + d));
    }
    __syncthreads();

    // a thread owns 16 bytes of the V row for every ks-th key: the first few are asked for now, under the scores
    constexpr int PV = 4;
    const int nvv = a.ldv / VE, ks = kDecThreads / nvv, vec = tid % nvv, slice = tid / nvv;
    const CT *vr = vc + (size_t)key0 * a.ldv + vec * VE;
    uint4 pv[PV];
#pragma unroll
    for (int u = 0; u < PV; u++) pv[u] = slice < ks && slice + u * ks < nk ? *reinterpret_cast<const uint4 *>(vr + (size_t)(slice + u * ks) * a.ldv) : make_uint4(0u, 0u, 0u, 0u);

    // scores: `lpk` lanes per key
    const int nvk = a.ldk / VE;
    int lpk = 1;
    while (lpk < nvk && lpk < 32) lpk *= 2;
    const int kpw = 32 / lpk, sub = lane / lpk, ln = lane % lpk;
    constexpr int UK = 4;                       // keys in flight per lane
    const int stride = (kDecThreads / 32) * kpw;
    for (int r0 = 0; r0 < rep; r0 += 4) {
        const int nr = min(4, rep - r0);
        for (int kk = warp * kpw + sub; kk - sub < nk; kk += UK * stride) {
            float acc[UK][4] = {};
            for (int v = ln; v < nvk; v += lpk) {
                float kv[UK][VE];
#pragma unroll
                for (int u = 0; u < UK; u++) Vec<CT>::load(kc + (size_t)(key0 + min(kk + u * stride, nk - 1)) * a.ldk + v * VE, kv[u]);
#pragma unroll
                for (int r = 0; r < 4; r++) {
                    if (r < nr) {
                        const float *qr = sq + (r0 + r) * a.ldk + v * VE;
#pragma unroll
                        for (int e4 = 0; e4 < VE; e4 += 4) {
                            const float4 q4 = *reinterpret_cast<const float4 *>(qr + e4);
                            const float q[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                            for (int e = 0; e < 4; e++)
#pragma unroll
                                for (int u = 0; u < UK; u++) acc[u][r] = fmaf(q[e], kv[u][e4 + e], acc[u][r]);
                        }
                    }
                }
            }
            for (int o = lpk >> 1; o; o >>= 1) {
#pragma unroll
                for (int u = 0; u < UK; u++)
#pragma unroll
                    for (int r = 0; r < 4; r++) acc[u][r] += __shfl_xor_sync(0xffffffffu, acc[u][r], o);
            }
#pragma unroll
            for (int u = 0; u < UK; u++) {
                const int key = kk + u * stride;
                if (ln == 0 && key < nk) {
#pragma unroll
                    for (int r = 0; r < 4; r++)
                        if (r < nr) sp_w[(r0 + r) * kDecKeys + key] = acc[u][r] * a.scale - s_b[(r0 + r) * kDecKeys + key];
                }
            }
        }
    }
    __syncthreads();
    for (int r = warp; r < rep; r += kDecThreads / 32) {
        float *w = sp_w + r * kDecKeys;
        float m = -INFINITY, l = 0.f;
        for (int k = lane; k < nk; k += 32) m = fmaxf(m, w[k]);
        for (int o = 16; o; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        for (int k = lane; k < nk; k += 32) { const float e = expf(w[k] - m); w[k] = e; l += e; }
        for (int o = 16; o; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
        if (lane == 0) { s_m[r] = m; s_l[r] = l; }
    }
    __syncthreads();

    // weighted sum of V
    const int prow = a.ldv + 4;                 // weighted sums, maximum, sum of exponentials; whole 16-byte lines
    float *part = j.partial + ((((size_t)b * a.KVH + g) * gridDim.x + sp) * rep) * prow;
    TO *out = reinterpret_cast<TO *>(j.out) + (size_t)b * j.ldo;
    for (int r0 = 0; r0 < rep; r0 += 4) {
        const int nr = min(4, rep - r0);
        float acc[4][VE] = {};
        if (slice < ks) {
            auto add = [&](int k, const uint4 &raw) {
                float vv[VE];
                Vec<CT>::unpack(raw, vv);
#pragma unroll
                for (int r = 0; r < 4; r++) {
                    if (r < nr) {
                        const float w = sp_w[(r0 + r) * kDecKeys + k];
#pragma unroll
                        for (int e = 0; e < VE; e++) acc[r][e] = fmaf(w, vv[e], acc[r][e]);
                    }
                }
            };
#pragma unroll
            for (int u = 0; u < PV; u++)
                if (slice + u * ks < nk) add(slice + u * ks, pv[u]);
            for (int k = slice + PV * ks; k < nk; k += ks) add(k, *reinterpret_cast<const uint4 *>(vr + (size_t)k * a.ldv));
#pragma unroll
            for (int r = 0; r < 4; r++)
                if (r < nr)
#pragma unroll
                    for (int e = 0; e < VE; e += 4)
                        *reinterpret_cast<float4 *>(s_red + ((size_t)slice * 4 + r) * a.ldv + vec * VE + e) = make_float4(acc[r][e], acc[r][e + 1], acc[r][e + 2], acc[r][e + 3]);
        }
        __syncthreads();
        for (int r = tid >> 6; r < nr; r += kDecThreads / 64) {
            for (int d = tid & 63; d < a.DV; d += 64) {
                float s = 0.f;
#pragma unroll 8
                for (int k = 0; k < min(ks, nk); k++) s += s_red[((size_t)k * 4 + r) * a.ldv + d];
                const int rr = r0 + r;
                if (nsplit == 1) {
                    const float m0 = s_m[rr];
                    float den = s_l[rr], f = 1.f;
                    if (a.sink) {
                        const float sk = a.sink[h0 + rr], m = fmaxf(m0, sk);
                        f = expf(m0 - m);
                        den = den * f + expf(sk - m);
                    }
                    store_act(out + (size_t)(h0 + rr) * a.DV + d, s * f / den);
                } else {
                    part[(size_t)rr * prow + d] = s;
                }
            }
        }
        __syncthreads();
    }
    if (nsplit == 1) return;
    for (int r = tid; r < rep; r += kDecThreads) { part[(size_t)r * prow + a.ldv] = s_m[r]; part[(size_t)r * prow + a.ldv + 1] = s_l[r]; }
    __threadfence();
    __syncthreads();
    if (tid == 0) last_cta = atomicAdd(j.counters + b * a.KVH + g, 1) == nsplit - 1;
    __syncthreads();
    if (!last_cta) return;
    __threadfence();
    const float *pall = j.partial + (((size_t)b * a.KVH + g) * gridDim.x * rep) * prow;
    // every split's factor exp(m - M) / denominator, a warp per head; then the weighted sums
    float *s_f = s_red;
    for (int r = warp; r < rep; r += kDecThreads / 32) {
        float m = a.sink ? a.sink[h0 + r] : -INFINITY, den = 0.f;
        for (int s = lane; s < nsplit; s += 32) m = fmaxf(m, __ldcg(pall + ((size_t)s * rep + r) * prow + a.ldv));
        for (int o = 16; o; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        for (int s = lane; s < nsplit; s += 32) {
            const float *ps = pall + ((size_t)s * rep + r) * prow + a.ldv, f = expf(__ldcg(ps) - m);
            s_f[r * nsplit + s] = f;
            den += f * __ldcg(ps + 1);
        }
        for (int o = 16; o; o >>= 1) den += __shfl_xor_sync(0xffffffffu, den, o);
        if (a.sink) den += expf(a.sink[h0 + r] - m);
        __syncwarp();
        for (int s = lane; s < nsplit; s += 32) s_f[r * nsplit + s] /= den;
    }
    __syncthreads();
    // 16 bytes of a head's row per thread; the splits are dealt over as many threads as there are
    const int q4 = a.ldv / 4, items = rep * q4, ng = max(1, kDecThreads / items), sub_s = (nsplit + ng - 1) / ng;
    float4 *s_o = reinterpret_cast<float4 *>(s_red + (rep * nsplit + 3) / 4 * 4);      // ng > 1: [ng][items]
    for (int i0 = 0; i0 < items; i0 += kDecThreads) {
        const int item = i0 + (ng > 1 ? tid % items : tid), gr = ng > 1 ? tid / items : 0;
        const bool in = item < items && gr < ng;
        const int r = in ? item / q4 : 0, d = in ? (item - r * q4) * 4 : 0;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        if (in) {
            const float *ps = pall + (size_t)r * prow + d;
            const int s1 = min(nsplit, (gr + 1) * sub_s);
#pragma unroll 16
            for (int s = gr * sub_s; s < s1; s++) {
                const float4 x = __ldcg(reinterpret_cast<const float4 *>(ps + (size_t)s * rep * prow));
                const float f = s_f[r * nsplit + s];
                o.x = fmaf(f, x.x, o.x); o.y = fmaf(f, x.y, o.y); o.z = fmaf(f, x.z, o.z); o.w = fmaf(f, x.w, o.w);
            }
            if (gr > 0) s_o[gr * items + item] = o;
        }
        if (ng > 1) __syncthreads();
        if (in && gr == 0) {
            for (int k = 1; k < ng; k++) {
                const float4 x = s_o[k * items + item];
                o.x += x.x; o.y += x.y; o.z += x.z; o.w += x.w;
            }
            const float v[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
            for (int e = 0; e < 4; e++)
                if (d + e < a.DV) store_act(out + (size_t)(h0 + r) * a.DV + d + e, v[e]);
        }
    }
    if (tid == 0) j.counters[b * a.KVH + g] = 0;
}

template <typename CT>
__global__ void mix_attn_append_kernel(const MixAttn a, int seq, int pos0)
{
    const int t = blockIdx.x;
    const float *row = a.proj + (size_t)t * a.ldp + (size_t)a.H * a.D;
    CT *kc = reinterpret_cast<CT *>(a.kcache) + (size_t)seq * a.seq_stride_k, *vc = reinterpret_cast<CT *>(a.vcache) + (size_t)seq * a.seq_stride_v;
    for (int i = threadIdx.x; i < a.KVH * a.D; i += blockDim.x) {
        const int g = i / a.D, d = i - g * a.D;
        store_cache(kc + ((size_t)g * a.max_seq + pos0 + t) * a.ldk + d, row[i]);
    }
    for (int i = threadIdx.x; i < a.KVH * a.DV; i += blockDim.x) {
        const int g = i / a.DV, d = i - g * a.DV;
        store_cache(vc + ((size_t)g * a.max_seq + pos0 + t) * a.ldv + d, row[a.KVH * a.D + i]);
    }
}

constexpr int kRowWarps = 4;

template <typename CT, typename TO>
__global__ void __launch_bounds__(kRowWarps * 32) mix_attn_rows_kernel(const MixAttn a, int seq, int T, int pos0, TO *__restrict__ out, int ldo)
{
    constexpr int VE = Vec<CT>::N;
    __shared__ __align__(16) float sq[kRowWarps][kMaxHeadDim];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x * kRowWarps + warp, h = blockIdx.y, g = h / (a.H / a.KVH);
    if (t >= T) return;
    const CT *kc = reinterpret_cast<const CT *>(a.kcache) + (size_t)seq * a.seq_stride_k + (size_t)g * a.max_seq * a.ldk;
    const CT *vc = reinterpret_cast<const CT *>(a.vcache) + (size_t)seq * a.seq_stride_v + (size_t)g * a.max_seq * a.ldv;
    const float *qrow = a.proj + (size_t)t * a.ldp + (size_t)h * a.D;
    for (int d = lane; d < a.ldk; d += 32) sq[warp][d] = d < a.D ? qrow[d] : 0.f;
    __syncwarp();
    const int pos = pos0 + t, first = max(0, pos - a.window + 1);
    float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f;
    float o[kMaxHeadDim / 32] = {};
    for (int k0 = first; k0 <= pos; k0 += 32) {
        const int key = k0 + lane;
        float s = -INFINITY;
        if (key <= pos) {
            const CT *kr = kc + (size_t)key * a.ldk;
            float acc = 0.f;
            for (int v = 0; v < a.ldk / VE; v++) {
                float kv[VE];
                Vec<CT>::load(kr + v * VE, kv);
#pragma unroll
                for (int e = 0; e < VE; e++) acc = fmaf(sq[warp][v * VE + e], kv[e], acc);
            }
            s = acc * a.scale;
            if (a.bias) s -= a.bias[(size_t)h * a.bias_n + (pos - key)];
        }
        float mx = s;
        for (int off = 16; off; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        const float mn = fmaxf(m, mx), corr = expf(m - mn);      // mn is finite: the first chunk holds at least one key
        const float p = expf(s - mn);
        float sum = p;
        for (int off = 16; off; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
        l = l * corr + sum;
        m = mn;
#pragma unroll
        for (int i = 0; i < kMaxHeadDim / 32; i++) o[i] *= corr;
        const int nk = min(32, pos + 1 - k0);
        for (int kk = 0; kk < nk; kk++) {
            const float w = __shfl_sync(0xffffffffu, p, kk);
            const CT *vr = vc + (size_t)(k0 + kk) * a.ldv;
#pragma unroll
            for (int i = 0; i < kMaxHeadDim / 32; i++)
                if (lane + 32 * i < a.DV) o[i] = fmaf(w, (float)vr[lane + 32 * i], o[i]);
        }
    }
    const float inv = 1.f / l;
    const float *gate = a.gate ? a.gate + (size_t)t * a.ld_gate + (size_t)h * a.DV : nullptr;
#pragma unroll
    for (int i = 0; i < kMaxHeadDim / 32; i++) {
        const int d = lane + 32 * i;
        if (d < a.DV) store_act(out + (size_t)t * ldo + (size_t)h * a.DV + d, gate ? o[i] * inv * sigmoidf(gate[d]) : o[i] * inv);
    }
}

int decode_splits(const MixAttn &a) { return (std::min(a.window, a.max_seq) + kDecKeys - 1) / kDecKeys; }

template <typename CT, typename TO>
tlb_status run_decode(const MixAttnDecode &j)
{
    const MixAttn &a = j.a;
    const int rep = a.H / a.KVH;
    const size_t smem = (size_t)(rep * a.ldk + 2 * rep * kDecKeys + 2 * rep + 4 + std::max(dec_red_floats<CT>(), rep * decode_splits(a) + 4 + 4 * kDecThreads)) * sizeof(float);
    if (smem > ctx()->smem_optin) return fail(TLB_ERR_SHAPE, "attention: %d query heads per KV head of size %d do not fit shared memory", rep, a.D);
    static size_t allowed = 40 << 10;      // with the static part, under the 48 KB that need no asking
    if (smem > allowed) {
        TLB_CUDA(cudaFuncSetAttribute(mix_attn_decode_kernel<CT, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        allowed = smem;
    }
    TLB_CUDA(launch_chained(mix_attn_decode_kernel<CT, TO>, dim3(decode_splits(a), a.KVH, j.batch), dim3(kDecThreads), smem, j.pdl, j));
    count_launch();
    return TLB_OK;
}

}  // namespace

bool mix_attn_supported(int D, int DV) { return D >= 1 && D <= kMaxHeadDim && DV >= 1 && DV <= kMaxHeadDim; }

size_t mix_attn_decode_partial_floats(const MixAttn &a, int batch) { return (size_t)batch * a.KVH * decode_splits(a) * (a.H / a.KVH) * (a.ldv + 4); }

tlb_status launch_mix_attn_decode(const MixAttnDecode &j)
{
    if (j.cache_f32) return j.out_f32 ? run_decode<float, float>(j) : run_decode<float, __nv_bfloat16>(j);
    return j.out_f32 ? run_decode<__half, float>(j) : run_decode<__half, __nv_bfloat16>(j);
}

tlb_status launch_mix_attn_prefill(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo, bool f32)
{
    Context *c = ctx();
    if (!c) return TLB_ERR_DEVICE;
    if (f32) mix_attn_append_kernel<float><<<T, 256, 0, c->stream>>>(a, seq, pos0);
    else mix_attn_append_kernel<__half><<<T, 256, 0, c->stream>>>(a, seq, pos0);
    count_launch();
    TLB_CUDA(cudaGetLastError());
    return launch_mix_attn_prompt(a, seq, T, pos0, out, ldo, f32);
}

tlb_status launch_mix_attn_prompt(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo, bool f32)
{
    Context *c = ctx();
    if (!f32 && mix_attn_prefill_tc5_supported(a.D, a.DV, T)) return launch_mix_attn_prefill_tc5(a, seq, T, pos0, out, ldo);
    if (!f32 && mix_attn_prefill_tc_supported(a.D, a.DV)) return launch_mix_attn_prefill_tc(a, seq, T, pos0, out, ldo);
    const dim3 grid((T + kRowWarps - 1) / kRowWarps, a.H);
    if (f32) mix_attn_rows_kernel<float, float><<<grid, kRowWarps * 32, 0, c->stream>>>(a, seq, T, pos0, (float *)out, ldo);
    else mix_attn_rows_kernel<__half, __nv_bfloat16><<<grid, kRowWarps * 32, 0, c->stream>>>(a, seq, T, pos0, (__nv_bfloat16 *)out, ldo);
    count_launch();
    TLB_CUDA(cudaGetLastError());
    return TLB_OK;
}

}  // namespace tlb
