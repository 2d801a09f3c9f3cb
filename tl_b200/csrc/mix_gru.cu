// Gated recurrence per channel (its gates read only the current token), in 32-bit floats:
//   S_t = (1 - z) S_(t-1) + z candidate(u),  out = S_t * silu(gate)
// A prompt is a linear recurrence with known coefficients: a CTA owns 32 channels (a lane each), its warps take consecutive runs of
// tokens, compose their steps into one (factor, term) pair, and every warp starts from the state the runs before it leave.
#include "act.cuh"
#include "layered_kernels.h"
#include "qmv_common.cuh"

namespace tlb {

namespace {

constexpr int kGruWarps = 16, kGruRun = 8, kGruTile = kGruWarps * kGruRun;

template <typename TO>
__global__ void __launch_bounds__(kGruWarps * 32) gru_scan_kernel(const MixGru m, int seq, int T, int pos0, TO *__restrict__ out, int ldo)
{
    __shared__ float s_a[2][kGruWarps][32], s_b[2][kGruWarps][32];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
    const bool live = c < m.width;
    const float *pz = m.proj + c;
    float state = live && pos0 > 0 ? m.state[(size_t)seq * m.width + c] : 0.f;
    float z[kGruRun], u[kGruRun], g[kGruRun];
    auto fetch = [&](int t0) {
        const int n = live ? T - (t0 + warp * kGruRun) : 0;       // tokens of the run that exist
        const float *row = pz + (size_t)(t0 + warp * kGruRun) * m.ldp;
#pragma unroll
        for (int i = 0; i < kGruRun; i++, row += m.ldp) {
            z[i] = i < n ? __ldcs(row) : -INFINITY;          // past the end: z = 0, the state stays
            u[i] = i < n ? __ldcs(row + m.width) : 0.f;
            g[i] = i < n ? __ldcs(row + 2 * m.width) : 0.f;
        }
    };
    fetch(0);
    for (int t0 = 0, b = 0; t0 < T; t0 += kGruTile, b ^= 1) {
        float k[kGruRun], v[kGruRun], w[kGruRun], A = 1.f, B = 0.f;
#pragma unroll
        for (int i = 0; i < kGruRun; i++) {
            const float s = sigmoidf(z[i]);
            k[i] = 1.f - s;
            v[i] = s * gru_candidate(u[i]);
            w[i] = siluf(g[i]);
            A *= k[i];
            B = fmaf(k[i], B, v[i]);
        }
        s_a[b][warp][lane] = A;
        s_b[b][warp][lane] = B;
        if (t0 + kGruTile < T) fetch(t0 + kGruTile);
        __syncthreads();
        float mine = state;
#pragma unroll
        for (int i = 0; i < kGruWarps; i++) {
            if (i == warp) mine = state;
            state = fmaf(s_a[b][i][lane], state, s_b[b][i][lane]);
        }
        const int n = live ? T - (t0 + warp * kGruRun) : 0;
        TO *dst = out + (size_t)(t0 + warp * kGruRun) * ldo + c;
#pragma unroll
        for (int i = 0; i < kGruRun; i++, dst += ldo) {
            mine = fmaf(k[i], mine, v[i]);
            if (i < n) store_actv(dst, mine * w[i]);
        }
    }
    if (live && warp == 0) m.state[(size_t)seq * m.width + c] = state;
}

template <typename TO>
__global__ void __launch_bounds__(128) gru_rows_kernel(const MixGru m, const int *__restrict__ pos, TO *__restrict__ out, int ldo)
{
    const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
    const bool live = c < m.width;
    float *s = m.state + (size_t)b * m.width + c;
    const float old = live && __ldcg(pos + b) > 0 ? *s : 0.f;       // both left by launches of an earlier step
    pdl_wait();
    pdl_launch_dependents();
    if (!live) return;
    const float *row = m.proj + (size_t)b * m.ldp + c;
    const float z = sigmoidf(__ldcg(row)), st = (1.f - z) * old + z * gru_candidate(__ldcg(row + m.width));
    *s = st;
    store_actv(out + (size_t)b * ldo + c, st * siluf(__ldcg(row + 2 * m.width)));
}

tlb_status launched(const char *what)
{
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return cuda_fail(e, what);
    count_launch();
    return TLB_OK;
}

}  // namespace

tlb_status launch_gru_rows(const MixGru &m, int batch, const int *pos, void *out, int ldo, bool out_f32, bool pdl)
{
    const dim3 grid((m.width + 127) / 128, batch);
    if (out_f32) TLB_CUDA(launch_chained(gru_rows_kernel<float>, grid, dim3(128), 0, pdl, m, pos, (float *)out, ldo));
    else TLB_CUDA(launch_chained(gru_rows_kernel<__nv_bfloat16>, grid, dim3(128), 0, pdl, m, pos, (__nv_bfloat16 *)out, ldo));
    count_launch();
    return TLB_OK;
}

tlb_status launch_gru_prefill(const MixGru &m, int seq, int T, int pos0, void *out, int ldo, bool f32)
{
    const int grid = (m.width + 31) / 32;
    if (f32) gru_scan_kernel<<<grid, kGruWarps * 32, 0, ctx()->stream>>>(m, seq, T, pos0, (float *)out, ldo);
    else gru_scan_kernel<<<grid, kGruWarps * 32, 0, ctx()->stream>>>(m, seq, T, pos0, (__nv_bfloat16 *)out, ldo);
    return launched("gated recurrence scan launch");
}

}  // namespace tlb
