#include "layered_kernels.h"
namespace tlb {
bool mix_attn_prefill_tc_supported(int D, int DV) { return false; }
tlb_status launch_mix_attn_prefill_tc(const MixAttn &a, int seq, int T, int pos0, void *out, int ldo) { return fail(TLB_ERR_SHAPE, "x"); }
}
