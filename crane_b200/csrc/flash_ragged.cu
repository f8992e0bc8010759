// Flash attention with operand widths given at run time (see flash.cuh).
#include "flash.cuh"

namespace cb {

template <int D, int DV>
static int ragged_dv(cudaStream_t st, const FlashArgs& a) {
    return a.q_lo_off ? flash_launch_t<D, DV, true, true, true, true>(st, a) : flash_launch_t<D, DV, true, true, false, true>(st, a);
}
template <int D>
static int ragged_d(cudaStream_t st, const FlashArgs& a) {
    if (a.v_w <= 64) return ragged_dv<D, 64>(st, a);
    if (a.v_w <= 128) return ragged_dv<D, 128>(st, a);
    if (a.v_w <= 192) return ragged_dv<D, 192>(st, a);
    if constexpr (D <= 384) return ragged_dv<D, 256>(st, a);
    return -1000;
}
int flash_ragged_launch(cudaStream_t st, const FlashArgs& a) {
    if (!flash_ragged_fits(a.k_w, a.v_w, a.dv) || !a.seq_len || (a.k_heads && a.nkv % a.k_heads)) return -1000;
    if (a.q_lo_off && (a.kv_lo_off == 0 || a.out_lo_off == 0)) return -1000;
    if (((a.q_stride | a.q_lo_off | a.kv_lo_off) & 7) || ((a.o_stride | a.out_lo_off) & 1)) return -1000;
    if (a.k_w <= 64) return ragged_d<64>(st, a);
    if (a.k_w <= 96) return ragged_d<96>(st, a);
    if (a.k_w <= 128) return ragged_d<128>(st, a);
    if (a.k_w <= 192) return ragged_d<192>(st, a);
    if (a.k_w <= 256) return ragged_d<256>(st, a);
    if (a.k_w <= 384) return ragged_d<384>(st, a);
    return ragged_d<512>(st, a);
}

}  // namespace cb
