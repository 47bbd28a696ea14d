// Instances of the per-phase decode kernels for the Q8_0 / Q4_0 / fp16 decode block.
#include "kernel_table.h"

namespace mg {

namespace {

template <int FMT>
phase_fn_t phase_fn_fmt(int epi, int R) {
    switch (epi) {
        case EPI_QKV: return phase_kernel<FMT, EPI_QKV, 2, 4>;
        case EPI_SWIGLU: return R == 4 ? phase_kernel<FMT, EPI_SWIGLU, 4, 2> : phase_kernel<FMT, EPI_SWIGLU, 2, 4>;
        case EPI_LOGITS: return phase_kernel<FMT, EPI_LOGITS, 4, 2>;
        default:
            return R == 4 ? phase_kernel<FMT, EPI_RESID, 4, 2>
                 : R == 2 ? phase_kernel<FMT, EPI_RESID, 2, 4>
                          : phase_kernel<FMT, EPI_RESID, 1, 8>;
    }
}

phase_fn_t phase_fn(int fmt, int epi, int R) {
    return fmt == FMT_Q8_0 ? phase_fn_fmt<FMT_Q8_0>(epi, R)
         : fmt == FMT_Q4_0 ? phase_fn_fmt<FMT_Q4_0>(epi, R)
                           : phase_fn_fmt<FMT_F16>(epi, R);
}

attn_fn_t attn_fn(int head_dim) {
    return head_dim == 64 ? attn_decode_kernel<64> : head_dim == 128 ? attn_decode_kernel<128> : attn_decode_kernel<32>;
}

const DenseKernels kTable = {phase_fn, attn_fn, mega_kernel_single, mega_kernel_tp};

}  // namespace

const DenseKernels* dense_kernels() { return &kTable; }

}  // namespace mg
