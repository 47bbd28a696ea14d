// Kernels of the fixed seven-matrix decode block, reached through a table instead of by name: the
// engine's host code then links without them, so that a build that serves only layer-described
// models (mongoose_b200/build.py, family "layered") does not compile them.
#pragma once

#include "decode_kernels.cuh"

namespace mg {

typedef void (*attn_fn_t)(const float*, const __half*, const __half*, float*, const StepState*, int, int, int);

struct DenseKernels {
    phase_fn_t (*phase)(int fmt, int epi, int R);
    attn_fn_t (*attn)(int head_dim);
    const void* (*mega)();      // persistent decode kernel, one GPU
    const void* (*mega_tp)();   // the same as one rank of a tensor-parallel group
};

const void* mega_kernel_single();
const void* mega_kernel_tp();

// NULL in a library built without the dense family.
__attribute__((weak)) const DenseKernels* dense_kernels();

}  // namespace mg
