// Instance of the persistent decode kernel for one rank of a tensor-parallel group.
#include "kernel_table.h"
#include "mega_kernel.cuh"

const void* mg::mega_kernel_tp() { return (const void*)mg::mega_decode_kernel<true>; }
