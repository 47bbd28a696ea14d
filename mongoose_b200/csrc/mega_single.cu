// Instance of the persistent decode kernel for one GPU.
#include "kernel_table.h"
#include "mega_kernel.cuh"

const void* mg::mega_kernel_single() { return (const void*)mg::mega_decode_kernel<false>; }
