// End of a step, the same for every model family: next token, position, trace.
#include "common.cuh"
#include "glue.cuh"

namespace alice {

// Turns the packed (ordered logit, ~row) maxima the output-head kernels accumulated - one per rank of a
// tensor-parallel group, each over that rank's rows, all present on every rank by now - into the next token,
// records it, advances the position and clears the keys for the next step.
__global__ void finish_step_kernel(unsigned long long* __restrict__ keys, uint32_t nkeys, int* __restrict__ token,
                                   int* __restrict__ pos, int* __restrict__ trace, int write_token, uint32_t advance,
                                   unsigned int* __restrict__ epoch) {
    pdl_launch_dependents();   // the next kernel may become resident (and prefetch its weights) while this one waits
    pdl_wait();
    if (threadIdx.x == 0 && blockIdx.x == 0) {
        unsigned long long k = 0ull;
        for (uint32_t i = 0; i < nkeys; i++) {
            const unsigned long long ki = __ldcg(keys + i);
            k = ki > k ? ki : k;
            keys[i] = 0ull;
        }
        const int p = *pos;
        if (write_token) {
            const int t = (int)(0xFFFFFFFFu - (uint32_t)(k & 0xFFFFFFFFull));
            *token = t;
            if (trace) trace[p] = t;
        }
        *pos = p + (int)advance;
        if (epoch) *epoch = *epoch + 1u;
    }
}

cudaError_t launch_finish_step(unsigned long long* keys, uint32_t nkeys, int* token, int* pos, int* trace, int write_token,
                               uint32_t advance, unsigned int* epoch, cudaStream_t st, bool pdl) {
    cudaLaunchConfig_t lc = {}; cudaLaunchAttribute at[1];
    lc.gridDim = dim3(1); lc.blockDim = dim3(32); lc.stream = st;
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = 1;
    lc.attrs = at; lc.numAttrs = pdl ? 1 : 0;
    return cudaLaunchKernelEx(&lc, finish_step_kernel, keys, nkeys, token, pos, trace, write_token, advance, epoch);
}


}  // namespace alice
