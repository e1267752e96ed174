// Kernels of the state-space recurrence with one decay per head and token on bfloat16 activations (float state and sums).
#include "ssd_kernels.cuh"
#define ELEM bf16
#define SSD_CHUNKED
#define FN(name) sllm_##name##_bf16
#include "ssd_launchers.inc"
