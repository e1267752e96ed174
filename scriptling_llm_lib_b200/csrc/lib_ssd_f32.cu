// Kernels of the state-space recurrence with one decay per head and token on float activations.
#include "ssd_kernels.cuh"
#define ELEM float
#define FN(name) sllm_##name##_f32
#include "ssd_launchers.inc"
