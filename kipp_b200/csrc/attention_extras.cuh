// Options of the attention kernels beside the plain causal form: what the CUDA-core and mma.sync
// kernels of attention_mix.cu and the tcgen05 prompt kernel of attention_tc.cu are handed.
// The layout is the host's AttentionExtras (host/kernels.hpp).
#pragma once

struct MixExtras {
    const float* sink;         // [n_q] or null
    int key_maps;              // score maps per head (at least 1)
    int values_in_keys;
    int diff;                  // 1: two maps per head are combined (key_maps must be 2)
    float lambda, diff_eps, diff_scale;
    const void* gate;          // [tokens, ld_gate] in the compute type, or null
    long long ld_gate;
    int gate_off;
    int chunk;                 // > 0: blocks of this many positions bound what a query sees (no window then)
    float softcap;             // > 0: a scaled score s becomes softcap * tanh(s / softcap) (before mix, mask and softmax)
    int gate_dims;             // 1: the gate is a number per element of every head instead of one per head
    const float* slopes;       // [n_q] or null
};

// The first key a query at `pos` sees: of its block, of its window, or of the sequence.
__host__ __device__ __forceinline__ int first_visible(int pos, int window, int chunk) {
    const int w = pos - window + 1;
    return chunk > 0 ? pos - pos % chunk : (window > 0 && w > 0 ? w : 0);
}
