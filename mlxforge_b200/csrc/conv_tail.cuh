// Moves the inputs that a short convolution over time keeps between steps on: after a step the slot of
// every sequence holds the last taps-1 rows of `x` (32-bit, rows `ld` floats apart, `C` channels), the
// step's own rows and, where it brought fewer, the newest of those that the slot held.
#pragma once
#include "common.cuh"

cudaError_t conv_tail_launch(const float* x, int ld, int C, int taps, float* state, long long state_stride,
                             long long tail_off, const int* seq_q_start, const int* seq_q_len, const int* slots, int n_seqs,
                             cudaStream_t stream);
