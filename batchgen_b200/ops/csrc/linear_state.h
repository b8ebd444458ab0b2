// Linear-attention recurrences behind one entry point (bg_recurrent_forward, retention.cu): a file per rule.
#pragma once
#include "state_rule.cuh"

namespace bg {
namespace rec {

int channel_delta_forward(const Args& p, cudaStream_t stream);      // channel_delta.cu
int mlstm_forward(const Args& p, cudaStream_t stream);              // mlstm.cu
int hgrn2_forward(const Args& p, cudaStream_t stream);              // hgrn2.cu

}  // namespace rec
}  // namespace bg
