// The mma.sync attention kernels for keys of up to 128 elements.
#include "attention_mma.cuh"

namespace b200
{
B200_ATTENTION_DK(128)
}    // namespace b200
