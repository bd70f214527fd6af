// The mma.sync attention kernels for keys of up to 64 elements.
#include "attention_mma.cuh"

namespace b200
{
B200_ATTENTION_DK(64)
}    // namespace b200
