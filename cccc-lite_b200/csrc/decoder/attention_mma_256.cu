// The mma.sync attention kernels for keys of up to 256 elements.
#include "attention_mma.cuh"

namespace b200
{
B200_ATTENTION_DK(256)
}    // namespace b200
