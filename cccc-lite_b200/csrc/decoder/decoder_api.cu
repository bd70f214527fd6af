// Library-wide state of the decoder operations: launch counter, device facts, the status word of bounded waits.
#include "decoder_common.cuh"

#include <atomic>

namespace b200
{

static std::atomic<unsigned long long> g_launches{ 0 };
void count_launch() { g_launches.fetch_add(1, std::memory_order_relaxed); }

int report_launch(const char* label)
{
    const cudaError_t e = cudaGetLastError();
    if (e == cudaSuccess) { return 0; }
    fprintf(stderr, "%s kernel launch failed: %s\n", label, cudaGetErrorString(e));
    return 1;
}

__device__ unsigned int g_decoder_status;

unsigned int* decoder_status_word()
{
    void* p = nullptr;
    if (cudaGetSymbolAddress(&p, g_decoder_status) != cudaSuccess)
    {
        cudaGetLastError();
        return nullptr;
    }
    return (unsigned int*)p;
}

const DecoderDevice* decoder_device()
{
    static DecoderDevice facts[64];
    static std::atomic<int> ready[64];
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) { return nullptr; }
    if (ready[dev].load(std::memory_order_acquire) == 0)
    {
        int sms = 0, smem = 0;
        if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess
            || cudaDeviceGetAttribute(&smem, cudaDevAttrMaxSharedMemoryPerBlockOptin, dev) != cudaSuccess)
        {
            return nullptr;
        }
        facts[dev].sm_count = sms;    // two threads may both write the same values: harmless
        facts[dev].max_smem = smem;
        ready[dev].store(1, std::memory_order_release);
    }
    return &facts[dev];
}

}    // namespace b200

using namespace b200;

C_EXPORT int cuda_b200_decoder_check(const char* label)
{
    const cudaError_t s = cudaDeviceSynchronize(), l = cudaGetLastError();
    const cudaError_t e = s != cudaSuccess ? s : l;
    if (e != cudaSuccess)
    {
        fprintf(stderr, "%s: %s\n", label ? label : "decoder", cudaGetErrorString(e));
        return 1;
    }
    unsigned int* w = decoder_status_word();
    unsigned int st = 0;
    if (w && cudaMemcpy(&st, w, sizeof(st), cudaMemcpyDeviceToHost) == cudaSuccess && st != 0)
    {
        fprintf(stderr, "%s: a bounded wait ran out (kernel %u, role %u, step %u)\n", label ? label : "decoder", st >> 28, (st >> 24) & 15u, st & 0xFFFFFFu);
        cudaMemset(w, 0, sizeof(st));
        return 1;
    }
    return 0;
}

C_EXPORT unsigned long long cuda_b200_decoder_launches(void) { return g_launches.load(std::memory_order_relaxed); }
