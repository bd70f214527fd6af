// Device, stream and memory ownership (cccc/GpuControl.cpp).
#include "cccc_host.h"

#include <cstdio>

#define LOG_ERR(...) fprintf(stderr, __VA_ARGS__)

namespace cccc
{

thread_local GpuControl* GpuControl::current_gpu_ = nullptr;

static GpuControl::DispatcherFactory g_make_dispatcher = nullptr;

bool GpuControl::setDispatcherFactory(DispatcherFactory f)
{
    g_make_dispatcher = f;
    return true;
}

int GpuControl::init(int device)
{
    int count = 0;
    if (cudaGetDeviceCount(&count) != cudaSuccess || device < 0 || device >= count)
    {
        cudaGetLastError();
        return 1;
    }
    device_ = device;
    if (cudaSetDevice(device_) != cudaSuccess) { return 1; }
    if (cudaStreamCreateWithFlags(&stream_, cudaStreamNonBlocking) != cudaSuccess) { return 1; }
    if (g_make_dispatcher)
    {
        cublas_ = g_make_dispatcher(stream_);
        if (!cublas_) { return 1; }
    }
    current_gpu_ = this;
    return 0;
}

GpuControl::~GpuControl()
{
    if (device_ < 0) { return; }
    cudaSetDevice(device_);
    cublas_.reset();
    for (auto& kv : allocs_) { cudaFree(kv.first); }
    allocs_.clear();
    if (stream_) { cudaStreamDestroy(stream_); }
    if (current_gpu_ == this) { current_gpu_ = nullptr; }
}

void GpuControl::setAsCurrent()
{
    if (current_gpu_ != this || true)
    {
        cudaSetDevice(device_);
        current_gpu_ = this;
    }
}

void* GpuControl::malloc(size_t bytes)
{
    setAsCurrent();
    void* p = nullptr;
    if (cudaMalloc(&p, bytes ? bytes : 1) != cudaSuccess)
    {
        cudaGetLastError();
        LOG_ERR("GpuControl::malloc: %zu bytes failed on device %d\n", bytes, device_);
        return nullptr;
    }
    allocs_[p] = bytes;
    allocated_ += bytes;
    return p;
}

void GpuControl::free(void* p)
{
    auto it = allocs_.find(p);
    if (it == allocs_.end()) { return; }
    setAsCurrent();
    cudaStreamSynchronize(stream_);
    cudaFree(p);
    allocated_ -= it->second;
    allocs_.erase(it);
}

void GpuControl::synchronize() const { cudaStreamSynchronize(stream_); }

}    // namespace cccc
