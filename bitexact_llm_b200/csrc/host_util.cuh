// Host-side helpers of the C-ABI translation units (one per shared library): launch accounting, the shadow of the
// device status word, per-device caches of kernel attributes, and the tensor-map encoder of the driver.
#pragma once

#include <cuda.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <atomic>

#include "bx_ptx.cuh"

#ifndef BX_OK
#error "include the C header of the library (status codes) before host_util.cuh"
#endif

namespace {

long long g_launches = 0;   // kernels launched through this library (host-side count)

// Host-side shadow of the device status word: non-zero once the host has SEEN a timed-out device-side wait
// (bx_device_status returned non-zero). Launching entry points then return BX_EDEVICE without
// launching, until bx_clear_device_status. Reading the device word itself needs a synchronising copy, which a
// launch path cannot afford; the engines' check() does that read.
std::atomic<int> g_status_seen{0};

inline int launched(int n) {
  if (cudaGetLastError() != cudaSuccess) return BX_ELAUNCH;
  g_launches += n;
  return BX_OK;
}

// Kernel attributes (opt-in dynamic shared memory) and device properties are per device: every cache of them is
// indexed by the ordinal of the current device. The flags are atomics so that concurrent first calls from several
// host threads are well defined (they would store the same value).
constexpr int BX_MAX_DEVICES = 64;

struct PerDevice {
  std::atomic<int> v[BX_MAX_DEVICES];
};

inline int current_device() {
  int dev = -1;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= BX_MAX_DEVICES) return -1;
  return dev;
}

// Runs `setup` (returns cudaError_t) once per device; BX_OK or BX_ELAUNCH.
template <class F>
inline int once_per_device(PerDevice& done, F&& setup) {
  const int dev = current_device();
  if (dev < 0) return BX_ELAUNCH;
  if (done.v[dev].load(std::memory_order_acquire)) return BX_OK;
  if (setup() != cudaSuccess) return BX_ELAUNCH;
  done.v[dev].store(1, std::memory_order_release);
  return BX_OK;
}

// Number of SMs of the current device (0 on error).
inline int device_sms() {
  static PerDevice sms;
  const int dev = current_device();
  if (dev < 0) return 0;
  int n = sms.v[dev].load(std::memory_order_acquire);
  if (n <= 0) {
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) return 0;
    sms.v[dev].store(n, std::memory_order_release);
  }
  return n;
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

inline EncodeTiledFn encode_fn() {
  static EncodeTiledFn fn = nullptr;
  if (!fn) {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &qres) != cudaSuccess ||
        qres != cudaDriverEntryPointSuccess)
      return nullptr;
    fn = reinterpret_cast<EncodeTiledFn>(p);
  }
  return fn;
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// The device status word of this library: read (synchronises), clear, write.
inline int status_read() {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, bx::g_wait_timeouts, sizeof(int)) != cudaSuccess) return BX_ELAUNCH;
  if (v != 0) g_status_seen.store(1);
  return v;
}

inline int status_clear() {
  int v = 0;
  if (cudaMemcpyToSymbol(bx::g_wait_timeouts, &v, sizeof(int)) != cudaSuccess) return BX_ELAUNCH;
  g_status_seen.store(0);
  return BX_OK;
}

// Only the device word: the host-side shadow follows when the host next reads the word, exactly as after a wait that
// really ran out on the device.
inline int status_write(int value) {
  if (value < 0) return BX_EARG;
  if (cudaMemcpyToSymbol(bx::g_wait_timeouts, &value, sizeof(int)) != cudaSuccess) return BX_ELAUNCH;
  return BX_OK;
}

}  // namespace
