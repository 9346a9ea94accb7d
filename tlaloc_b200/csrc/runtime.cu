// What every part of the library shares at run time: the thread's error message, the launch counter, the parity-mode
// switch, per-device kernel set-up and device-side status words (each translation unit registers its own), and the
// driver's tensor-map encoder.
#include <atomic>

#include "common.cuh"

namespace tlaloc_b200 {

char* ErrorBuffer()
{
  static thread_local char buf[kErrorBufferBytes] = {0};
  return buf;
}

namespace {
std::atomic<long long> g_launches{0};
std::atomic<int> g_order_faithful{0};

KernelSetup*& SetupList()
{
  static KernelSetup* head = nullptr;
  return head;
}
}  // namespace

KernelSetup::KernelSetup(cudaError_t (*prepare_fn)(), int (*status_fn)()) : prepare(prepare_fn), status(status_fn), next(SetupList())
{
  SetupList() = this;
}

void CountLaunches(int n) { g_launches.fetch_add(n, std::memory_order_relaxed); }
bool OrderFaithful() { return g_order_faithful.load(std::memory_order_relaxed) != 0; }

bool PdlEnabled()
{
  static const bool on = [] {
    const char* e = std::getenv("TLALOC_B200_PDL");
    return e == nullptr || std::atoi(e) != 0;
  }();
  return on;
}

// Resolved once, from kernel set-up, so that no launch has to do it inside a stream capture.
void* TensorMapEncoder()
{
  static void* fn = [] {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult res;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &res) != cudaSuccess || res != cudaDriverEntryPointSuccess) {
      cudaGetLastError();
      ptr = nullptr;
    }
    return ptr;
  }();
  return fn;
}

}  // namespace tlaloc_b200

using namespace tlaloc_b200;

extern "C" int tlaloc_b200_abi_version(void) { return TLALOC_B200_ABI_VERSION; }

extern "C" const char* tlaloc_b200_last_error(void) { return ErrorBuffer(); }

extern "C" long long tlaloc_b200_launch_count(void) { return g_launches.load(std::memory_order_relaxed); }

extern "C" int tlaloc_b200_device_status(void)
{
  int all = 0;
  for (KernelSetup* s = SetupList(); s != nullptr; s = s->next) {
    if (s->status == nullptr) continue;
    const int v = s->status();
    if (v < 0) return -1;
    all |= v;
  }
  return all;
}

extern "C" int tlaloc_b200_set_order_faithful(int on)
{
  return g_order_faithful.exchange(on != 0 ? 1 : 0, std::memory_order_relaxed);
}

extern "C" int tlaloc_b200_init(void)
{
  for (KernelSetup* s = SetupList(); s != nullptr; s = s->next) {
    const cudaError_t e = s->prepare != nullptr ? s->prepare() : cudaSuccess;
    if (e != cudaSuccess) return CudaFail("kernel set-up", e);
  }
  return kOk;
}
