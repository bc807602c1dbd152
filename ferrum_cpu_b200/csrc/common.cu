// What every model family of the library shares: the error text of a thread, device selection, f32
// uploads, the launch counter, the wait-budget hook and the end-of-step bookkeeping kernel.
#include <cstdarg>
#include <cstdio>

#include "fc_common.cuh"
#include "pdl.cuh"

namespace fc {

// ------------------------------------------------------------------------------- errors
static thread_local char g_err[512] = "";
thread_local int64_t g_launches = 0;
DebugKnobs g_debug;

void set_error(const char* fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_err, sizeof g_err, fmt, ap);
    va_end(ap);
}
const char* g_err_text() { return g_err; }
int fail(int code, const char* fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_err, sizeof g_err, fmt, ap);
    va_end(ap);
    return code;
}
int cuda_fail(cudaError_t e, const char* what, const char* file, int line) {
    snprintf(g_err, sizeof g_err, "CUDA error %d (%s) at %s:%d in %s", (int)e, cudaGetErrorString(e), file, line, what);
    return FC_E_CUDA;
}

// Refuses anything but a Blackwell data-centre part: there is no other code path.
int select_device(int device) {
    int n = 0;
    if (cudaGetDeviceCount(&n) != cudaSuccess || n == 0) {
        cudaGetLastError();
        return fail(FC_E_CUDA, "no CUDA device is visible: libferrum_cuda has no CPU fallback");
    }
    if (device < 0 || device >= n) return fail(FC_E_ARG, "device %d out of range (0..%d)", device, n - 1);
    int major = 0;
    FC_CUDA(cudaDeviceGetAttribute(&major, cudaDevAttrComputeCapabilityMajor, device));
    if (major != 10) return fail(FC_E_CUDA, "device %d has compute capability %d.x; this library is built for sm_100a only", device, major);
    FC_CUDA(cudaSetDevice(device));
    return FC_OK;
}

int upload_f32(Arena& ar, const float* host, size_t n, float** dev, cudaStream_t st) {
    if (!host) return fail(FC_E_FORMAT, "a required f32 tensor is null");
    FC_TRY(ar.alloc_n(dev, n));
    FC_CUDA(cudaMemcpyAsync(*dev, host, n * sizeof(float), cudaMemcpyHostToDevice, st));
    return FC_OK;
}

// ------------------------------------------------------------------- end-of-step bookkeeping
__global__ void step_set_kernel(StepState* st, int pos, int fed, int tail) {
    st->pos = pos; st->fed = fed; st->tail = tail; st->done = 0; st->eos = -1; st->error = 0;
}
int launch_step_set(StepState* state, int pos, int fed, int tail, cudaStream_t st) {
    step_set_kernel<<<1, 1, 0, st>>>(state, pos, fed, tail);
    FC_LAUNCHED();
    return FC_OK;
}
__global__ void step_advance_kernel(StepState* st) {
    pdl_trigger();
    pdl_wait();
    if (st->done | st->error) return;
    st->pos += 1;
    st->fed += 1;
}
int launch_step_advance(StepState* state, cudaStream_t st) {
    step_advance_kernel<<<1, 1, 0, st>>>(state);
    FC_LAUNCHED();
    return FC_OK;
}
// The same as a programmatic dependent of the kernel ahead (steps whose kernels all wait first).
int launch_step_advance_pdl(StepState* state, cudaStream_t st) {
    FC_CUDA(launch_pdl(step_advance_kernel, dim3(1), dim3(1), 0, st, state));
    ++g_launches;
    return FC_OK;
}

}  // namespace fc

using namespace fc;

extern "C" {

const char* fc_last_error(void) { return fc::g_err; }

int fc_device_count(void) {
    int n = 0;
    if (cudaGetDeviceCount(&n) != cudaSuccess) { cudaGetLastError(); return 0; }
    int ok = 0;
    for (int i = 0; i < n; ++i) {
        int major = 0;
        if (cudaDeviceGetAttribute(&major, cudaDevAttrComputeCapabilityMajor, i) == cudaSuccess && major == 10) ++ok;
    }
    return ok;
}

int64_t fc_take_launch_count(void) {
    const int64_t n = g_launches;
    g_launches = 0;
    return n;
}

int fc_debug_set_wait_budget(long long cycles, int withhold_producers) {
    if (cycles <= 0) return fail(FC_E_ARG, "fc_debug_set_wait_budget: cycles = %lld", cycles);
    g_debug.wait_cycles = cycles;
    g_debug.withhold = withhold_producers != 0;
    return FC_OK;
}

}  // extern "C"
