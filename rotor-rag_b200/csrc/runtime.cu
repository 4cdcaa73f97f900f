// Process- and device-wide state every kernel file shares: launch count, launch attributes, the status
// word that bounded device-side waits write to, device properties.
#include "model.cuh"

namespace rb {

unsigned long long g_launch_count = 0;

int g_use_pdl = 1;  // programmatic dependent launch for the kernels that call pdl_wait()

// Device status word shared by every launch of the library on one device (one word per device).
static PerDevice<unsigned*> g_status_words;
static int ensure_status() {
    unsigned*& w = g_status_words.here();
    if (w) return ROTOR_B200_OK;
    RB_CUDA(cudaMalloc(&w, sizeof(unsigned)));
    RB_CUDA(cudaMemset(w, 0, sizeof(unsigned)));
    return ROTOR_B200_OK;
}
unsigned* library_status_word() { return ensure_status() ? nullptr : g_status_words.here(); }
PerDevice<unsigned*> g_extra_status;

int fused_sm_count() {
    static PerDevice<int> counts;
    int& n = counts.here();
    if (!n) {
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, current_device()) != cudaSuccess || n <= 0)
            n = 148;
    }
    return n;
}

__global__ void empty_kernel() {
    pdl_wait();
    pdl_trigger();
}

}  // namespace rb

using namespace rb;

extern "C" {

int rotor_b200_version(void) { return 100; }

unsigned long long rotor_b200_launch_count(void) { return g_launch_count; }

const char* rotor_b200_status_string(int status) {
    switch (status) {
        case ROTOR_B200_OK: return "ok";
        case ROTOR_B200_ERR_ARG: return "invalid argument";
        case ROTOR_B200_ERR_CUDA: return "CUDA error";
        case ROTOR_B200_ERR_SHAPE: return "unsupported shape";
        case ROTOR_B200_ERR_WORKSPACE: return "workspace too small";
        case ROTOR_B200_ERR_TIMEOUT: return "device-side wait timed out";
        case ROTOR_B200_ERR_TOO_LARGE: return "problem exceeds the library's built-in scratch array";
        default: return "unknown status";
    }
}

/* Programmatic dependent launch for the kernels of the decode chain: 1 lets each kernel start
 * (and prefetch its weight tiles) while its predecessor drains.  Applies to later launches and
 * to graphs captured afterwards.  Returns the previous setting. */
int rotor_b200_set_pdl(int enable) {
    const int old = g_use_pdl;
    g_use_pdl = enable ? 1 : 0;
    return old;
}

/* Measurement aid: one launch of a kernel that does nothing, with the same launch attributes
 * (programmatic dependent launch when enabled) as the kernels of the decode chain.  A chain of
 * these in a CUDA graph gives the floor that any chain of dependent launches pays per launch. */
int rotor_b200_launch_empty(void* stream) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(148);
    cfg.blockDim = dim3(128);
    cfg.stream = as_stream(stream);
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = g_use_pdl ? 1 : 0;
    if (cudaLaunchKernelEx(&cfg, rb::empty_kernel) != cudaSuccess) {
        ++g_launch_count;
        return ROTOR_B200_ERR_CUDA;
    }
    return launch_status();
}

/* Reads and clears the status words of the current device that bounded waits write to: the
 * library's own word and the one at the start of the fixed scratch array of
 * rotor_b200_bitlinear_forward_static (once that entry point has run on this device).  Allocates
 * nothing. */
int rotor_b200_device_status(void) {
    unsigned v = 0, vs = 0;
    if (unsigned* w = g_status_words.here()) {
        RB_CUDA(cudaMemcpy(&v, w, sizeof(v), cudaMemcpyDeviceToHost));
        if (v) RB_CUDA(cudaMemset(w, 0, sizeof(v)));
    }
    if (unsigned* a = g_extra_status.here()) {
        RB_CUDA(cudaMemcpy(&vs, a, sizeof(vs), cudaMemcpyDeviceToHost));
        if (vs) RB_CUDA(cudaMemset(a, 0, sizeof(vs)));
    }
    return (int)(v ? v : vs);
}

}  // extern "C"
