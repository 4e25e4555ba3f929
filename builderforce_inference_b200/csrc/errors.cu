// Error reporting shared by every exported function of one library.
#include "common.cuh"

static thread_local char g_error[1024] = "";

extern "C" const char* bfi_last_error() { return g_error; }

int bfi_fail(const char* fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_error, sizeof(g_error), fmt, ap);
    va_end(ap);
    return 1;
}

int bfi_check_launch(const char* what) {
    cudaError_t e = cudaPeekAtLastError();
    if (e != cudaSuccess) {
        cudaGetLastError();
        return bfi_fail("%s: launch failed: %s", what, cudaGetErrorString(e));
    }
    return 0;
}

// Off unless asked for: measured on the decode step, early launch of dependents did not pay.
int g_bfi_pdl = 1;

// Turns programmatic dependent launch on (1) or off (0) for every later launch of this library.
extern "C" int bfi_set_pdl(int on) {
    g_bfi_pdl = on ? 1 : 0;
    return 0;
}

// The constants of the gated epilogue for the products this host thread launches from now on.
thread_local GateAct g_bfi_gate = {1.0f, 0.0f, 0.0f, BFI_GATE_SIGMOID, nullptr, 0, 1};

extern "C" int bfi_set_gate(float alpha, float limit, float shift) {
    g_bfi_gate.alpha = alpha, g_bfi_gate.limit = limit, g_bfi_gate.shift = shift;
    g_bfi_gate.kind = BFI_GATE_SIGMOID;
    return 0;
}

// The same, naming the activation's kind (BFI_GATE_*) as well.
extern "C" int bfi_set_gate_kind(int kind, float alpha, float limit, float shift) {
    if (kind != BFI_GATE_SIGMOID && kind != BFI_GATE_GELU_TANH) return bfi_fail("set_gate_kind: unknown activation kind %d", kind);
    g_bfi_gate.alpha = alpha, g_bfi_gate.limit = limit, g_bfi_gate.shift = shift;
    g_bfi_gate.kind = kind;
    return 0;
}

// The factors on the gated products' inputs (null: none), for the products launched from now on.
extern "C" int bfi_set_gate_in_scale(const float* scale, long stride, int cols) {
    if (scale != nullptr && (cols < 1 || stride < 1)) return bfi_fail("set_gate_in_scale: bad sizes cols=%d stride=%ld", cols, stride);
    g_bfi_gate.in_scale = scale, g_bfi_gate.in_stride = stride, g_bfi_gate.in_cols = cols;
    return 0;
}

// Multiprocessors of the current device, asked of the driver once per device: launchers size
// their grids and work splits by it instead of by a constant.
int bfi_sm_count() {
    static int cached[64] = {0};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
    if (cached[dev] == 0) {
        int n = 0;
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) {
            cudaGetLastError();
            n = 148;      // no device to ask (a build check without a GPU): a B200's count
        }
        cached[dev] = n;
    }
    return cached[dev];
}

extern "C" int bfi_device_sm_count() { return bfi_sm_count(); }

// Identifies the build: the architecture the device code was compiled for.
extern "C" const char* bfi_build_arch() { return "sm_100a"; }
