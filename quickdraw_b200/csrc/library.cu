// Entry points every library of this package exports: version, error text, the chained-launch switch.
#include "common.cuh"

extern "C" int qd_version(void) { return 1; }

extern "C" const char* qd_error_string(int code) {
    switch (code) {
        case QD_OK: return "ok";
        case QD_ERR_ARG: return "invalid argument";
        case QD_ERR_LAUNCH: return "CUDA launch failed";
        case QD_ERR_TIMEOUT: return "bounded device wait ran out";
        case QD_ERR_UNSUPPORTED: return "shape not covered by this kernel";
        case QD_ERR_TOO_LARGE: return "shape exceeds the fixed capacity of a built-in buffer";
        default: return "unknown";
    }
}

// Kernels of the chunk and batch paths open with a wait for the kernel before them and are launched as
// its programmatic dependents, so that their launch overlaps its last blocks.  on = 0 launches them
// ordinarily (measured faster inside a captured graph, whose edges are cheaper than the overlap gains;
// the few-row products stay dependents of their conversion kernels either way).  Returns the old setting.
extern "C" int qd_set_chained_launches(int on) {
    int& current = qd_chain_switch();
    const int before = current;
    current = on != 0;
    return before;
}

