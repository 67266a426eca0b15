// Shared declarations of the sm_100a kernels.
//
// Every launcher is an extern "C" function that takes raw device pointers, sizes
// and the CUDA stream, launches on that stream, allocates nothing and returns 0
// or a negative error code (see gl_error_string in the Python wrapper).
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define GL_API extern "C" __attribute__((visibility("default")))

// element types of buffers passed by void*
enum GlDtype { GL_F32 = 0, GL_BF16 = 1 };

// activation applied in an epilogue
enum GlAct { GL_ACT_NONE = 0, GL_ACT_GELU_TANH = 1, GL_ACT_GELU_ERF = 2, GL_ACT_RELU = 3,
             GL_ACT_RELU_SQ = 4,      // max(x, 0)^2
             GL_ACT_SILU = 5,         // x * sigmoid(x)
             GL_ACT_XIELU = 6 };      // two numbers (up, down) come with it: up x^2 + x/2 above zero,
                                      // down (e^x - 1 - x) + x/2 at and below zero

// error codes
enum GlError {
    GL_OK = 0,
    GL_ERR_DTYPE = -1,      // combination of element types not built
    GL_ERR_SHAPE = -2,      // a size the kernel does not take
    GL_ERR_ALIGN = -3,      // a pointer or stride not aligned as required
    GL_ERR_LAUNCH = -4,     // cudaGetLastError() after the launch was not success
    GL_ERR_SMEM = -5,       // shared memory need exceeds the device limit
    GL_ERR_DRIVER = -6,     // a driver entry point could not be obtained or failed
    GL_ERR_SCRATCH = -7,    // the call needs more scratch than a built-in array holds
};

// tokens of the cache that share one page
#define GL_PAGE 64

// Programmatic dependent launch.  A kernel launched through gl_launch may begin while the
// kernel before it in the stream is still finishing: blocks are scheduled and run up to
// gl_grid_wait(), which returns once every kernel it depends on has completed and its writes
// are visible.  Everything a kernel reads from or writes to memory that an earlier kernel
// touches must therefore come after gl_grid_wait(); only constants of the launch (weights,
// barrier set-up) may come before.  gl_grid_launch_dependents() lets the next kernel start
// being scheduled.  Both are no-ops in a kernel launched the ordinary way.
static int gl_pdl = 1;
GL_API void gl_set_pdl(int on) { gl_pdl = on; }

#ifdef __CUDACC__
__device__ __forceinline__ void gl_grid_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void gl_grid_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

template <typename... KArgs, typename... Args>
static int gl_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                     int cluster_x, Args... args);

// The same launch without the early start.  For a long kernel of few blocks: started early, its blocks are
// placed on whichever SMs have room beside the kernel before, several to an SM, and stay there.
template <typename... KArgs, typename... Args>
static int gl_launch_in_order(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args... args) {
    const int keep = gl_pdl;
    gl_pdl = 0;
    const int rc = gl_launch(kernel, grid, block, smem, stream, 1, args...);
    gl_pdl = keep;
    return rc;
}

template <typename... KArgs, typename... Args>
static int gl_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                     int cluster_x, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (gl_pdl) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    if (cluster_x > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = cluster_x;
        attr[n].val.clusterDim.y = 1;
        attr[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    if (cudaLaunchKernelEx(&cfg, kernel, args...) != cudaSuccess) {
        cudaGetLastError();
        return -4;
    }
    return 0;
}
#endif

// A build with -DGL_DEBUG_BOUNDS checks the indices that kernels take from memory (token ids, page
// numbers, positions within a page table) before they use them.  A bad index is recorded (which kind,
// its value, the limit it broke, how many were seen) in a word the host reads, and the access is made at
// index 0 instead: the kernel runs on with a wrong result and an error on record, it never traps and
// never touches memory outside its buffers.  The host checks the same things before a step is launched;
// this is the second net, for an index that a kernel or a caller of the C entry points got wrong.
enum GlBoundsKind { GL_BAD_TOKEN = 1, GL_BAD_PAGE = 2, GL_BAD_POSITION = 3, GL_BAD_ROW = 4 };
#if defined(GL_DEBUG_BOUNDS) && defined(__CUDACC__)
__device__ int gl_bounds_word[4];      // [0] kind of the first bad index (0: none), [1] its value, [2] the limit, [3] how many
__device__ __forceinline__ int gl_checked(int v, int limit, int kind) {
    if ((unsigned)v < (unsigned)limit) return v;
    if (atomicCAS(&gl_bounds_word[0], 0, kind) == 0) { gl_bounds_word[1] = v; gl_bounds_word[2] = limit; }
    atomicAdd(&gl_bounds_word[3], 1);
    return 0;
}
// out4 receives the four words; clear sets them back to zero.  -1 if they could not be read.
GL_API int gl_bounds_status(int* out4, int clear) {
    if (cudaMemcpyFromSymbol(out4, gl_bounds_word, 4 * sizeof(int)) != cudaSuccess) return -1;
    if (clear && out4[0] != 0) {
        const int zero[4] = {0, 0, 0, 0};
        if (cudaMemcpyToSymbol(gl_bounds_word, zero, sizeof(zero)) != cudaSuccess) return -1;
    }
    return 0;
}
#else
#define gl_checked(v, limit, kind) (v)
#endif

#ifdef __CUDACC__
// The first position whose key a query at position p sees (it sees that one to p): all of them, the last ``window``
// positions, or, with chunk > 0, the positions of its own chunk, chunks of that many positions counted from a
// sequence's start.  Never decreases with p.
__device__ __forceinline__ int gl_first_key(int p, int window, int chunk) {
    if (chunk > 0) return p - p % chunk;
    return (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
}
#endif

static inline int gl_check_launch() {
    return cudaGetLastError() == cudaSuccess ? GL_OK : GL_ERR_LAUNCH;
}

__device__ __forceinline__ float gl_load(const float* p) { return *p; }
__device__ __forceinline__ float gl_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void gl_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void gl_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float gl_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float gl_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Activations in 32-bit.  gelu "tanh form" is x*sigmoid(2*sqrt(2/pi)*(x+0.044715x^3)),
// the form the reference evaluates (fastmath.go:138-141); the erf form is
// 0.5*x*(1+erf(x/sqrt(2))) (bert.go:742-744).
// For results that are rounded to bfloat16 right away: the tanh form through the hardware's
// tanh.approx (relative error about 2^-11, below bfloat16's 2^-9 rounding).
__device__ __forceinline__ float gl_activate_bf16_grade(float x, int act) {
    if (act == GL_ACT_GELU_TANH) {
        float th;
        const float u = 0.7978845608028654f * x * fmaf(0.044715f * x, x, 1.0f);
        asm("tanh.approx.f32 %0, %1;" : "=f"(th) : "f"(u));
        const float hx = 0.5f * x;
        return fmaf(hx, th, hx);
    }
    if (act == GL_ACT_GELU_ERF) return 0.5f * x * (1.0f + erff(x * 0.70710678118654752440f));
    if (act == GL_ACT_RELU) return fmaxf(x, 0.0f);
    if (act == GL_ACT_RELU_SQ) { const float r = fmaxf(x, 0.0f); return r * r; }
    if (act == GL_ACT_SILU) return x / (1.0f + __expf(-x));
    return x;
}

// the activation with two numbers of its own (the same slope on both sides of zero)
template <bool EXACT>
__device__ __forceinline__ float gl_xielu(float x, float up, float down) {
    if (EXACT) {
        if (x > 0.f) return fmaf(up * x, x, 0.5f * x);
        return fmaf(down, expm1f(x) - x, 0.5f * x);
    }
    // for results that are rounded to 16 bits right away: down e^x - down + (1/2 - down) x, four operations and no
    // branch (what the difference of the first two terms loses near zero is 2^-22 of ``down``, far below the rounding)
    const float pos = x * fmaf(up, x, 0.5f);
    const float neg = fmaf(down, __expf(x), fmaf(0.5f - down, x, -down));
    return x > 0.f ? pos : neg;
}

template <bool EXACT>
__device__ __forceinline__ float gl_activate(float x, int act) {
    switch (act) {
        case GL_ACT_GELU_TANH: {
            const float z = 1.5957691216057308f * (x + 0.044715f * x * x * x);
            const float e = EXACT ? expf(-z) : __expf(-z);
            return x / (1.0f + e);
        }
        case GL_ACT_GELU_ERF:
            return 0.5f * x * (1.0f + erff(x * 0.70710678118654752440f));
        case GL_ACT_RELU:
            return fmaxf(x, 0.0f);
        case GL_ACT_RELU_SQ: {
            const float r = fmaxf(x, 0.0f);
            return r * r;
        }
        case GL_ACT_SILU:
            return x / (1.0f + (EXACT ? expf(-x) : __expf(-x)));
        default:
            return x;
    }
}

// A gated feed-forward's inner value from its gate and its up projection: act(gate) * up, or with GL_GATED_CLIPPED (a
// sigmoid-weighted gate with both sides clipped: numbers limit, slope, shift)
//   g = min(gate, limit), u = clamp(up, -limit, limit):   g * sigmoid(slope * g) * (u + shift).
#define GL_GATED_CLIPPED 32
struct GlGated { int act; float limit, slope, shift; };
template <bool EXACT>
__device__ __forceinline__ float gl_gated(float g, float u, const GlGated& p) {
    if (p.act != GL_GATED_CLIPPED) return gl_activate<EXACT>(g, p.act) * u;
    g = fminf(g, p.limit);
    u = fminf(fmaxf(u, -p.limit), p.limit);
    if (EXACT) return g / (1.0f + expf(-p.slope * g)) * (u + p.shift);
    return __fdividef(g, 1.0f + __expf(-p.slope * g)) * (u + p.shift);       // for results that are rounded to 16 bits right away
}

// the same for callers that carry an activation's own numbers along
template <bool EXACT>
__device__ __forceinline__ float gl_activate(float x, int act, float p0, float p1) {
    return act == GL_ACT_XIELU ? gl_xielu<EXACT>(x, p0, p1) : gl_activate<EXACT>(x, act);
}
__device__ __forceinline__ float gl_activate_bf16_grade(float x, int act, float p0, float p1) {
    return act == GL_ACT_XIELU ? gl_xielu<false>(x, p0, p1) : gl_activate_bf16_grade(x, act);
}
