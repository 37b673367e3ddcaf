// The gated activation of a dense feed-forward after a library product: x [rows, 2n] = [gate | up] -> out [rows, n], in
// 32-bit, rounded once (glu.cuh says which activations).  Eight elements at a time where width and addresses allow it.
#include "common.cuh"
#include "glu.cuh"

namespace se {

template <typename T>
__global__ void __launch_bounds__(256)
glu_kernel(const T* x, T* out, size_t items, int chunks, int width, int kind, float limit, float alpha) {
    grid_dependency_trigger();
    grid_dependency_wait();
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (size_t k = (size_t)blockIdx.x * blockDim.x + threadIdx.x; k < items; k += stride) {
        const size_t t = k / chunks;
        const int c = (int)(k - t * chunks);
        if (chunks != width) {
            float g[8], u[8];
            load8(x + t * 2 * width + c * 8, g);
            load8(x + t * 2 * width + width + c * 8, u);
#pragma unroll
            for (int j = 0; j < 8; ++j) g[j] = glu_value<T>(g[j], u[j], kind, limit, alpha);
            store8(out + t * width + c * 8, g);
        } else {
            out[t * width + c] = from_float<T>(glu_value<T>(to_float(x[t * 2 * width + c]), to_float(x[t * 2 * width + width + c]), kind, limit, alpha));
        }
    }
}

}  // namespace se

extern "C" int se_glu(const void* x, void* out, int rows, int width, int kind, float limit, float alpha, int dtype, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (width <= 0 || kind < SE_GLU_SILU || kind > SE_GLU_GELU) return SE_ERR_ARGUMENT;
    const bool vec = width % 8 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    const int chunks = vec ? width / 8 : width;        // chunks == width: element by element (a width of at least 8 has fewer chunks)
    const size_t items = (size_t)rows * chunks;
    const int blocks = (int)((items + 255) / 256 < 148 * 16 ? (items + 255) / 256 : 148 * 16);
    SE_DISPATCH_DTYPE(dtype, T, {
        cudaError_t e = SE_LAUNCH_DEPENDENT("act", se::glu_kernel<T>, dim3(blocks), dim3(256), 0, stream, (const T*)x, (T*)out, items,
                                             chunks, width, kind, limit, alpha);
        if (e != cudaSuccess) return (int)e;
    });
    SE_LAUNCH_CHECK();
}
