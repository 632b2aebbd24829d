// CUDA-core GEMM behind the same descriptor as gemm_tcgen05.cu: Y[b][t][n] = sum_k X[b][t][k] * W[b][n][k], optional second
// weight (act(X W^T) * (X W2^T)) or a function of the single product, optional residual, optional expert segments.
//
// Two uses: fp32 operands in true 32-bit arithmetic (the tensor cores have no such mode), and bf16 operands whose rows are
// not 16-byte multiples, which TMA cannot address.  A plain 64 x 64 tile with 4 x 4 results per thread.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "jib_kernels.h"
#include "pdl.cuh"

namespace {

typedef __nv_bfloat16 bf16;
constexpr int TM = 64, TN = 64, TK = 16, NT = 256, PAD = 4;

__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
// act(z) = z * sigmoid(gate_arg(z)): 0.5 (1 + tanh(u)) is sigmoid(2 u)
__device__ __forceinline__ float gate_arg(float z, int act) {
    return act == JIB_ACT_GELU_TANH ? 1.5957691216057308f * (z + 0.044715f * z * z * z) : z;
}

__device__ __forceinline__ float unary(float v, const jib_gemm_desc & d, long long row) {
    if (d.unary == JIB_UNARY_GELU) {
        if (d.row_scale != nullptr) v *= d.row_scale[row];
        return 0.5f * v * (1.f + erff(v * 0.70710678118654752f));
    }
    if (d.unary == JIB_UNARY_NONE) return v;
    if (d.unary == JIB_UNARY_RELU2) return v > 0.f ? v * v : 0.f;
    v *= d.scale;
    return d.softcap > 0.f ? d.softcap * tanhf(v / d.softcap) : v;
}

template <typename T, bool DUAL>
__global__ void __launch_bounds__(NT) gemm_simt_kernel(const jib_gemm_desc d) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    __shared__ float xs[TK][TM + PAD], ws[TK][TN + PAD], us[DUAL ? TK : 1][TN + PAD];
    const int batch = blockIdx.z;
    const int n0 = blockIdx.x * TN;
    long long row_base = 0, rows = d.T;
    if (d.seg != nullptr) {
        row_base = d.seg[batch];
        rows = d.seg[batch + 1] - row_base;
    }
    const int t0 = blockIdx.y * TM;
    if (t0 >= rows) return;
    const T * x = (const T *) d.x + (d.seg != nullptr ? 0 : (long long) batch * d.x_batch_stride) + row_base * d.x_row_stride;
    const T * w = (const T *) d.w + (long long) batch * d.w_batch_stride;
    const T * u = DUAL ? (const T *) d.w2 + (long long) batch * d.w_batch_stride : nullptr;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {}, acu[4][4] = {};
    for (int k0 = 0; k0 < d.K; k0 += TK) {
#pragma unroll
        for (int i = 0; i < TM * TK / NT; ++i) {
            const int e = threadIdx.x + i * NT, r = e / TK, kk = e % TK, k = k0 + kk;
            xs[kk][r] = (t0 + r < rows && k < d.K) ? to_f(x[(long long) (t0 + r) * d.x_row_stride + k]) : 0.f;
            const bool in = n0 + r < d.N && k < d.K;
            ws[kk][r] = in ? to_f(w[(long long) (n0 + r) * d.w_row_stride + k]) : 0.f;
            if (DUAL) us[kk][r] = in ? to_f(u[(long long) (n0 + r) * d.w_row_stride + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < TK; ++kk) {
            float a[4], b[4], c[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = xs[kk][ty + 16 * i];
                b[i] = ws[kk][tx + 16 * i];
                if (DUAL) c[i] = us[kk][tx + 16 * i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] += a[i] * b[j];
                    if (DUAL) acu[i][j] += a[i] * c[j];
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const long long t = t0 + ty + 16 * i;
        if (t >= rows) continue;
        const long long row = row_base + t;
        if (d.seg != nullptr && row >= d.x_rows_total) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx + 16 * j;
            if (n >= d.N) continue;
            float y = DUAL ? acc[i][j] / (1.f + expf(-gate_arg(acc[i][j], d.act))) * acu[i][j] : unary(acc[i][j], d, row);
            if (d.residual != nullptr) {
                const long long ri = (long long) batch * d.res_batch_stride + row * d.ldr + n;
                y += d.res_f32 ? ((const float *) d.residual)[ri] : to_f(((const bf16 *) d.residual)[ri]);
            }
            const long long oi = (long long) batch * d.out_batch_stride + row * d.ldo + n;
            if (d.out_f32) ((float *) d.out)[oi] = y;
            else ((bf16 *) d.out)[oi] = __float2bfloat16(y);
        }
    }
}

}  // namespace

// f32: x, w, w2 and out are fp32 (d->out_f32 must be set).  Fused collectives, row pointers and expert lists are not supported.
extern "C" JIB_EXPORT int jib_gemm_simt(const jib_gemm_desc * d, int f32, void * stream) {
    if (d->T <= 0 || d->N <= 0 || d->K <= 0) return 0;
    if (d->ar != nullptr || d->ag_flags != nullptr || d->out_row_ptr != nullptr || d->src_token != nullptr || (f32 && !d->out_f32))
        return JIB_E_ARG;
    const int batch = d->batch > 0 ? d->batch : 1;
    const int rows = d->seg != nullptr && d->max_rows > 0 ? d->max_rows : d->T;
    const dim3 grid((d->N + TN - 1) / TN, (rows + TM - 1) / TM, batch);
    cudaStream_t s = (cudaStream_t) stream;
    if (grid.y > 65535 || grid.z > 65535) return JIB_E_ARG;
    if (f32) {
        if (d->w2 != nullptr) JIB_LAUNCH((gemm_simt_kernel<float, true>), grid, NT, 0, s, *d);
        else JIB_LAUNCH((gemm_simt_kernel<float, false>), grid, NT, 0, s, *d);
    } else {
        if (d->w2 != nullptr) JIB_LAUNCH((gemm_simt_kernel<bf16, true>), grid, NT, 0, s, *d);
        else JIB_LAUNCH((gemm_simt_kernel<bf16, false>), grid, NT, 0, s, *d);
    }
    return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH;
}
