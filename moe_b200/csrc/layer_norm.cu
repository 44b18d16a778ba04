// Layer norm of the residual stream with the residual add in front of it:
//   v = x (+ delta), stored back into x;   y = (v - mean) / sqrt(mean((v - mean)^2) + eps) * w (+ b)
// The row stays in registers (or, for very wide rows, in shared memory) between the two sums, so that the
// deviations are formed from the mean itself and not as a difference of two large sums.  All arithmetic
// is 32-bit; only the optional second output is rounded to bfloat16.
#include "common.cuh"

namespace {

// One block per output row i; source row r = rows ? rows[i] : i.  UNITS: 16-byte units of the row a thread
// holds in registers (0: any width, the row in shared memory, element by element).
template <int UNITS>
__global__ void __launch_bounds__(512)
layernorm_kernel(float* __restrict__ x, const float* __restrict__ delta, const float* __restrict__ w,
                 const float* __restrict__ b, const int* __restrict__ rows, float* __restrict__ out32,
                 __nv_bfloat16* __restrict__ out16, int hidden, float eps, int write_back, int num_src_rows, int* status) {
    extern __shared__ float ln_row[];
    __shared__ float red_mean[32], red_var[32];
    const int i = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    constexpr int U = UNITS > 0 ? UNITS : 1;
    const int units = hidden / 4;
    float4 v[U], nwt[U];
    if (UNITS > 0) {      // the weight does not come from the predecessor
#pragma unroll
        for (int u = 0; u < U; u++) {
            const int j = threadIdx.x + u * blockDim.x;
            nwt[u] = j < units ? reinterpret_cast<const float4*>(w)[j] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    pdl_sync();
    int r = rows ? rows[i] : i;
    if (r < 0 || r >= num_src_rows) {
        if (threadIdx.x == 0) atomicOr(status, ST_BAD_ROW);
        r = 0;
    }
    float* xr = x + (size_t)r * hidden;
    const float* dr = delta ? delta + (size_t)r * hidden : nullptr;
    // the block's sum of one number a thread, the same to the bit in every thread
    auto total = [&](float s, float* red) {
        s = warp_sum(s);
        if (lane == 0) red[warp] = s;
        __syncthreads();
        return warp_sum(lane < nw ? red[lane] : 0.f);
    };
    float s = 0.f;
    if (UNITS > 0) {
#pragma unroll
        for (int u = 0; u < U; u++) {
            const int j = threadIdx.x + u * blockDim.x;
            v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (j < units) {
                v[u] = reinterpret_cast<const float4*>(xr)[j];
                if (dr) {
                    const float4 d = reinterpret_cast<const float4*>(dr)[j];
                    v[u].x += d.x, v[u].y += d.y, v[u].z += d.z, v[u].w += d.w;
                }
            }
            s += (v[u].x + v[u].y) + (v[u].z + v[u].w);
        }
    } else {
        for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
            float e = xr[j];
            if (dr) {
                e += dr[j];
                if (write_back) xr[j] = e;
            }
            ln_row[j] = e;
            s += e;
        }
    }
    const float mean = total(s, red_mean) / (float)hidden;
    float ss = 0.f;
    if (UNITS > 0) {
#pragma unroll
        for (int u = 0; u < U; u++) {
            const int j = threadIdx.x + u * blockDim.x;
            if (j < units) {
                if (dr && write_back) reinterpret_cast<float4*>(xr)[j] = v[u];
                v[u].x -= mean, v[u].y -= mean, v[u].z -= mean, v[u].w -= mean;
                ss += v[u].x * v[u].x, ss += v[u].y * v[u].y, ss += v[u].z * v[u].z, ss += v[u].w * v[u].w;
            }
        }
    } else {
        for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
            const float e = ln_row[j] - mean;
            ss += e * e;
        }
    }
    const float scale = 1.0f / sqrtf(total(ss, red_var) / (float)hidden + eps);
    if (UNITS > 0) {
#pragma unroll
        for (int u = 0; u < U; u++) {
            const int j = threadIdx.x + u * blockDim.x;
            if (j >= units) continue;
            float4 y = make_float4(v[u].x * scale * nwt[u].x, v[u].y * scale * nwt[u].y, v[u].z * scale * nwt[u].z,
                                   v[u].w * scale * nwt[u].w);
            if (b) {
                const float4 c = reinterpret_cast<const float4*>(b)[j];
                y.x += c.x, y.y += c.y, y.z += c.z, y.w += c.w;
            }
            if (out32) reinterpret_cast<float4*>(out32 + (size_t)i * hidden)[j] = y;
            if (out16) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(y.x, y.y), hi = __floats2bfloat162_rn(y.z, y.w);
                uint2 p;
                p.x = *reinterpret_cast<unsigned*>(&lo), p.y = *reinterpret_cast<unsigned*>(&hi);
                reinterpret_cast<uint2*>(out16 + (size_t)i * hidden)[j] = p;
            }
        }
    } else {
        for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
            float y = (ln_row[j] - mean) * scale * w[j];
            if (b) y += b[j];
            if (out32) out32[(size_t)i * hidden + j] = y;
            if (out16) out16[(size_t)i * hidden + j] = __float2bfloat16_rn(y);
        }
    }
}

}  // namespace

// x, delta: [num_src_rows, hidden]; w, b (may be null): [hidden]; out32 / out16: [num_out_rows, hidden] or null.
MOE_API int moe_layernorm(float* x, const float* delta, const float* w, const float* b, const int* rows, float* out32,
                          void* out16, int num_out_rows, int num_src_rows, int hidden, float eps, int write_back,
                          int* status, cudaStream_t stream) {
    if (num_out_rows <= 0) return 0;
    if (!x || !w || hidden <= 0 || (size_t)hidden * sizeof(float) > 200 * 1024) return (int)cudaErrorInvalidValue;
    const bool vec = hidden % 4 == 0 && (((uintptr_t)x | (uintptr_t)delta | (uintptr_t)w | (uintptr_t)b | (uintptr_t)out32) % 16) == 0 &&
                     (uintptr_t)out16 % 8 == 0 && hidden <= 4 * 4 * 512;
    const int units = (hidden + 3) / 4;
#define LN(U_, THREADS_, SMEM_)                                                                                       \
    return launch_pdl(layernorm_kernel<U_>, dim3(num_out_rows), dim3(THREADS_), (size_t)(SMEM_), stream, x, delta, w, b, rows, \
                      out32, (__nv_bfloat16*)out16, hidden, eps, write_back, num_src_rows, status)
    auto warps = [](int n) { return ((n + 31) / 32) * 32; };
    if (vec) {
        if (units <= 256) LN(1, warps(units), 0);
        if (units <= 1024) LN(2, warps((units + 1) / 2), 0);
        LN(4, warps((units + 3) / 4), 0);
    }
    const size_t smem = (size_t)hidden * sizeof(float);
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(layernorm_kernel<0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    LN(0, hidden >= 1024 ? 512 : 128, smem);
#undef LN
}
