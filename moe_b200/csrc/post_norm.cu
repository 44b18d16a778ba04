// The end of a sublayer whose OUTPUT is normed before it joins the stream, in one kernel:
//
//   y = what the sublayer left: a[r] sa + b[r] sb (b may be null; sa, sb constants), or routed experts' outputs before
//       their combine, sum_j w[r, j] e[pos[r, j]] + shared[r] (w null: weights of 1)
//   v = x[r] + y / sqrt(mean(y^2) + post_eps) * post_w;   if write_back: x[r] = v      (the 32-bit residual stream)
//   out = v, or with w: v / sqrt(mean(v^2) + eps) * w (the norm that comes next, if there is one);  out32[i], out16[i] = bf16(out)
//
// One block per output row i; source row r = rows ? rows[i] : i.  Everything is 32-bit; only out16 is rounded.  With x
// alone (no y) the row is passed on, or normed, as it is.
#include "common.cuh"

namespace {

struct PostNorm {
    float* x;
    const int* rows;
    int num_src_rows;
    const float* a;            // null, with e null: nothing is added
    const float* b;
    float sa, sb;
    const float* e;            // [pairs, hidden]
    const int* pos;            // [T, top_k], -1: no expert
    const float* ew;           // [T, top_k] or null
    const float* shared;       // [T, hidden] or null
    int top_k;
    const float* post_w;
    float post_eps;
    const float* w;
    float eps;
    float* out32;
    __nv_bfloat16* out16;
    int hidden, write_back;
    int* status;
};

__device__ __forceinline__ float4 fma4(float s, float4 v, float4 acc) {
    return make_float4(fmaf(s, v.x, acc.x), fmaf(s, v.y, acc.y), fmaf(s, v.z, acc.z), fmaf(s, v.w, acc.w));
}
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float sq4(float4 v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))); }

__device__ __forceinline__ int source_row(const PostNorm& p, int i) {
    int r = p.rows ? p.rows[i] : i;
    if (r < 0 || r >= p.num_src_rows) {
        if (threadIdx.x == 0 && p.status) atomicOr(p.status, ST_BAD_ROW);
        r = 0;
    }
    return r;
}

// NV: 16-byte units a thread; the row stays in registers.
template <int NV>
__global__ void __launch_bounds__(512)
post_norm_vec_kernel(const PostNorm p) {
    __shared__ float red[32];
    const int units = p.hidden / 4, H = p.hidden;
    float4 pw[NV];                                    // (weights do not depend on the predecessor)
#pragma unroll
    for (int u = 0; u < NV; u++) {
        const int j = threadIdx.x + u * blockDim.x;
        pw[u] = (p.post_w && j < units) ? ld4(p.post_w + 4 * j) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_sync();
    const int r = source_row(p, blockIdx.x);
    float* xr = p.x + (size_t)r * H;
    float4 v[NV], y[NV];
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < NV; u++) {
        const int j = threadIdx.x + u * blockDim.x;
        y[u] = v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j >= units) continue;
        v[u] = ld4(xr + 4 * j);
        if (p.e) {
            for (int q = 0; q < p.top_k; q++) {
                const int at = p.pos[(size_t)r * p.top_k + q];
                if (at >= 0) y[u] = fma4(p.ew ? p.ew[(size_t)r * p.top_k + q] : 1.f, ld4(p.e + (size_t)at * H + 4 * j), y[u]);
            }
            if (p.shared) y[u] = fma4(1.f, ld4(p.shared + (size_t)r * H + 4 * j), y[u]);
        } else if (p.a) {
            y[u] = fma4(p.sa, ld4(p.a + (size_t)r * H + 4 * j), y[u]);
            if (p.b) y[u] = fma4(p.sb, ld4(p.b + (size_t)r * H + 4 * j), y[u]);
        }
        ss += sq4(y[u]);
    }
    if (p.post_w) {
        const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)H + p.post_eps);
#pragma unroll
        for (int u = 0; u < NV; u++) {
            const int j = threadIdx.x + u * blockDim.x;
            if (j >= units) continue;
            v[u].x = fmaf(y[u].x * inv, pw[u].x, v[u].x), v[u].y = fmaf(y[u].y * inv, pw[u].y, v[u].y);
            v[u].z = fmaf(y[u].z * inv, pw[u].z, v[u].z), v[u].w = fmaf(y[u].w * inv, pw[u].w, v[u].w);
            if (p.write_back) *reinterpret_cast<float4*>(xr + 4 * j) = v[u];
        }
    }
    float inv2 = 1.f;
    if (p.w) {
        ss = 0.f;
#pragma unroll
        for (int u = 0; u < NV; u++) ss += sq4(v[u]);
        inv2 = 1.0f / sqrtf(block_sum(ss, red) / (float)H + p.eps);
    }
#pragma unroll
    for (int u = 0; u < NV; u++) {
        const int j = threadIdx.x + u * blockDim.x;
        if (j >= units) continue;
        float4 o = v[u];
        if (p.w) {
            const float4 g = ld4(p.w + 4 * j);
            o = make_float4(o.x * inv2 * g.x, o.y * inv2 * g.y, o.z * inv2 * g.z, o.w * inv2 * g.w);
        }
        if (p.out32) *reinterpret_cast<float4*>(p.out32 + (size_t)blockIdx.x * H + 4 * j) = o;
        if (p.out16) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(o.x, o.y), hi = __floats2bfloat162_rn(o.z, o.w);
            uint2 w2;
            w2.x = *reinterpret_cast<const unsigned*>(&lo), w2.y = *reinterpret_cast<const unsigned*>(&hi);
            *reinterpret_cast<uint2*>(p.out16 + (size_t)blockIdx.x * H + 4 * j) = w2;
        }
    }
}

// Any width and alignment: the row in shared memory.
__global__ void __launch_bounds__(256)
post_norm_kernel(const PostNorm p) {
    extern __shared__ float pn_row[];
    __shared__ float red[32];
    const int H = p.hidden;
    pdl_sync();
    const int r = source_row(p, blockIdx.x);
    float* xr = p.x + (size_t)r * H;
    float ss = 0.f;
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
        float y = 0.f;
        if (p.e) {
            for (int q = 0; q < p.top_k; q++) {
                const int at = p.pos[(size_t)r * p.top_k + q];
                if (at >= 0) y = fmaf(p.ew ? p.ew[(size_t)r * p.top_k + q] : 1.f, p.e[(size_t)at * H + j], y);
            }
            if (p.shared) y += p.shared[(size_t)r * H + j];
        } else if (p.a) {
            y = p.sa * p.a[(size_t)r * H + j];
            if (p.b) y = fmaf(p.sb, p.b[(size_t)r * H + j], y);
        }
        pn_row[j] = y;
        ss = fmaf(y, y, ss);
    }
    const float inv = p.post_w ? 1.0f / sqrtf(block_sum(ss, red) / (float)H + p.post_eps) : 0.f;
    ss = 0.f;
    for (int j = threadIdx.x; j < H; j += blockDim.x) {           // (a thread's own entries)
        const float v = p.post_w ? fmaf(pn_row[j] * inv, p.post_w[j], xr[j]) : xr[j];
        if (p.post_w && p.write_back) xr[j] = v;
        pn_row[j] = v;
        ss = fmaf(v, v, ss);
    }
    const float inv2 = p.w ? 1.0f / sqrtf(block_sum(ss, red) / (float)H + p.eps) : 1.f;
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
        const float o = p.w ? pn_row[j] * inv2 * p.w[j] : pn_row[j];
        if (p.out32) p.out32[(size_t)blockIdx.x * H + j] = o;
        if (p.out16) p.out16[(size_t)blockIdx.x * H + j] = __float2bfloat16_rn(o);
    }
}

}  // namespace

// x: [num_src_rows, hidden].  Either a (and b) or e with pos, or neither (then post_w is null and x is passed on).
MOE_API int moe_post_norm(float* x, const float* a, float sa, const float* b, float sb, const float* e, const int* pos,
                          const float* ew, int top_k, const float* shared, const float* post_w, float post_eps,
                          const float* w, float eps, const int* rows, float* out32, void* out16, int num_out_rows,
                          int num_src_rows, int hidden, int write_back, int* status, cudaStream_t stream) {
    if (num_out_rows <= 0) return 0;
    if (!x || hidden <= 0 || (a && e) || (b && !a) || (e && (!pos || top_k <= 0)) || ((a || e) != (post_w != nullptr)) ||
        (rows && write_back))
        return (int)cudaErrorInvalidValue;
    const PostNorm p{x, rows, num_src_rows, a, b, sa, sb, e, pos, ew, shared, top_k, post_w, post_eps, w, eps,
                     out32, (__nv_bfloat16*)out16, hidden, write_back, status};
    auto al = [](const void* q, size_t n) { return ((uintptr_t)q % n) == 0; };
    const bool vec = hidden % 4 == 0 && al(x, 16) && al(a, 16) && al(b, 16) && al(e, 16) && al(shared, 16) && al(post_w, 16) &&
                     al(w, 16) && al(out32, 16) && al(out16, 8);
    const int units = hidden / 4;
    if (vec && units <= 512 * 8) {
        const int threads = units >= 512 ? 512 : units >= 256 ? 256 : units >= 128 ? 128 : 64;
        const int nv = (units + threads - 1) / threads;
#define POST(NV_) return launch_pdl(post_norm_vec_kernel<NV_>, dim3(num_out_rows), threads, 0, stream, p)
        if (nv <= 1) POST(1);
        if (nv <= 2) POST(2);
        if (nv <= 4) POST(4);
        POST(8);
#undef POST
    }
    const size_t smem = (size_t)hidden * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    if (smem > 48 * 1024) {
        const cudaError_t err = cudaFuncSetAttribute(post_norm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (err != cudaSuccess) return (int)err;
    }
    return launch_pdl(post_norm_kernel, dim3(num_out_rows), 256, smem, stream, p);
}
