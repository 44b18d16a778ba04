// Kernels around two kinds of attention layer that need more than a rotation and a split:
//
// LATENT attention.  A layer projects its input to queries (heads of d) and to ONE small latent c of
// r numbers per position; a head's keys and values are W_uk_h c and W_uv_h c.  Since
//     q_h . (W_uk_h c) = (W_uk_h^T q_h) . c        and        sum_j p_j W_uv_h c_j = W_uv_h (sum_j p_j c_j),
// the attention itself runs over the cached latents alone: every query head reads the same single
// record c as key AND as value, with queries W_uk_h^T q_h of r numbers, and the head's values are
// formed from the r numbers that come out.  The two per-head products are grouped products (a group
// a head) over rows laid out head by head, hence the transposes here.  A head may have a ROTATED part of
// `rot` dimensions beside the d: its key is one vector per position that all heads share and follows
// the latent in the record, [c | rotated key part], and a query is [W_uk_h^T q_h | rotated query part].
//   latent_prepare    KEYS: from the 32-bit projection row, c = x / sqrt(mean(x^2) + eps) * w over the
//                     latent, then the key part after it rotated by the token's position, written as the
//                     step's key record of width D >= r + rot (zero-filled) and, optionally, appended to the
//                     paged cache; the same norm over a latent of the queries, if they have one, rounded
//                     to the activation dtype for the product that follows.
//                     QUERIES: from 32-bit rows of heads [unrotated | rot], the rotation and the layout: token
//                     by token as records q[t][h][0..D) (zero-filled), or the unrotated part head by head,
//                     q_t[h][t][0..d), with the rotated part put into the records' columns from r on.
//                     Either half may be left out.
//   heads_transpose   dst[b][a][0..wd) = src[a][b][0..n) (zero-filled beyond n), any of the two
//                     storage types on either side, optionally times sigmoid(gate[b][a]).
// The rotation turns pairs (i, i + rot/2) or, interleaved, (2i, 2i + 1) by pos * freq[i], cos and sin times
// a factor.
//
// DIFFERENTIAL attention.  Every head runs two softmax attentions ("maps") over the same values and
// joins them:  o = a1 - lambda a2;  o <- o / sqrt(mean(o^2) + eps) * mult;  o <- o * sigmoid(g_h),
// one gate logit a head.  The maps come as heads of their own (map 1 of all heads, then map 2).
//   diff_combine      out[t, h * dv + j] from ctx[t, h, j] and ctx[t, nh + h, j].
//
//   add_row           x[t, :] += delta[t, :] + row[:]   (a learned vector added to every token's
//                     stream, with whatever was still pending; 32-bit)
// Norms, the difference and the gate are 32-bit; only stores round to the activation dtype.
#include "common.cuh"

namespace {

struct LatentCommit {
    void* k_cache;            // null: no append
    void* v_cache;            // may equal k_cache (the values are the keys)
    const int* seq_end;
    const int* slots;
    const int* tables;
    int table_stride, ring, page_size, num_pages;
};

// four consecutive elements at once (the pointer is aligned to four elements)
__device__ __forceinline__ void ld4(const float* p, float* v) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
}
__device__ __forceinline__ void ld4(const __nv_bfloat16* p, float* v) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(x.x << 16), v[1] = __uint_as_float(x.x & 0xffff0000u);
    v[2] = __uint_as_float(x.y << 16), v[3] = __uint_as_float(x.y & 0xffff0000u);
}
__device__ __forceinline__ void st4(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void st4(__nv_bfloat16* p, const float* v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 x;
    x.x = *reinterpret_cast<const unsigned*>(&a), x.y = *reinterpret_cast<const unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = x;
}

constexpr int LATENT_MAX_ROT = 512;

struct LatentArgs {
    const int* pos;
    const int* seq_of_token;
    // keys
    const float* proj;        // [T, ld] the projection row: the latent from column lat_at, its rotated part after it
    int ld, lat_at, r;
    const float* w;           // [r]
    float eps;
    const float* cq_w;        // [q_rank] the norm weight of the queries' latent (columns 0 ... q_rank); null: none
    int q_rank;
    // queries
    const float* q32;         // [T, ldq] heads of dq + rot; null: none
    int ldq, nh, dq;
    int q_major;              // records token by token; else head by head and the rotated part into q_rec
    // the rotation
    const float* freq;
    int rot, interleaved;
    float mscale;
    int num_tokens, D;
};

// One block a token.  CQ_UNITS: 16-byte units of the queries' latent a thread keeps in registers (0: there is none, so
// that the other forms do not pay for its registers).
template <typename OT, int CQ_UNITS>
__global__ void __launch_bounds__(256)
latent_prepare_kernel(const LatentArgs a, OT* __restrict__ q_t, OT* __restrict__ q_rec, OT* __restrict__ k_new,
                      OT* __restrict__ cq, const LatentCommit c, int* status, int vec4, int cq_vec) {
    __shared__ float red[32];
    __shared__ __align__(16) float ang[LATENT_MAX_ROT];        // cos[rot / 2], sin[rot / 2]
    const int t = blockIdx.x, rot = a.rot, half = rot / 2, D = a.D, r = a.r;
    pdl_sync();
    auto angles = [&]() {      // (read after the next barrier)
        if (rot > 0) {
            const float p = (float)a.pos[t];
            for (int i = threadIdx.x; i < half; i += blockDim.x) {
                float sn, cs;
                sincosf(p * a.freq[i], &sn, &cs);
                ang[i] = cs * a.mscale, ang[half + i] = sn * a.mscale;
            }
        }
    };
    if (!k_new) {
        angles();
        __syncthreads();
    }
    // element j of the rotated vector whose rotated part starts at v
    auto turned = [&](const float* v, int j) {
        const int i = a.interleaved ? j >> 1 : (j < half ? j : j - half);
        const bool second = a.interleaved ? (j & 1) != 0 : j >= half;
        const float lo = v[a.interleaved ? 2 * i : i], hi = v[a.interleaved ? 2 * i + 1 : i + half];
        return second ? rot_hi(lo, hi, ang[i], ang[half + i]) : rot_lo(lo, hi, ang[i], ang[half + i]);
    };
    if (k_new) {
        // Both latents' loads are on their way before either sum is formed; the queries' latent stays in
        // registers (four elements a unit) where it fits, and both sums share their barriers.
        const float* row = a.proj + (size_t)t * a.ld;
        const float* lat = row + a.lat_at;
        const float lat0 = (int)threadIdx.x < r ? lat[threadIdx.x] : 0.f;
        float4 cu[CQ_UNITS > 0 ? CQ_UNITS : 1];
        const bool cq_regs = cq_vec && a.q_rank <= 4 * CQ_UNITS * (int)blockDim.x;
        float ss = 0.f, sq = 0.f;
        if (CQ_UNITS > 0 && a.cq_w && cq_regs) {
#pragma unroll
            for (int u = 0; u < CQ_UNITS; u++) {
                const int i = (threadIdx.x + u * blockDim.x) * 4;
                cu[u] = i < a.q_rank ? *reinterpret_cast<const float4*>(row + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
        angles();
        ss = lat0 * lat0;
        for (int i = threadIdx.x + blockDim.x; i < r; i += blockDim.x) ss += lat[i] * lat[i];
        if (CQ_UNITS > 0 && a.cq_w) {
            if (cq_regs) {
#pragma unroll
                for (int u = 0; u < CQ_UNITS; u++)
                    sq += cu[u].x * cu[u].x, sq += cu[u].y * cu[u].y, sq += cu[u].z * cu[u].z, sq += cu[u].w * cu[u].w;
            } else {
                for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x) sq += row[i] * row[i];
            }
        }
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
        ss = warp_sum(ss), sq = warp_sum(sq);
        if (lane == 0) red[warp] = ss, red[16 + warp] = sq;
        __syncthreads();
        ss = warp_sum(lane < nw ? red[lane] : 0.f), sq = warp_sum(lane < nw ? red[16 + lane] : 0.f);
        const float inv = 1.0f / sqrtf(ss / (float)r + a.eps);
        OT* cd = nullptr;
        OT* cv = nullptr;
        if (c.k_cache) {
            const int s = a.seq_of_token[t];
            const int p = a.pos[t];
            if (s >= 0 && !(c.ring > 0 && p < c.seq_end[s] - c.ring)) {
                const CachePos cp = cache_pos(p, c.ring, c.tables + (size_t)c.slots[s] * c.table_stride, c.page_size,
                                              c.num_pages, status);
                const size_t at = cache_index(cp, 0, 1, c.page_size, D);
                cd = (OT*)c.k_cache + at;
                if (c.v_cache && c.v_cache != c.k_cache) cv = (OT*)c.v_cache + at;
            }
        }
        OT* kd = k_new + (size_t)t * D;
        for (int i = threadIdx.x; i < D; i += blockDim.x) {
            const float x = i < r ? lat[i] * inv * a.w[i] : i < r + rot ? turned(lat + r, i - r) : 0.f;
            st_f(kd + i, x);
            if (cd) st_f(cd + i, x);
            if (cv) st_f(cv + i, x);
        }
        if (CQ_UNITS > 0 && a.cq_w) {
            const float qi = 1.0f / sqrtf(sq / (float)a.q_rank + a.eps);
            OT* cr = cq + (size_t)t * a.q_rank;
            if (cq_regs) {
#pragma unroll
                for (int u = 0; u < CQ_UNITS; u++) {
                    const int i = (threadIdx.x + u * blockDim.x) * 4;
                    if (i < a.q_rank) {
                        const float4 w = *reinterpret_cast<const float4*>(a.cq_w + i);
                        const float v[4] = {cu[u].x * qi * w.x, cu[u].y * qi * w.y, cu[u].z * qi * w.z, cu[u].w * qi * w.w};
                        st4(cr + i, v);
                    }
                }
            } else {
                for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x) st_f(cr + i, row[i] * qi * a.cq_w[i]);
            }
        }
    }
    if (!a.q32) return;
    const int nh = a.nh, dq = a.dq, hd = dq + rot;
    const float* row = a.q32 + (size_t)t * a.ldq;
    if (a.q_major) {     // the queries token by token, q[t][h][0..D), zero-filled beyond dq + rot
        OT* qd = q_t + (size_t)t * nh * D;
        if (vec4) {
            for (int i = threadIdx.x * 4; i < nh * D; i += blockDim.x * 4) {
                const int h = i / D, j = i - h * D;
                const float* head = row + (size_t)h * hd;
                float v[4] = {0.f, 0.f, 0.f, 0.f};
                if (j < dq) {
                    ld4(head + j, v);
                } else if (j < hd) {
                    const float* rp = head + dq;
                    const int jj = j - dq;
                    ld4(rp + jj, v);
                    if (a.interleaved) {
                        const int i0 = jj >> 1;
#pragma unroll
                        for (int e = 0; e < 2; e++) {
                            const float lo = v[2 * e], hi = v[2 * e + 1], cs = ang[i0 + e], sn = ang[half + i0 + e];
                            v[2 * e] = rot_lo(lo, hi, cs, sn), v[2 * e + 1] = rot_hi(lo, hi, cs, sn);
                        }
                    } else {
                        const bool second = jj >= half;
                        const int i0 = second ? jj - half : jj;
                        float o[4];
                        ld4(rp + (second ? i0 : i0 + half), o);
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            const float cs = ang[i0 + e], sn = ang[half + i0 + e];
                            v[e] = second ? rot_hi(o[e], v[e], cs, sn) : rot_lo(v[e], o[e], cs, sn);
                        }
                    }
                }
                st4(qd + i, v);
            }
        } else {
            for (int i = threadIdx.x; i < nh * D; i += blockDim.x) {
                const int h = i / D, j = i - h * D;
                const float* head = row + (size_t)h * hd;
                st_f(qd + i, j < dq ? head[j] : j < hd ? turned(head + dq, j - dq) : 0.f);
            }
        }
        return;
    }
    if (rot > 0) {       // the records' columns from r on; the ones before come from the per-head product
        const int tail = D - r;
        for (int i = threadIdx.x; i < nh * tail; i += blockDim.x) {
            const int h = i / tail, j = i - h * tail;
            st_f(q_rec + ((size_t)t * nh + h) * D + r + j, j < rot ? turned(row + (size_t)h * hd + dq, j) : 0.f);
        }
    }
    if (vec4) {
        for (int i = threadIdx.x * 4; i < nh * dq; i += blockDim.x * 4) {
            const int h = i / dq, j = i - h * dq;
            float v[4];
            ld4(row + (size_t)h * hd + j, v);
            st4(q_t + ((size_t)h * a.num_tokens + t) * dq + j, v);
        }
        return;
    }
    for (int i = threadIdx.x; i < nh * dq; i += blockDim.x) {
        const int h = i / dq, j = i - h * dq;
        st_f(q_t + ((size_t)h * a.num_tokens + t) * dq + j, row[(size_t)h * hd + j]);
    }
}

// Keys and the queries' latent of many tokens: a warp a token, no barrier between loads, sums and stores.  CU: 16-byte
// units of the queries' latent a lane holds (q_rank <= 128 CU); latents of up to 256, rotated parts of up to 64.
constexpr int LK_WARPS = 4;
template <typename OT, int CU>
__global__ void __launch_bounds__(LK_WARPS * 32)
latent_keys_kernel(const LatentArgs a, OT* __restrict__ k_new, OT* __restrict__ cq, const LatentCommit c, int* status) {
    const int lane = threadIdx.x & 31;
    const int t = blockIdx.x * LK_WARPS + (threadIdx.x >> 5);
    pdl_sync();
    if (t >= a.num_tokens) return;                   // (the whole warp)
    const int r = a.r, rot = a.rot, half = rot / 2, D = a.D;
    const float* row = a.proj + (size_t)t * a.ld;
    const float* lat = row + a.lat_at;
    float4 cu[CU];
    float lx[8];
#pragma unroll
    for (int u = 0; u < CU; u++) {
        const int i = (u * 32 + lane) * 4;
        cu[u] = i < a.q_rank ? *reinterpret_cast<const float4*>(row + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int u = 0; u < 8; u++) lx[u] = u * 32 + lane < r ? lat[u * 32 + lane] : 0.f;
    // lane i < rot / 2 turns pair i
    float lo = 0.f, hi = 0.f, sn = 0.f, cs = 1.f;
    const int at_lo = a.interleaved ? 2 * lane : lane, at_hi = a.interleaved ? 2 * lane + 1 : lane + half;
    if (lane < half) {
        lo = lat[r + at_lo], hi = lat[r + at_hi];
        sincosf((float)a.pos[t] * a.freq[lane], &sn, &cs);
        sn *= a.mscale, cs *= a.mscale;
    }
    OT* cd = nullptr;
    OT* cv = nullptr;
    if (c.k_cache) {
        const int s = a.seq_of_token[t], p = a.pos[t];
        if (s >= 0 && !(c.ring > 0 && p < c.seq_end[s] - c.ring)) {
            const CachePos cp = cache_pos(p, c.ring, c.tables + (size_t)c.slots[s] * c.table_stride, c.page_size, c.num_pages, status);
            const size_t at = cache_index(cp, 0, 1, c.page_size, D);
            cd = (OT*)c.k_cache + at;
            if (c.v_cache && c.v_cache != c.k_cache) cv = (OT*)c.v_cache + at;
        }
    }
    float ss = 0.f, sq = 0.f;
#pragma unroll
    for (int u = 0; u < 8; u++) ss = fmaf(lx[u], lx[u], ss);
#pragma unroll
    for (int u = 0; u < CU; u++)
        sq = fmaf(cu[u].x, cu[u].x, fmaf(cu[u].y, cu[u].y, fmaf(cu[u].z, cu[u].z, fmaf(cu[u].w, cu[u].w, sq))));
    ss = warp_sum(ss), sq = warp_sum(sq);
    const float inv = 1.0f / sqrtf(ss / (float)r + a.eps), qi = 1.0f / sqrtf(sq / (float)a.q_rank + a.eps);
    OT* kd = k_new + (size_t)t * D;
    auto put = [&](int i, float x) {
        st_f(kd + i, x);
        if (cd) st_f(cd + i, x);
        if (cv) st_f(cv + i, x);
    };
#pragma unroll
    for (int u = 0; u < 8; u++)
        if (u * 32 + lane < r) put(u * 32 + lane, lx[u] * inv * a.w[u * 32 + lane]);
    if (lane < half) put(r + at_lo, rot_lo(lo, hi, cs, sn)), put(r + at_hi, rot_hi(lo, hi, cs, sn));
    for (int i = r + rot + lane; i < D; i += 32) put(i, 0.f);
    OT* cr = cq + (size_t)t * a.q_rank;
#pragma unroll
    for (int u = 0; u < CU; u++) {
        const int i = (u * 32 + lane) * 4;
        if (i < a.q_rank) {
            const float4 w = *reinterpret_cast<const float4*>(a.cq_w + i);
            const float v[4] = {cu[u].x * qi * w.x, cu[u].y * qi * w.y, cu[u].z * qi * w.z, cu[u].w * qi * w.w};
            st4(cr + i, v);
        }
    }
}

__device__ __forceinline__ void ld2(const float* p, float* v) {
    const float2 x = *reinterpret_cast<const float2*>(p);
    v[0] = x.x, v[1] = x.y;
}
__device__ __forceinline__ void ld2(const __nv_bfloat16* p, float* v) {
    const unsigned x = *reinterpret_cast<const unsigned*>(p);
    v[0] = __uint_as_float(x << 16), v[1] = __uint_as_float(x & 0xffff0000u);
}
__device__ __forceinline__ void st2(float* p, const float* v) { *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]); }
__device__ __forceinline__ void st2(__nv_bfloat16* p, const float* v) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
}

// VEC = 4: n, wd and all pitches are multiples of four and both pointers aligned to four elements.
template <typename ST, typename DT, int VEC>
__global__ void heads_transpose_kernel(const ST* __restrict__ src, long long s_outer, long long s_inner, int A, int B,
                                       int n, int wd, DT* __restrict__ dst, int ldd, const float* __restrict__ gate,
                                       int gate_ld) {
    pdl_sync();
    const int wv = wd / VEC;
    const long long total = (long long)A * B * wv;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int j = (int)(i % wv) * VEC;
    const long long ba = i / wv;
    const int a = (int)(ba % A), b = (int)(ba / A);
    const ST* from = src + (size_t)a * s_outer + (size_t)b * s_inner + j;
    DT* to = dst + ba * ldd + j;
    const float f = gate ? 1.0f / (1.0f + expf(-gate[(size_t)b * gate_ld + a])) : 1.0f;
    if (VEC == 4) {
        float v[4] = {0.f, 0.f, 0.f, 0.f};
        if (j < n) ld4(from, v);
        v[0] *= f, v[1] *= f, v[2] *= f, v[3] *= f;
        st4(to, v);
    } else {
        st_f(to, j < n ? ld_f(from) * f : 0.f);
    }
}

// One warp a (token, head).  The head's difference stays in registers between the norm's sum and the
// store (dv <= 256: up to eight elements a lane); with an even dv (and 4-byte aligned rows) a lane
// takes two neighbouring elements a load.
template <typename T, int VEC>
__global__ void __launch_bounds__(128)
diff_combine_kernel(const T* __restrict__ ctx, const float* __restrict__ gate, int gate_ld, long long pairs, int nh,
                    int dv, int D, float lambda, float eps, float mult, T* __restrict__ out) {
    pdl_sync();
    const long long w = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (w >= pairs) return;
    const long long t = w / nh;
    const int h = (int)(w % nh);
    const T* a1 = ctx + ((size_t)t * 2 * nh + h) * D;
    const T* a2 = ctx + ((size_t)t * 2 * nh + nh + h) * D;
    constexpr int SLOTS = 256 / (32 * VEC);
    float o[SLOTS][VEC];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < SLOTS; i++) {
        const int j = (i * 32 + lane) * VEC;
#pragma unroll
        for (int e = 0; e < VEC; e++) o[i][e] = 0.f;
        if (j < dv) {
            if (VEC == 2) {
                float x[2], y[2];
                ld2(a1 + j, x), ld2(a2 + j, y);
                o[i][0] = x[0] - lambda * y[0], o[i][1] = x[1] - lambda * y[1];
            } else {
                o[i][0] = ld_f(a1 + j) - lambda * ld_f(a2 + j);
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; e++) ss += o[i][e] * o[i][e];
    }
    ss = warp_sum(ss);
    float f = mult / sqrtf(ss / (float)dv + eps);
    if (gate) f *= 1.0f / (1.0f + expf(-gate[(size_t)t * gate_ld + h]));
    T* o_row = out + ((size_t)t * nh + h) * dv;
#pragma unroll
    for (int i = 0; i < SLOTS; i++) {
        const int j = (i * 32 + lane) * VEC;
        if (j < dv) {
            if (VEC == 2) {
                const float v[2] = {o[i][0] * f, o[i][1] * f};
                st2(o_row + j, v);
            } else {
                st_f(o_row + j, o[i][0] * f);
            }
        }
    }
}

__global__ void add_row_kernel(float* __restrict__ x, const float* __restrict__ delta, const float* __restrict__ row,
                               long long total, int width) {
    pdl_sync();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    float v = x[i];
    if (delta) v += delta[i];
    x[i] = v + row[i % width];
}

}  // namespace

// Keys (k_new given): proj [T, ld] 32-bit with the latent's r columns from lat_at, then `rot` columns of the
// rotated key part; k_new: [T, D], D >= r + rot; with cq_w the columns 0 ... q_rank are normed into cq [T, q_rank].
// Queries (q32 given): [T, ldq] 32-bit, nh heads of dq + rot; q_major: q_t is [T, nh, D], zero-filled beyond
// dq + rot <= D; else q_t is [nh, T, dq] and, with rot > 0, columns r ... D of q_rec [T, nh, D] are written.
MOE_API int moe_latent_prepare(const float* proj, int ld, int lat_at, int r, const float* w, float eps, const float* cq_w,
                               int q_rank, void* cq, const float* q32, int ldq, int nh, int dq, int q_major,
                               const float* freq, int rot, int interleaved, float mscale, const int* pos,
                               const int* seq_of_token, int num_tokens, int D, void* q_t, void* q_rec, void* k_new,
                               int out_dt, void* k_cache, void* v_cache, const int* seq_end, const int* slots,
                               const int* tables, int table_stride, int ring, int page_size, int num_pages,
                               int* status, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    if (rot < 0 || rot % 2 || rot > LATENT_MAX_ROT || (rot > 0 && (!freq || !pos)) || r <= 0 || D < r + rot)
        return (int)cudaErrorInvalidValue;
    if (!k_new && !q32) return (int)cudaErrorInvalidValue;
    if (k_new && (!proj || !w || lat_at < 0 || ld < lat_at + r + rot)) return (int)cudaErrorInvalidValue;
    if (cq_w && (!k_new || !cq || q_rank <= 0 || q_rank > lat_at)) return (int)cudaErrorInvalidValue;
    if (q32 && (nh <= 0 || dq <= 0 || ldq < nh * (dq + rot) || !q_t || (q_major && dq + rot > D) || (!q_major && rot > 0 && !q_rec)))
        return (int)cudaErrorInvalidValue;
    if (k_cache && (!k_new || !seq_end || !slots || !tables || !seq_of_token || !pos)) return (int)cudaErrorInvalidValue;
    const LatentCommit c{k_cache, v_cache, seq_end, slots, tables, table_stride, ring, page_size, num_pages};
    const LatentArgs a{pos, seq_of_token, proj, ld, lat_at, r, w, eps, cq_w, q_rank, q32, ldq, nh, dq, q_major,
                       freq, rot, interleaved, mscale, num_tokens, D};
    const int vec4 = dq % 4 == 0 && ldq % 4 == 0 && (uintptr_t)q32 % 16 == 0 && rot % (interleaved ? 4 : 8) == 0 &&
                     (!q_major || D % 4 == 0) && (uintptr_t)q_t % (out_dt == DT_F32 ? 16 : 8) == 0;
    const int al = out_dt == DT_F32 ? 16 : 8;
    const int cq_vec = cq_w && q_rank % 4 == 0 && ld % 4 == 0 && ((uintptr_t)proj | (uintptr_t)cq_w) % 16 == 0 && (uintptr_t)cq % al == 0;
    if (cq_vec && !q32 && num_tokens >= 512 && q_rank <= 2048 && r <= 256 && rot <= 64) {
#define KEYS(OT_, CU_)                                                                                                 \
    return launch_pdl(latent_keys_kernel<OT_, CU_>, (num_tokens + LK_WARPS - 1) / LK_WARPS, LK_WARPS * 32, 0, stream, a, \
                      (OT_*)k_new, (OT_*)cq, c, status)
        if (out_dt == DT_F32) {
            if (q_rank <= 1024) KEYS(float, 8);
            KEYS(float, 16);
        }
        if (q_rank <= 1024) KEYS(__nv_bfloat16, 8);
        KEYS(__nv_bfloat16, 16);
#undef KEYS
    }
    // keys alone are little work a token: smaller blocks, more of them on an SM
    const int threads = q32 || num_tokens < 512 ? 256 : 128;
#define PREP(OT_, U_)                                                                                                  \
    return launch_pdl(latent_prepare_kernel<OT_, U_>, num_tokens, threads, 0, stream, a, (OT_*)q_t, (OT_*)q_rec,       \
                      (OT_*)k_new, (OT_*)cq, c, status, vec4, cq_vec)
    if (out_dt == DT_F32) {
        if (cq_w) PREP(float, 4);
        PREP(float, 0);
    }
    if (cq_w) PREP(__nv_bfloat16, 4);
    PREP(__nv_bfloat16, 0);
#undef PREP
}

// src: element (a, b, j) at a * s_outer + b * s_inner + j, j < n; dst: [B, A, wd] with rows of ldd elements (dense
// otherwise); gate: 32-bit logits [B, A], rows of gate_ld, or null.
MOE_API int moe_heads_transpose(const void* src, int src_dt, long long s_outer, long long s_inner, int A, int B, int n,
                                int wd, void* dst, int dst_dt, int ldd, const float* gate, int gate_ld,
                                cudaStream_t stream) {
    const long long total = (long long)A * B * wd;
    if (total <= 0) return 0;
    if (n < 0 || n > wd || ldd < wd || !src || !dst || (gate && gate_ld < A)) return (int)cudaErrorInvalidValue;
    const size_t se = src_dt == DT_F32 ? 4 : 2, de = dst_dt == DT_F32 ? 4 : 2;
    const bool vec = n % 4 == 0 && wd % 4 == 0 && ldd % 4 == 0 && s_outer % 4 == 0 && s_inner % 4 == 0 &&
                     (uintptr_t)src % (4 * se) == 0 && (uintptr_t)dst % (4 * de) == 0;
    const unsigned blocks = (unsigned)(((vec ? total / 4 : total) + 255) / 256);
#define TR(ST_, DT_)                                                                                                \
    return vec ? launch_pdl(heads_transpose_kernel<ST_, DT_, 4>, blocks, 256, 0, stream, (const ST_*)src, s_outer,      \
                            s_inner, A, B, n, wd, (DT_*)dst, ldd, gate, gate_ld)                                        \
               : launch_pdl(heads_transpose_kernel<ST_, DT_, 1>, blocks, 256, 0, stream, (const ST_*)src, s_outer,      \
                            s_inner, A, B, n, wd, (DT_*)dst, ldd, gate, gate_ld)
    if (src_dt == DT_F32) {
        if (dst_dt == DT_F32) TR(float, float);
        TR(float, __nv_bfloat16);
    }
    if (dst_dt == DT_F32) TR(__nv_bfloat16, float);
    TR(__nv_bfloat16, __nv_bfloat16);
#undef TR
}

// ctx: [T, 2 nh, D] (map 1 of every head, then map 2); gate: first gate logit of token 0 (row pitch
// gate_ld, 32-bit) or null; out: [T, nh * dv].
MOE_API int moe_diff_combine(const void* ctx, const float* gate, int gate_ld, int num_tokens, int nh, int dv, int D,
                             float lambda, float eps, float mult, void* out, int dt, cudaStream_t stream) {
    const long long pairs = (long long)num_tokens * nh;
    if (pairs <= 0) return 0;
    if (dv <= 0 || D < dv || !ctx || !out) return (int)cudaErrorInvalidValue;
    if (dv > 256) return (int)cudaErrorInvalidValue;
    const unsigned blocks = (unsigned)((pairs + 3) / 4);
    const size_t el = dt == DT_F32 ? 4 : 2;
    const bool vec = dv % 2 == 0 && D % 2 == 0 && (uintptr_t)ctx % (2 * el) == 0 && (uintptr_t)out % (2 * el) == 0;
#define DC(T_, V_)                                                                                                 \
    return launch_pdl(diff_combine_kernel<T_, V_>, blocks, 128, 0, stream, (const T_*)ctx, gate, gate_ld, pairs, nh, dv, \
                      D, lambda, eps, mult, (T_*)out)
    if (dt == DT_F32) {
        if (vec) DC(float, 2);
        DC(float, 1);
    }
    if (vec) DC(__nv_bfloat16, 2);
    DC(__nv_bfloat16, 1);
#undef DC
}

MOE_API int moe_add_row(float* x, const float* delta, const float* row, long long num_tokens, int width,
                        cudaStream_t stream) {
    const long long total = num_tokens * width;
    if (total <= 0) return 0;
    if (!x || !row) return (int)cudaErrorInvalidValue;
    return launch_pdl(add_row_kernel, (unsigned)((total + 255) / 256), 256, 0, stream, x, delta, row, total, width);
}
