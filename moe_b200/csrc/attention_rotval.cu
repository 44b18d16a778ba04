// Between projection and attention, and between attention and output projection, for attention
// layers whose queries and keys are normed over the WHOLE projection and whose values carry a
// position of their own:
//
//   whole_prepare   from a token's 32-bit projection row [q heads | k heads | v heads]: an optional RMS
//                   norm over all query channels at once (x / sqrt(mean(x^2) + eps) * w, one weight a
//                   channel) and the same over all key channels; the rotation of the first `rot`
//                   dimensions of every query and key head (pairs (i, i + rot/2), angle pos * freq[i]);
//                   optionally the rotation of every value head over all its dv dimensions (pairs
//                   (m, m + dv/2), angle pos * vfreq[m]); the split into q, k and v records of the
//                   cache's width D >= max(d, dv), zero-filled; optionally the append to the paged cache.
//   unrotate_pack   out[t, h * dv + :] = the head's attention output turned back by the QUERY's position
//                   (pair m by -pos * vfreq[m]), which leaves every value turned by its distance to the
//                   query; the padding columns of the record are dropped.
//   whole_conv_prepare   the same place for layers whose queries and keys first pass a short causal convolution
//                   over time (per channel y_t = sum_j w[j] u_(t - taps + 1 + j); rows before the step come from the
//                   sequence's state, the last taps - 1 projected rows, and are zero before position 0), then the
//                   norms over the whole of q and of k, then the rotation, of pairs (2i, 2i + 1) or (i, i + rot/2).
//                   Values have rows of their own in the projection and pass the convolution too, or ARE the
//                   convolved keys, neither normed nor turned.  In a step of one token a
//                   sequence the same launch moves the convolution's state on.
// Convolution, norm, angles and rotations are 32-bit; only the stores round to the activation dtype.
#include "common.cuh"

namespace {

struct WholeCommit {
    void* k_cache;            // null: no append
    void* v_cache;
    const int* seq_end;
    const int* slots;
    const int* tables;
    int table_stride, ring, page_size, num_pages, pinned;
};

constexpr int WP_THREADS = 256;

template <typename OT>
__global__ void __launch_bounds__(WP_THREADS)
whole_prepare_kernel(const float* __restrict__ proj, int ld, const int* __restrict__ pos,
                     const int* __restrict__ seq_of_token, const float* __restrict__ q_norm,
                     const float* __restrict__ k_norm, float eps, const float* __restrict__ freq, int rot,
                     const float* __restrict__ vfreq, int nh, int nkv, int d, int dv, int D, OT* __restrict__ q,
                     OT* __restrict__ k, OT* __restrict__ v, long long ldq, long long ldkv, const WholeCommit c,
                     int* status) {
    extern __shared__ __align__(16) float wp_smem[];
    __shared__ float red[32];
    const int half = rot / 2, vhalf = vfreq ? dv / 2 : 0;
    float* ang = wp_smem;                 // cos[half], sin[half]
    float* vang = wp_smem + 2 * half;     // cos[vhalf], sin[vhalf]
    const int t = blockIdx.x;
    pdl_sync();
    const int p_int = pos[t];
    const float p = (float)p_int;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cs;
        sincosf(p * freq[i], &sn, &cs);
        ang[i] = cs, ang[half + i] = sn;
    }
    for (int i = threadIdx.x; i < vhalf; i += blockDim.x) {
        float sn, cs;
        sincosf(p * vfreq[i], &sn, &cs);
        vang[i] = cs, vang[vhalf + i] = sn;
    }
    const float* row = proj + (size_t)t * ld;
    const int nq = nh * d, nk = nkv * d;
    float inv_q = 1.f, inv_k = 1.f;
    const int my_per = (nh + 2 * nkv + gridDim.y - 1) / gridDim.y;
    const bool has_q = blockIdx.y * my_per < nh;
    const bool has_k = blockIdx.y * my_per < nh + nkv && (blockIdx.y + 1) * my_per > nh;
    if (q_norm && has_q) {
        float ss = 0.f;
        for (int e = threadIdx.x; e < nq; e += blockDim.x) ss = fmaf(row[e], row[e], ss);
        inv_q = 1.0f / sqrtf(block_sum(ss, red) / (float)nq + eps);
    }
    if (k_norm && has_k) {
        float ss = 0.f;
        for (int e = threadIdx.x; e < nk; e += blockDim.x) ss = fmaf(row[nq + e], row[nq + e], ss);
        inv_k = 1.0f / sqrtf(block_sum(ss, red) / (float)nk + eps);
    }
    __syncthreads();
    bool append = false;
    CachePos cp;
    cp.page = 0, cp.off = 0;
    if (c.k_cache) {
        const int s = seq_of_token[t];
        if (s >= 0 && cache_holds(p_int, c.seq_end[s], c.ring, c.pinned)) {
            cp = cache_pos(p_int, c.ring, c.tables + (size_t)c.slots[s] * c.table_stride, c.page_size, c.num_pages,
                           status, c.pinned);
            append = true;
        }
    }
    // (few tokens: gridDim.y blocks share a token's head slots, each forming the sums of squares for itself)
    const int hs_count = nh + 2 * nkv;
    const int per = (hs_count + gridDim.y - 1) / gridDim.y;
    const int hs_lo = blockIdx.y * per, hs_hi = min(hs_count, hs_lo + per);
    for (int idx = hs_lo * D + threadIdx.x; idx < hs_hi * D; idx += blockDim.x) {
        const int hs = idx / D, e = idx % D;
        const bool is_q = hs < nh, is_k = !is_q && hs < nh + nkv;
        const int head = is_q ? hs : is_k ? hs - nh : hs - nh - nkv;
        float x = 0.f;
        if (is_q || is_k) {
            if (e < d) {
                const int c0 = (is_q ? 0 : nq) + head * d;          // the head's first channel in the row
                const float inv = is_q ? inv_q : inv_k;
                const float* nw = is_q ? q_norm : k_norm;
                const int wc = head * d;                            // ... and in the norm's weight
                auto val = [&](int i) { return nw ? row[c0 + i] * inv * nw[wc + i] : row[c0 + i]; };
                if (e < rot) {
                    const int i = e < half ? e : e - half;
                    const float a = val(i), b = val(i + half), cs = ang[i], sn = ang[half + i];
                    x = e < half ? rot_lo(a, b, cs, sn) : rot_hi(a, b, cs, sn);
                } else {
                    x = val(e);
                }
            }
        } else if (e < dv) {
            const float* src = row + nq + nk + head * dv;
            if (vhalf && e < 2 * vhalf) {
                const int i = e < vhalf ? e : e - vhalf;
                const float a = src[i], b = src[i + vhalf], cs = vang[i], sn = vang[vhalf + i];
                x = e < vhalf ? rot_lo(a, b, cs, sn) : rot_hi(a, b, cs, sn);
            } else {
                x = src[e];
            }
        }
        OT* dst = is_q ? q + (size_t)t * ldq + (size_t)head * D : (is_k ? k : v) + (size_t)t * ldkv + (size_t)head * D;
        st_f(dst + e, x);
        if (!is_q && append)
            st_f((OT*)(is_k ? c.k_cache : c.v_cache) + cache_index(cp, head, nkv, c.page_size, D) + e, x);
    }
}

struct WholeConv {
    const float* proj;         // [T, ld]: q heads (nh * d) | k heads (nkv * d) | v heads (nkv * dv, unless the values are the keys)
    int ld;
    const int* pos;
    const int* seq_of_token;
    const int* cu_seqlens;
    const int* slots;
    const float* taps_w;       // [taps, channels]
    float* state;              // per slot (taps - 1) * channels floats, oldest row first
    long long state_pitch;
    const float* q_norm;       // [nh * d] or null
    const float* k_norm;       // [nkv * d] or null
    float eps;
    const float* freq;
    int taps, shift, rot, neighbours, shared_v, nh, nkv, d, dv, D;
    long long ldq, ldkv;
};

template <int W>
__device__ __forceinline__ void store_run(float* p, const float* x) {
    if (W == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1 % W], x[2 % W], x[3 % W]);
    else p[0] = x[0];
}
template <int W>
__device__ __forceinline__ void store_run(__nv_bfloat16* p, const float* x) {
    if (W == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(x[0], x[1 % W]), hi = __floats2bfloat162_rn(x[2 % W], x[3 % W]);
        uint2 u;
        u.x = *reinterpret_cast<const unsigned*>(&lo), u.y = *reinterpret_cast<const unsigned*>(&hi);
        *reinterpret_cast<uint2*>(p) = u;
    } else {
        p[0] = __float2bfloat16_rn(x[0]);
    }
}

// grid (token, 2): block (t, 0) takes the token's queries, block (t, 1) its keys and values, so that a channel's state
// belongs to one block alone.  The convolved channels stay in shared memory between the norm's sum and the
// rotation.  W: channels a thread works on at a time.
template <typename OT, int W>
__global__ void __launch_bounds__(WP_THREADS)
whole_conv_prepare_kernel(const WholeConv p, OT* __restrict__ q, OT* __restrict__ k, OT* __restrict__ v,
                          const WholeCommit c, int* status) {
    extern __shared__ __align__(16) float wc_smem[];
    __shared__ float red[32];
    const int half = p.rot / 2, t = blockIdx.x;
    const bool keys = blockIdx.y == 1;
    float* row = wc_smem;                                     // this block's channels
    const int channels = (p.nh + p.nkv) * p.d + (p.shared_v ? 0 : p.nkv * p.dv);
    const int c0 = keys ? p.nh * p.d : 0, cnt = keys ? channels - c0 : p.nh * p.d;
    const int normed = keys ? p.nkv * p.d : cnt;
    float* ang = row + ((cnt + 3) & ~3);                      // cos[half], sin[half]
    pdl_sync();
    const int s = p.seq_of_token[t];
    const int p_int = s < 0 ? 0 : p.pos[t];
    const int head_slots = keys ? 2 * p.nkv : p.nh;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    auto dst_of = [&](int hs) {
        return !keys ? q + (size_t)t * p.ldq + (size_t)hs * p.D
                     : (hs < p.nkv ? k + (size_t)hs * p.D : v + (size_t)(hs - p.nkv) * p.D) + (size_t)t * p.ldkv;
    };
    if (s < 0) {                                              // a row of no sequence: zeros
        for (int i = threadIdx.x; i < head_slots * p.D; i += blockDim.x) st_f(dst_of(i / p.D) + i % p.D, 0.f);
        return;
    }
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cs;
        sincosf((float)p_int * p.freq[i], &sn, &cs);
        ang[i] = cs, ang[half + i] = sn;
    }
    // ---- convolution and sum of squares ---------------------------------------------------------------
    const int li = t - p.cu_seqlens[s];
    float* st = p.taps > 1 ? p.state + (size_t)p.slots[s] * p.state_pitch : nullptr;
    float ss = 0.f;
    for (int u = threadIdx.x * W; u < cnt; u += WP_THREADS * W) {
        const int ch = c0 + u;
        float y[W];
#pragma unroll
        for (int e = 0; e < W; e++) y[e] = 0.f;
        if (!p.taps_w) {
#pragma unroll
            for (int e = 0; e < W; e++) y[e] = p.proj[(size_t)t * p.ld + ch + e];
        } else {
            for (int j = 0; j < p.taps; j++) {
                const int r = li - (p.taps - 1) + j;
                if (p_int - (p.taps - 1) + j < 0 && !p.shift) continue;        // before position 0
                const float* src = r >= 0 ? p.proj + (size_t)(t - li + r) * p.ld + ch
                                          : st + (size_t)(p.taps - 1 + r) * channels + ch;
                const float* wj = p.taps_w + (size_t)j * channels + ch;
                float x[W];
                if (W == 4) {
                    const float4 x4 = *reinterpret_cast<const float4*>(src), w4 = *reinterpret_cast<const float4*>(wj);
                    x[0] = x4.x, x[1 % W] = x4.y, x[2 % W] = x4.z, x[3 % W] = x4.w;
                    y[0] = fmaf(w4.x, x4.x, y[0]), y[1 % W] = fmaf(w4.y, x4.y, y[1 % W]);
                    y[2 % W] = fmaf(w4.z, x4.z, y[2 % W]), y[3 % W] = fmaf(w4.w, x4.w, y[3 % W]);
                } else {
                    x[0] = *src;
                    y[0] = fmaf(*wj, x[0], y[0]);
                }
                // (one row a sequence: the state's rows move one place down; a slot's state starts as zeros)
                if (p.shift && j >= 1) store_run<W>(st + (size_t)(j - 1) * channels + ch, x);
            }
        }
#pragma unroll
        for (int e = 0; e < W; e++) {
            row[u + e] = y[e];
            if (u < normed) ss = fmaf(y[e], y[e], ss);
        }
    }
    const float* nw = keys ? p.k_norm : p.q_norm;
    const float inv = nw ? 1.0f / sqrtf(block_sum(ss, red) / (float)normed + p.eps) : 1.f;
    __syncthreads();
    CachePos cp;
    cp.page = 0, cp.off = 0;
    const bool append = keys && c.k_cache && cache_holds(p_int, c.seq_end[s], c.ring, c.pinned);
    if (append)
        cp = cache_pos(p_int, c.ring, c.tables + (size_t)p.slots[s] * c.table_stride, c.page_size, c.num_pages, status, c.pinned);
    // ---- a warp a head: norm, rotation, records ----------------------------------------------------------
    for (int hs = warp; hs < head_slots; hs += WP_THREADS / 32) {
        const bool is_v = keys && hs >= p.nkv;
        const int head = is_v ? hs - p.nkv : hs;
        const int at = is_v && !p.shared_v ? normed + head * p.dv : head * p.d, n = is_v ? p.dv : p.d;
        auto val = [&](int i) { return nw && !is_v ? row[at + i] * inv * nw[at + i] : row[at + i]; };
        OT* dst = dst_of(hs);
        OT* cd = append ? (OT*)(is_v ? c.v_cache : c.k_cache) + cache_index(cp, head, p.nkv, c.page_size, p.D) : nullptr;
        for (int e0 = lane * W; e0 < p.D; e0 += 32 * W) {
            float x[W];
#pragma unroll
            for (int z = 0; z < W; z++) {
                const int e = e0 + z;
                if (e >= n) {
                    x[z] = 0.f;
                } else if (is_v || e >= p.rot) {
                    x[z] = val(e);
                } else {
                    const int i = p.neighbours ? e >> 1 : e < half ? e : e - half;
                    const int a = p.neighbours ? e & ~1 : i, b = p.neighbours ? a + 1 : i + half;
                    x[z] = e == a ? rot_lo(val(a), val(b), ang[i], ang[half + i]) : rot_hi(val(a), val(b), ang[i], ang[half + i]);
                }
            }
            store_run<W>(dst + e0, x);
            if (cd) store_run<W>(cd + e0, x);
        }
    }
}

// A block per token: the token's angles once in shared memory, then every pair of every head.
template <typename OT>
__global__ void __launch_bounds__(128)
unrotate_pack_kernel(const OT* __restrict__ ctx, const int* __restrict__ pos, const float* __restrict__ vfreq, int nh,
                     int dv, int D, OT* __restrict__ out) {
    extern __shared__ __align__(16) float up_smem[];
    const int t = blockIdx.x, vhalf = dv / 2;
    pdl_sync();
    const float p = (float)pos[t];
    for (int i = threadIdx.x; i < vhalf; i += blockDim.x) {
        float sn, cs;
        sincosf(p * vfreq[i], &sn, &cs);
        up_smem[i] = cs, up_smem[vhalf + i] = -sn;      // the turn back
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < nh * vhalf; idx += blockDim.x) {
        const int h = idx / vhalf, m = idx % vhalf;
        const OT* src = ctx + ((size_t)t * nh + h) * D;
        OT* dst = out + ((size_t)t * nh + h) * dv;
        const float a = ld_f(src + m), b = ld_f(src + m + vhalf), cs = up_smem[m], sn = up_smem[vhalf + m];
        st_f(dst + m, rot_lo(a, b, cs, sn));
        st_f(dst + m + vhalf, rot_hi(a, b, cs, sn));
    }
    if (dv & 1)
        for (int h = threadIdx.x; h < nh; h += blockDim.x)
            st_f(out + ((size_t)t * nh + h) * dv + dv - 1, ld_f(ctx + ((size_t)t * nh + h) * D + dv - 1));
}

}  // namespace

// proj: [T, ld] 32-bit: q heads (nh * d), k heads (nkv * d), v heads (nkv * dv).  q_norm [nh * d], k_norm
// [nkv * d] or null (no norm); freq [rot / 2]; vfreq [dv / 2] or null (values are not rotated).
// q: [T, nh, D] with a token pitch of ldq elements; k, v: [T, nkv, D] with a token pitch of ldkv.
MOE_API int moe_whole_prepare(const float* proj, int ld, const int* pos, const int* seq_of_token, const float* q_norm,
                              const float* k_norm, float eps, const float* freq, int rot, const float* vfreq,
                              int num_tokens, int nh, int nkv, int d, int dv, int D, void* q, void* k, void* v,
                              long long ldq, long long ldkv, int out_dt, void* k_cache, void* v_cache,
                              const int* seq_end, const int* slots, const int* tables, int table_stride, int ring,
                              int page_size, int num_pages, int pinned, int* status, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    if (rot < 0 || rot > d || (rot & 1) || (rot > 0 && !freq) || d <= 0 || dv <= 0 || D < d || D < dv || !q || !k ||
        !v || ld < (nh + nkv) * d + nkv * dv || ldq < (long long)nh * D || ldkv < (long long)nkv * D)
        return (int)cudaErrorInvalidValue;
    if (k_cache && (!v_cache || !seq_end || !slots || !tables || !seq_of_token)) return (int)cudaErrorInvalidValue;
    const WholeCommit c{k_cache, v_cache, seq_end, slots, tables, table_stride, ring, page_size, num_pages, pinned};
    const size_t smem = (size_t)(rot + (vfreq ? (dv / 2) * 2 : 0) + 4) * sizeof(float);
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    // from 128 tokens on the blocks fill the GPU anyway; fewer tokens are spread over more blocks
    const int hs_count = nh + 2 * nkv;
    const dim3 grid(num_tokens, num_tokens >= 128 ? 1 : min(hs_count, max(1, (hs_count + 3) / 4)));
    if (out_dt == DT_F32)
        return launch_pdl(whole_prepare_kernel<float>, grid, WP_THREADS, smem, stream, proj, ld, pos,
                          seq_of_token, q_norm, k_norm, eps, freq, rot, vfreq, nh, nkv, d, dv, D, (float*)q, (float*)k,
                          (float*)v, ldq, ldkv, c, status);
    return launch_pdl(whole_prepare_kernel<__nv_bfloat16>, grid, WP_THREADS, smem, stream, proj, ld, pos,
                      seq_of_token, q_norm, k_norm, eps, freq, rot, vfreq, nh, nkv, d, dv, D, (__nv_bfloat16*)q,
                      (__nv_bfloat16*)k, (__nv_bfloat16*)v, ldq, ldkv, c, status);
}

// proj: [T, ld] 32-bit: q heads (nh * d), k heads (nkv * d) and, unless shared_v (the values are the convolved keys; then
// dv == d), v heads (nkv * dv).  taps_w: [taps, channels] 32-bit or null (no convolution); state: (taps - 1) * channels floats
// a slot; shift: the step brings one token a sequence and the state moves on here.  neighbours: pairs (2i, 2i + 1)
// are turned, else (i, i + rot/2).  The rest as moe_whole_prepare.
MOE_API int moe_whole_conv_prepare(const float* proj, int ld, const float* taps_w, int taps, float* state,
                                   long long state_pitch, int shift, const int* pos, const int* seq_of_token,
                                   const int* cu_seqlens, const int* slots, const float* q_norm, const float* k_norm,
                                   float eps, const float* freq, int rot, int neighbours, int shared_v, int num_tokens,
                                   int nh, int nkv, int d, int dv, int D, void* q, void* k, void* v, long long ldq,
                                   long long ldkv, int out_dt, void* k_cache, void* v_cache, const int* seq_end,
                                   const int* tables, int table_stride, int ring, int page_size, int num_pages, int pinned,
                                   int* status, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    const int channels = (nh + nkv) * d + (shared_v ? 0 : nkv * dv);
    if (!proj || !pos || !seq_of_token || !cu_seqlens || !slots || !q || !k || !v || rot < 0 || rot > d || (rot & 1) ||
        (rot > 0 && !freq) || d <= 0 || dv <= 0 || (shared_v && dv != d) || D < d || D < dv || ld < channels ||
        ldq < (long long)nh * D || ldkv < (long long)nkv * D)
        return (int)cudaErrorInvalidValue;
    if (taps_w ? (taps < 1 || taps > 16 || (taps > 1 && (!state || state_pitch < (long long)(taps - 1) * channels))) : taps != 1)
        return (int)cudaErrorInvalidValue;
    if (k_cache && (!v_cache || !seq_end || !tables)) return (int)cudaErrorInvalidValue;
    const WholeCommit c{k_cache, v_cache, seq_end, slots, tables, table_stride, ring, page_size, num_pages, pinned};
    const WholeConv p{proj, ld, pos, seq_of_token, cu_seqlens, slots, taps_w, state, state_pitch, q_norm, k_norm, eps, freq,
                      taps, shift && taps > 1, rot, neighbours, shared_v, nh, nkv, d, dv, D, ldq, ldkv};
    const int most = nh * d > channels - nh * d ? nh * d : channels - nh * d;
    const size_t smem = (size_t)(((most + 3) & ~3) + rot + 4) * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const size_t esz = out_dt == DT_F32 ? 4 : 2;
    auto al = [](const void* x, size_t a) { return ((uintptr_t)x % a) == 0; };
    const bool vec = d % 4 == 0 && dv % 4 == 0 && D % 4 == 0 && ld % 4 == 0 && ldq % 4 == 0 && ldkv % 4 == 0 &&
                     state_pitch % 4 == 0 && al(proj, 16) && al(taps_w, 16) && al(state, 16) && al(q, 4 * esz) &&
                     al(k, 4 * esz) && al(v, 4 * esz) && al(k_cache, 4 * esz) && al(v_cache, 4 * esz);
#define WHOLE_CONV(OT_, W_)                                                                                            \
    do {                                                                                                               \
        if (smem > 48 * 1024) {                                                                                        \
            cudaError_t e = cudaFuncSetAttribute(whole_conv_prepare_kernel<OT_, W_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                       \
        }                                                                                                              \
        return launch_pdl(whole_conv_prepare_kernel<OT_, W_>, dim3(num_tokens, 2), WP_THREADS, smem, stream, p, (OT_*)q, \
                          (OT_*)k, (OT_*)v, c, status);                                                                \
    } while (0)
    if (out_dt == DT_F32) {
        if (vec) WHOLE_CONV(float, 4);
        WHOLE_CONV(float, 1);
    }
    if (vec) WHOLE_CONV(__nv_bfloat16, 4);
    WHOLE_CONV(__nv_bfloat16, 1);
#undef WHOLE_CONV
}

// ctx: [T, nh, D]; out: [T, nh * dv]; vfreq: [dv / 2].
MOE_API int moe_unrotate_pack(const void* ctx, const int* pos, const float* vfreq, int num_tokens, int nh, int dv,
                              int D, void* out, int dt, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    if (!ctx || !pos || !vfreq || !out || nh <= 0 || dv <= 0 || D < dv) return (int)cudaErrorInvalidValue;
    const size_t smem = (size_t)((dv / 2) * 2 + 4) * sizeof(float);
    if (dt == DT_F32)
        return launch_pdl(unrotate_pack_kernel<float>, dim3(num_tokens), 128, smem, stream, (const float*)ctx, pos,
                          vfreq, nh, dv, D, (float*)out);
    return launch_pdl(unrotate_pack_kernel<__nv_bfloat16>, dim3(num_tokens), 128, smem, stream,
                      (const __nv_bfloat16*)ctx, pos, vfreq, nh, dv, D, (__nv_bfloat16*)out);
}
