// The gated delta rule: a recurrent mixer whose state is corrected towards each token's value.
//
// Per value head h (query/key head h / (heads / kv_heads)), with a state S [d, dv] that starts at zero:
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
//   delta_prepare   from the 32-bit projection row [q heads | k heads | v heads | ... | b | a ...]: a causal
//                   convolution over time on every channel of q, k and v (the last taps - 1 rows a
//                   sequence has seen are its state, oldest first) and silu; query and key heads divided
//                   by sqrt(sum(x^2) + eps), queries also times d^(-1/2); per value head
//                   beta = sigmoid(b) and the logarithm of the decay, -exp(A_log) softplus(a + dt_bias).
//                   In a step of one token a sequence the same launch moves the convolution's state on.
//   delta_step      one token a sequence: the recurrence with the state read once and written once, and
//                   the output's norm and gate behind it, a block a (head, sequence).
//   delta_scan      several tokens a sequence, four at a time, the state in registers.
// The decay g is one number a value head, or one a value head and key channel (the rows of S then shrink each by their
// own): delta_prepare forms those from a product's rows of their own, g = exp(-exp(A_log_h) softplus(a + dt_bias)).
// Everything here is 32-bit arithmetic; only the normed, gated output of delta_step is rounded.
#include "common.cuh"

namespace {

constexpr int DP_WARPS = 8;
constexpr int DP_MAX_D = 256;

__device__ __forceinline__ float silu32(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_dt(float z) { return z > 20.f ? z : log1pf(expf(z)); }

struct DeltaPrep {
    const float* proj;         // [T, ld]: q (G d), k (G d), v (H dv) from column 0; b and a from columns b_at, a_at
    long long ld;
    int b_at, a_at;
    const float* taps_w;       // [taps, channels]
    float* state;              // per slot (taps - 1) * channels floats, oldest row first
    long long state_pitch;
    const float* a_log;        // [H]
    const float* dt_bias;      // [H]
    const int* seq_of_token;
    const int* cu_seqlens;
    const int* slots;
    int num_tokens, taps, H, G, d, dv, shift;
    float eps, q_scale;
    float* out;                // [T, channels]: q, k, v
    float* step;               // [T, 2 H]: beta, logarithm of the decay
    // decays of a channel (decay not null): a's rows, [T, lda] with H * d columns; dt_bias is [H * d]
    const float* a_rows;
    long long lda;
    float* decay;              // [T, H * d]: the decays themselves
};

// W neighbouring channels of row t convolved and passed through silu; `st`: the sequence's state, li: the row's place
// among the sequence's rows of the step.  With `shift` (one row a sequence) the state's rows move one place down.
template <int W, int TAPS>
__device__ __forceinline__ void conv_silu(const DeltaPrep& p, int t, int li, float* st, int ch, int channels, float* y) {
    const int taps = TAPS > 0 ? TAPS : p.taps;
#pragma unroll
    for (int e = 0; e < W; e++) y[e] = 0.f;
#pragma unroll
    for (int j = 0; j < taps; j++) {
        const int r = li - (taps - 1) + j;
        const float* src = r >= 0 ? p.proj + (size_t)(t - li + r) * p.ld + ch : st + (size_t)(taps - 1 + r) * channels + ch;
        const float* wj = p.taps_w + (size_t)j * channels + ch;
        if (W == 4) {
            const float4 x = *reinterpret_cast<const float4*>(src), w = *reinterpret_cast<const float4*>(wj);
            y[0] = fmaf(w.x, x.x, y[0]), y[1] = fmaf(w.y, x.y, y[1]), y[2] = fmaf(w.z, x.z, y[2]), y[3] = fmaf(w.w, x.w, y[3]);
            if (p.shift && j >= 1) *reinterpret_cast<float4*>(st + (size_t)(j - 1) * channels + ch) = x;
        } else {
            const float x = *src;
            y[0] = fmaf(*wj, x, y[0]);
            if (p.shift && j >= 1) st[(size_t)(j - 1) * channels + ch] = x;
        }
    }
#pragma unroll
    for (int e = 0; e < W; e++) y[e] = silu32(y[e]);
}

// grid (token, parts of its heads); a warp takes one head of q or k, or one run of 32 W channels of v, in turn.
template <int W, int TAPS>
__global__ void __launch_bounds__(DP_WARPS * 32)
delta_prepare_kernel(const DeltaPrep p) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t = blockIdx.x;
    const int qk = 2 * p.G * p.d, channels = qk + p.H * p.dv;
    const int vruns = (p.H * p.dv + 32 * W - 1) / (32 * W);
    const int druns = p.decay ? (p.H * p.d + 32 * W - 1) / (32 * W) : 0;
    const int items = 2 * p.G + vruns + 1 + druns;
    pdl_sync();
    const int s = p.seq_of_token[t];
    float* out = p.out + (size_t)t * channels;
    float* stp = p.step + (size_t)t * 2 * p.H;
    const int li = s >= 0 ? t - p.cu_seqlens[s] : 0;
    float* st = (s >= 0 && p.taps > 1) ? p.state + (size_t)p.slots[s] * p.state_pitch : nullptr;
    for (int item = blockIdx.y * DP_WARPS + warp; item < items; item += gridDim.y * DP_WARPS) {
        if (s < 0) {           // a row of no sequence: something finite, no state touched
            if (item < 2 * p.G) {
                for (int e = lane; e < p.d; e += 32) out[item * p.d + e] = 0.f;
            } else if (item < 2 * p.G + vruns) {
                for (int e = (item - 2 * p.G) * 32 * W + lane; e < min(p.H * p.dv, (item - 2 * p.G + 1) * 32 * W); e += 32)
                    out[qk + e] = 0.f;
            } else if (item == 2 * p.G + vruns) {
                for (int h = lane; h < 2 * p.H; h += 32) stp[h] = 0.f;
            } else {
                const int r0 = (item - 2 * p.G - vruns - 1) * 32 * W;
                for (int e = r0 + lane; e < min(p.H * p.d, r0 + 32 * W); e += 32) p.decay[(size_t)t * p.H * p.d + e] = 1.f;
            }
            continue;
        }
        if (item < 2 * p.G) {
            const int ch0 = item * p.d;
            constexpr int PASSES = DP_MAX_D / (32 * W);
            float y[PASSES][W];
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < PASSES; i++) {
                const int e = (i * 32 + lane) * W;
                if (e < p.d) {
                    conv_silu<W, TAPS>(p, t, li, st, ch0 + e, channels, y[i]);
#pragma unroll
                    for (int z = 0; z < W; z++) ss = fmaf(y[i][z], y[i][z], ss);
                }
            }
            ss = warp_sum(ss);
            float inv = 1.0f / sqrtf(ss + p.eps);
            if (item < p.G) inv *= p.q_scale;
#pragma unroll
            for (int i = 0; i < PASSES; i++) {
                const int e = (i * 32 + lane) * W;
                if (e < p.d) {
                    if (W == 4)
                        *reinterpret_cast<float4*>(out + ch0 + e) =
                            make_float4(y[i][0] * inv, y[i][1 % W] * inv, y[i][2 % W] * inv, y[i][3 % W] * inv);
                    else
                        out[ch0 + e] = y[i][0] * inv;
                }
            }
        } else if (item < 2 * p.G + vruns) {
            const int e = ((item - 2 * p.G) * 32 + lane) * W;
            if (e < p.H * p.dv) {
                float y[W];
                conv_silu<W, TAPS>(p, t, li, st, qk + e, channels, y);
                if (W == 4)
                    *reinterpret_cast<float4*>(out + qk + e) = make_float4(y[0], y[1 % W], y[2 % W], y[3 % W]);
                else
                    out[qk + e] = y[0];
            }
        } else if (item == 2 * p.G + vruns) {
            const float* row = p.proj + (size_t)t * p.ld;
            for (int h = lane; h < p.H; h += 32) {
                stp[h] = 1.0f / (1.0f + expf(-row[p.b_at + h]));
                stp[p.H + h] = p.decay ? 0.f : -expf(p.a_log[h]) * softplus_dt(row[p.a_at + h] + p.dt_bias[h]);
            }
        } else {
            const int e = ((item - 2 * p.G - vruns - 1) * 32 + lane) * W;
            if (e < p.H * p.d) {
                const float* a = p.a_rows + (size_t)t * p.lda + e;
                const float rate = expf(p.a_log[e / p.d]);            // (W neighbours lie in one head)
                float* dst = p.decay + (size_t)t * p.H * p.d + e;
                if (W == 4) {
                    const float4 x = *reinterpret_cast<const float4*>(a), b = *reinterpret_cast<const float4*>(p.dt_bias + e);
                    *reinterpret_cast<float4*>(dst) = make_float4(expf(-rate * softplus_dt(x.x + b.x)), expf(-rate * softplus_dt(x.y + b.y)),
                                                                  expf(-rate * softplus_dt(x.z + b.z)), expf(-rate * softplus_dt(x.w + b.w)));
                } else {
                    *dst = expf(-rate * softplus_dt(*a + p.dt_bias[e]));
                }
            }
        }
    }
}

struct DeltaSeq {
    const float* qkv;          // [T, channels] prepared q, k, v
    const float* step;         // [T, 2 H]
    float* state;              // per slot H * d * dv floats ([head][d][dv]) from the pointer given
    long long state_pitch;
    const int* cu_seqlens;
    const int* slots;
    int H, G, d, dv;
    const float* decay;        // [T, H d]: a decay a channel; null: one a head (step)
};

// ---- one token a sequence --------------------------------------------------------------------------
// A block a (head, sequence): thread (cg, kp) holds four neighbouring columns of every KP-th row of S.  The
// state is asked for before the wait for the predecessor: nothing since the step before has written it.
template <typename OT, int UNITS, bool CH>
__global__ void __launch_bounds__(256)
delta_step_kernel(const DeltaSeq p, const float* __restrict__ gate, long long ldg, const float* __restrict__ norm_w,
                  float norm_eps, const int* __restrict__ seq_of_token, int num_tokens, int gate_fn, OT* __restrict__ out) {
    extern __shared__ __align__(16) float ds_smem[];         // k [d] | q [d] | u [dv] | parts [KP][dv] | CH: decays [d]
    __shared__ float red[32];
    const int h = blockIdx.x, s = blockIdx.y, d = p.d, dv = p.dv;
    const int CG = dv / 4, KP = blockDim.x / CG, cg = threadIdx.x % CG, kp = threadIdx.x / CG;
    const bool worker = kp < KP;
    float* sk = ds_smem;
    float* sq = sk + d;
    float* su = sq + d;
    float* parts = su + dv;
    float* sg = parts + KP * dv;
    const int t = p.cu_seqlens[s];
    const bool live = p.cu_seqlens[s + 1] > t && t < num_tokens && seq_of_token[t] >= 0;
    float* S = p.state + (size_t)p.slots[s] * p.state_pitch + (size_t)h * d * dv;
    float4 r[UNITS];
#pragma unroll
    for (int i = 0; i < UNITS; i++) {
        const int row = kp + i * KP;
        r[i] = (live && worker && row < d) ? *reinterpret_cast<const float4*>(S + (size_t)row * dv + cg * 4)
                                           : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_sync();
    if (!live) {                                             // row s is a row of no sequence: something finite
        if (s < num_tokens && seq_of_token[s] < 0)
            for (int c = threadIdx.x; c < dv; c += blockDim.x) st_f(out + ((size_t)s * p.H + h) * dv + c, 0.f);
        return;
    }
    const int g = h / (p.H / p.G), channels = 2 * p.G * d + p.H * dv;
    const float* row = p.qkv + (size_t)t * channels;
    for (int i = threadIdx.x; i < d; i += blockDim.x) sq[i] = row[(size_t)g * d + i], sk[i] = row[(size_t)(p.G + g) * d + i];
    if (CH)
        for (int i = threadIdx.x; i < d; i += blockDim.x) sg[i] = p.decay[((size_t)t * p.H + h) * d + i];
    const float beta = p.step[(size_t)t * 2 * p.H + h];
    float decay = CH ? 1.f : expf(p.step[(size_t)t * 2 * p.H + p.H + h]);
    __syncthreads();
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < UNITS; i++) {
        const int rr = kp + i * KP;
        if (CH) decay = (worker && rr < d) ? sg[rr] : 0.f;
        r[i].x *= decay, r[i].y *= decay, r[i].z *= decay, r[i].w *= decay;
        if (worker && rr < d) {
            const float k = sk[rr];
            acc.x = fmaf(k, r[i].x, acc.x), acc.y = fmaf(k, r[i].y, acc.y);
            acc.z = fmaf(k, r[i].z, acc.z), acc.w = fmaf(k, r[i].w, acc.w);
        }
    }
    if (worker) *reinterpret_cast<float4*>(parts + (size_t)kp * dv + cg * 4) = acc;
    __syncthreads();
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        float held = 0.f;
        for (int q = 0; q < KP; q++) held += parts[(size_t)q * dv + c];
        su[c] = beta * (row[(size_t)2 * p.G * d + (size_t)h * dv + c] - held);
    }
    __syncthreads();
    acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (worker) {
        const float4 u = *reinterpret_cast<const float4*>(su + cg * 4);
#pragma unroll
        for (int i = 0; i < UNITS; i++) {
            const int rr = kp + i * KP;
            if (rr < d) {
                const float k = sk[rr], q = sq[rr];
                r[i].x = fmaf(k, u.x, r[i].x), r[i].y = fmaf(k, u.y, r[i].y), r[i].z = fmaf(k, u.z, r[i].z), r[i].w = fmaf(k, u.w, r[i].w);
                acc.x = fmaf(q, r[i].x, acc.x), acc.y = fmaf(q, r[i].y, acc.y);
                acc.z = fmaf(q, r[i].z, acc.z), acc.w = fmaf(q, r[i].w, acc.w);
                *reinterpret_cast<float4*>(S + (size_t)rr * dv + cg * 4) = r[i];
            }
        }
        *reinterpret_cast<float4*>(parts + (size_t)kp * dv + cg * 4) = acc;
    }
    __syncthreads();
    // the output's norm over the head and its gate
    float ss = 0.f;
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        float o = 0.f;
        for (int q = 0; q < KP; q++) o += parts[(size_t)q * dv + c];
        su[c] = o;
        ss = fmaf(o, o, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)dv + norm_eps);
    for (int c = threadIdx.x; c < dv; c += blockDim.x)
        st_f(out + ((size_t)t * p.H + h) * dv + c,
             su[c] * inv * norm_w[(size_t)h * dv + c] * gate_value(gate_fn, gate[(size_t)t * ldg + (size_t)h * dv + c]));
}

// ---- several tokens a sequence: four at a time ------------------------------------------------------------
// With b_i the sum of the decays' logarithms from a group's first token to its i-th, S the state before the group,
// and the index pairs j < i (or j <= i) inside the group,
//     u_i = beta_i v_i - beta_i e^(b_i) S^T k_i - sum_(j<i) beta_i e^(b_i - b_j) (k_i . k_j) u_j
//     o_i = e^(b_i) S^T q_i + sum_(j<=i) e^(b_i - b_j) (q_i . k_j) u_j
//     S   <- e^(b_4) S + sum_j k_j (e^(b_4 - b_j) u_j)^T
// (CH, a decay a channel: with G_i the product of the channel's decays from the group's first token to its i-th and
// D_ij that from the one after j to i, e^(b_i) S^T k_i becomes S^T (G_i k_i), e^(b_i - b_j) (k_i . k_j) the sum over the
// channels of D_ij k_i k_j, and S <- G_4 S + sum_j (D_4j k_j) u_j^T; every factor is a product of decays, none a
// quotient.  The warp that forms a group's scalars puts G_i k_i, G_i q_i and D_4j k_j in the place of k, q and the decays.)
// which is the recurrence written out: every exponent is <= 0, only the order of additions differs.  Against
// one token at a time the products with S are eight independent sums instead of two with an update between
// them, their sums over the threads are formed together, and the state is multiplied by a decay once.
//
// grid (ceil(dv / COLS), heads, sequences), 128 threads: thread (kp = tid % KP, cg = tid / KP) holds four neighbouring
// columns of rows 4 kp ... 4 kp + 3 of every 4 KP rows of S in registers (rows beyond d stay zero; the KP
// threads' reads of a token's k and q are then neighbours in shared memory).  KP = 16 (32 columns a block) or, where those
// blocks would leave SMs idle, 32 (16 columns a block, half as many rows a thread).  A run of sixteen tokens is staged
// in shared memory as [k | q | the block's columns of v] a token (cp.async, two buffers; rows beyond the
// sequence's last token are zeros with beta 0 and decay 1: they change nothing); warp w forms the scalars of the
// run's group w.  Within a run the groups follow one another without a block barrier.
constexpr int DG = 4, DRUN = 16, DTHREADS = 128;
__host__ __device__ constexpr int dcols(int kp) { return 4 * (DTHREADS / kp); }

__device__ __forceinline__ void cp_zfill(float* dst, const float* src, int bytes, bool on) {
    const unsigned at = (unsigned)__cvta_generic_to_shared(dst);
    const int n = on ? bytes : 0;
    if (bytes == 16)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(at), "l"(src), "r"(n) : "memory");
    else
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(at), "l"(src), "r"(n) : "memory");
}

// VEC: rows of q, k and v start on 16-byte boundaries and hold whole 16-byte units.
template <int RPT, int KP, bool CH>
__host__ __device__ constexpr size_t delta_scan_floats() {
    return (size_t)2 * DRUN * ((CH ? 3 : 2) * RPT * KP + dcols(KP)) + 4 * DRUN + 4 * 32 + DG * dcols(KP) + (CH ? 4 * RPT * KP : 0);
}
template <int RPT, int KP, bool VEC, bool CH>
__global__ void __launch_bounds__(DTHREADS, RPT <= 8 ? (CH && RPT == 8 ? 3 : 4) : 2)
delta_scan_kernel(const DeltaSeq p, float* __restrict__ o) {
    constexpr int NP = RPT * KP, DCOLS = dcols(KP);
    constexpr int V_AT = (CH ? 3 : 2) * NP;                   // a token's row: k, q, CH: its decays, then v
    constexpr int ROWLEN = V_AT + DCOLS;
    extern __shared__ __align__(16) float sm[];               // [2][DRUN][ROWLEN] | steps [2][2][DRUN] | scalars [4][32] | u [DG][DCOLS]
    float* s_step = sm + 2 * DRUN * ROWLEN;                   // | CH: a group's decay of a channel [4][NP]
    float* s_coef = s_step + 4 * DRUN;
    float* s_u = s_coef + 4 * 32;
    float* s_g4 = s_u + DG * DCOLS;
    const int tid = threadIdx.x, kp = tid % KP, cg = tid / KP, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, s = blockIdx.z, g = h / (p.H / p.G), d = p.d, dv = p.dv;
    const int c0 = blockIdx.x * DCOLS, col = c0 + cg * 4;
    for (int i = tid; i < 2 * DRUN * ROWLEN; i += DTHREADS) sm[i] = 0.f;         // columns that no copy writes stay zero
    pdl_sync();
    const int tok0 = p.cu_seqlens[s], cnt = p.cu_seqlens[s + 1] - tok0;
    if (cnt <= 0) return;
    const int channels = 2 * p.G * d + p.H * dv, ncols = min(DCOLS, dv - c0);
    float* S = p.state + (size_t)p.slots[s] * p.state_pitch + (size_t)h * d * dv;
    const bool vec_state = dv % 4 == 0 && ((uintptr_t)S) % 16 == 0;
    float sreg[RPT][4];
#pragma unroll
    for (int m = 0; m < RPT; m++) {
        const int n = (m / 4) * 4 * KP + kp * 4 + m % 4;
        if (vec_state && n < d && col < dv) {
            const float4 t4 = *reinterpret_cast<const float4*>(S + (size_t)n * dv + col);
            sreg[m][0] = t4.x, sreg[m][1] = t4.y, sreg[m][2] = t4.z, sreg[m][3] = t4.w;
        } else {
#pragma unroll
            for (int c = 0; c < 4; c++) sreg[m][c] = (n < d && col + c < dv) ? S[(size_t)n * dv + col + c] : 0.f;
        }
    }
    const float* base = p.qkv + (size_t)tok0 * channels;
    const float* sbase = p.step + (size_t)tok0 * 2 * p.H + h;
    const float* gbase = CH ? p.decay + ((size_t)tok0 * p.H + h) * d : nullptr;
    const int k_at = (p.G + g) * d, q_at = g * d, v_at = 2 * p.G * d + h * dv + c0;
    auto stage = [&](int t0, int buf) {
        float* dst = sm + buf * DRUN * ROWLEN;
        constexpr int W = VEC ? 4 : 1;
        const int kw = d / W, vw = ncols / W, per = 2 * kw + vw + (CH ? kw : 0);
        for (int tt = warp; tt < DRUN; tt += DTHREADS / 32) {           // a warp a token
            const bool on = t0 + tt < cnt;
            const float* row = base + (size_t)min(t0 + tt, cnt - 1) * channels;
            float* to = dst + tt * ROWLEN;
            for (int e = lane; e < per; e += 32) {
                if (CH && e >= 2 * kw + vw) {
                    const int x = e - 2 * kw - vw;
                    cp_zfill(to + 2 * NP + x * W, gbase + (size_t)min(t0 + tt, cnt - 1) * p.H * d + x * W, 4 * W, on);
                    continue;
                }
                const int x = e < kw ? e : e < 2 * kw ? e - kw : e - 2 * kw;
                cp_zfill(to + (e < kw ? 0 : e < 2 * kw ? NP : V_AT) + x * W, row + (e < kw ? k_at : e < 2 * kw ? q_at : v_at) + x * W, 4 * W, on);
            }
        }
        if (tid < 2 * DRUN) {
            const int tt = tid % DRUN, which = tid / DRUN;
            cp_zfill(s_step + (buf * 2 + which) * DRUN + tt, sbase + (size_t)min(t0 + tt, cnt - 1) * 2 * p.H + which * p.H, 4, t0 + tt < cnt);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    __syncthreads();                                  // the zeros are there before any copy writes
    stage(0, 0);
    const bool b0 = (kp & 1) != 0, b1 = (kp & 2) != 0, b2 = (kp & 4) != 0, b3 = (kp & 8) != 0;
    const int my_col = (b0 ? 2 : 0) + (b1 ? 1 : 0);
    for (int t0 = 0, buf = 0; t0 < cnt; t0 += DRUN, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                              // this run is there, and the one before is no longer read
        if (t0 + DRUN < cnt) stage(t0 + DRUN, buf ^ 1);
        float* run = sm + buf * DRUN * ROWLEN;
        {
            // the scalars of group `warp`: products of its keys and queries, then everything made of them
            float* row = run + warp * DG * ROWLEN;
            float dots[16];                           // [0 ... 5] k_i . k_j, j < i;  [6 ... 15] q_i . k_j, j <= i
#pragma unroll
            for (int i = 0; i < 16; i++) dots[i] = 0.f;
            for (int e = lane * 4; e < NP; e += 128) {
                float4 k4[DG], q4[DG];
#pragma unroll
                for (int i = 0; i < DG; i++) {
                    k4[i] = *reinterpret_cast<const float4*>(row + i * ROWLEN + e);
                    q4[i] = *reinterpret_cast<const float4*>(row + i * ROWLEN + NP + e);
                }
                if (CH) {
                    const int left = cnt - t0 - warp * DG;        // tokens of the group; places beyond keep what there is
                    float4 g4[DG];
#pragma unroll
                    for (int i = 0; i < DG; i++)
                        g4[i] = i < left ? *reinterpret_cast<const float4*>(row + i * ROWLEN + 2 * NP + e) : make_float4(1.f, 1.f, 1.f, 1.f);
                    auto mul = [](float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); };
                    auto dot3 = [](float4 a, float4 b, float4 c, float s) {
                        return fmaf(a.x * c.x, b.x, fmaf(a.y * c.y, b.y, fmaf(a.z * c.z, b.z, fmaf(a.w * c.w, b.w, s))));
                    };
                    float4 all = make_float4(1.f, 1.f, 1.f, 1.f);
#pragma unroll
                    for (int j = 0; j < DG; j++) {
                        float4 since = make_float4(1.f, 1.f, 1.f, 1.f);        // from the token after j to i
#pragma unroll
                        for (int i = j; i < DG; i++) {
                            if (i > j) since = mul(since, g4[i]), dots[i * (i - 1) / 2 + j] = dot3(k4[i], k4[j], since, dots[i * (i - 1) / 2 + j]);
                            dots[6 + i * (i + 1) / 2 + j] = dot3(q4[i], k4[j], since, dots[6 + i * (i + 1) / 2 + j]);
                        }
                        all = mul(all, g4[j]);
                        *reinterpret_cast<float4*>(row + j * ROWLEN + e) = mul(k4[j], all);
                        *reinterpret_cast<float4*>(row + j * ROWLEN + NP + e) = mul(q4[j], all);
                        *reinterpret_cast<float4*>(row + j * ROWLEN + 2 * NP + e) = mul(k4[j], since);
                    }
                    *reinterpret_cast<float4*>(s_g4 + warp * NP + e) = all;
                    continue;
                }
                int x = 0;
#pragma unroll
                for (int i = 1; i < DG; i++)
#pragma unroll
                    for (int j = 0; j < i; j++, x++)
                        dots[x] = fmaf(k4[i].x, k4[j].x, fmaf(k4[i].y, k4[j].y, fmaf(k4[i].z, k4[j].z, fmaf(k4[i].w, k4[j].w, dots[x]))));
#pragma unroll
                for (int i = 0; i < DG; i++)
#pragma unroll
                    for (int j = 0; j <= i; j++, x++)
                        dots[x] = fmaf(q4[i].x, k4[j].x, fmaf(q4[i].y, k4[j].y, fmaf(q4[i].z, k4[j].z, fmaf(q4[i].w, k4[j].w, dots[x]))));
            }
            // sixteen sums over the warp; lane l ends with number l & 15
            float v8[8], v4[4], v2[2];
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const bool up = (lane & 8) != 0;
                v8[i] = (up ? dots[8 + i] : dots[i]) + __shfl_xor_sync(0xffffffffu, up ? dots[i] : dots[8 + i], 8);
            }
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const bool up = (lane & 4) != 0;
                v4[i] = (up ? v8[4 + i] : v8[i]) + __shfl_xor_sync(0xffffffffu, up ? v8[i] : v8[4 + i], 4);
            }
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const bool up = (lane & 2) != 0;
                v2[i] = (up ? v4[2 + i] : v4[i]) + __shfl_xor_sync(0xffffffffu, up ? v4[i] : v4[2 + i], 2);
            }
            const bool up = (lane & 1) != 0;
            float dot = (up ? v2[1] : v2[0]) + __shfl_xor_sync(0xffffffffu, up ? v2[0] : v2[1], 1);
            dot += __shfl_xor_sync(0xffffffffu, dot, 16);
            // [0 ... 3] beta_i  [4 ... 7] beta_i e^(b_i)  [8 ... 11] e^(b_i)  [12 ... 15] e^(b_4 - b_i)  [16 ... 21] beta_i e^(b_i - b_j) k_i . k_j
            // [22 ... 31] e^(b_i - b_j) q_i . k_j
            const float* be = s_step + buf * 2 * DRUN + warp * DG;
            const float* lg = be + DRUN;
            const float bs[DG] = {lg[0], lg[0] + lg[1], lg[0] + lg[1] + lg[2], lg[0] + lg[1] + lg[2] + lg[3]};
            const int n = lane & 15;
            if (lane < 16) {
                const int i = n & 3;
                const float ei = CH ? 1.f : expf(i == 0 ? bs[0] : i == 1 ? bs[1] : i == 2 ? bs[2] : bs[3]);
                float rest = 0.f;                     // b_4 - b_i, added up and not subtracted
                for (int e = i + 1; e < DG; e++) rest += lg[e];
                s_coef[warp * 32 + n] = n < 4 ? be[i] : n < 8 ? be[i] * ei : n < 12 ? ei : CH ? 1.f : expf(rest);
            } else {
                // pair number n: j < i of the keys, then j <= i of queries and keys
                const int i = n < 6 ? (n < 1 ? 1 : n < 3 ? 2 : 3) : (n < 7 ? 0 : n < 9 ? 1 : n < 12 ? 2 : 3);
                const int j = n < 6 ? n - i * (i - 1) / 2 : n - 6 - i * (i + 1) / 2;
                float decay = 0.f;                    // b_i - b_j, the same
                for (int e = j + 1; e <= i; e++) decay += lg[e];
                s_coef[warp * 32 + 16 + n] = dot * (CH ? 1.f : expf(decay)) * (n < 6 ? be[i] : 1.f);
            }
        }
        __syncthreads();
        const int groups = (min(DRUN, cnt - t0) + DG - 1) / DG;
        for (int gr = 0; gr < groups; gr++) {
            const float* row = run + gr * DG * ROWLEN + kp * 4;
            float kr[DG][RPT];
            float hk[DG][4], hq[DG][4];
#pragma unroll
            for (int i = 0; i < DG; i++)
#pragma unroll
                for (int c = 0; c < 4; c++) hk[i][c] = 0.f, hq[i][c] = 0.f;
#pragma unroll
            for (int m0 = 0; m0 < RPT; m0 += 4) {
#pragma unroll
                for (int i = 0; i < DG; i++) {
                    const float4 k4 = *reinterpret_cast<const float4*>(row + i * ROWLEN + m0 * KP);
                    const float4 q4 = *reinterpret_cast<const float4*>(row + i * ROWLEN + NP + m0 * KP);
                    kr[i][m0] = k4.x, kr[i][m0 + 1] = k4.y, kr[i][m0 + 2] = k4.z, kr[i][m0 + 3] = k4.w;
                    const float qi[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int z = 0; z < 4; z++)
#pragma unroll
                        for (int c = 0; c < 4; c++) {
                            hk[i][c] = fmaf(kr[i][m0 + z], sreg[m0 + z][c], hk[i][c]);
                            hq[i][c] = fmaf(qi[z], sreg[m0 + z][c], hq[i][c]);
                        }
                }
            }
            // Sums over the threads of a column group.  On the way every thread drops what another one
            // carries on: bits 0 and 1 of kp pick the column, bit 2 the product with the keys or the queries.
            float r2[2 * DG][2], r1[2 * DG], rr[DG];
#pragma unroll
            for (int i = 0; i < DG; i++)
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    r2[i][c] = (b0 ? hk[i][2 + c] : hk[i][c]) + __shfl_xor_sync(0xffffffffu, b0 ? hk[i][c] : hk[i][2 + c], 1);
                    r2[DG + i][c] = (b0 ? hq[i][2 + c] : hq[i][c]) + __shfl_xor_sync(0xffffffffu, b0 ? hq[i][c] : hq[i][2 + c], 1);
                }
#pragma unroll
            for (int i = 0; i < 2 * DG; i++)
                r1[i] = (b1 ? r2[i][1] : r2[i][0]) + __shfl_xor_sync(0xffffffffu, b1 ? r2[i][0] : r2[i][1], 2);
#pragma unroll
            for (int i = 0; i < DG; i++) {
                rr[i] = (b2 ? r1[DG + i] : r1[i]) + __shfl_xor_sync(0xffffffffu, b2 ? r1[i] : r1[DG + i], 4);
                rr[i] += __shfl_xor_sync(0xffffffffu, rr[i], 8);
                if (KP == 32) rr[i] += __shfl_xor_sync(0xffffffffu, rr[i], 16);
            }
            float cf[32];
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const float4 c4 = *reinterpret_cast<const float4*>(s_coef + gr * 32 + i * 4);
                cf[4 * i] = c4.x, cf[4 * i + 1] = c4.y, cf[4 * i + 2] = c4.z, cf[4 * i + 3] = c4.w;
            }
            // (threads of the queries' half go through the same motions with their own sums; their u is not used)
            float u[DG];
            const float* vrow = run + gr * DG * ROWLEN + V_AT + cg * 4 + my_col;
            u[0] = cf[0] * vrow[0] - cf[4] * rr[0];
            u[1] = cf[1] * vrow[ROWLEN] - cf[5] * rr[1] - cf[16] * u[0];
            u[2] = cf[2] * vrow[2 * ROWLEN] - cf[6] * rr[2] - cf[17] * u[0] - cf[18] * u[1];
            u[3] = cf[3] * vrow[3 * ROWLEN] - cf[7] * rr[3] - cf[19] * u[0] - cf[20] * u[1] - cf[21] * u[2];
#pragma unroll
            for (int i = 0; i < DG; i++) {
                if (!b2 && !b3 && kp < 16) s_u[i * DCOLS + cg * 4 + my_col] = cf[12 + i] * u[i];
                const float other = __shfl_xor_sync(0xffffffffu, u[i], 4);
                u[i] = b2 ? other : u[i];
            }
            __syncwarp();                             // a column group's threads lie in one warp
            if (b2 && !b3 && kp < 16 && col + my_col < dv) {
                const float out[DG] = {cf[8] * rr[0] + cf[22] * u[0], cf[9] * rr[1] + cf[23] * u[0] + cf[24] * u[1],
                                       cf[10] * rr[2] + cf[25] * u[0] + cf[26] * u[1] + cf[27] * u[2],
                                       cf[11] * rr[3] + cf[28] * u[0] + cf[29] * u[1] + cf[30] * u[2] + cf[31] * u[3]};
                const int t = t0 + gr * DG;
#pragma unroll
                for (int i = 0; i < DG; i++)
                    if (t + i < cnt) o[(size_t)(tok0 + t + i) * p.H * dv + (size_t)h * dv + col + my_col] = out[i];
            }
            float uw[DG][4];
#pragma unroll
            for (int i = 0; i < DG; i++) {
                const float4 u4 = *reinterpret_cast<const float4*>(s_u + i * DCOLS + cg * 4);
                uw[i][0] = u4.x, uw[i][1] = u4.y, uw[i][2] = u4.z, uw[i][3] = u4.w;
            }
            __syncwarp();                             // read by all before the next group's are written
            if (CH) {                                 // the decays and the keys of the update, row by row
#pragma unroll
                for (int m0 = 0; m0 < RPT; m0 += 4) {
                    const float4 g4 = *reinterpret_cast<const float4*>(s_g4 + gr * NP + kp * 4 + m0 * KP);
                    const float gm[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
                    for (int z = 0; z < 4; z++)
#pragma unroll
                        for (int c = 0; c < 4; c++) sreg[m0 + z][c] *= gm[z];
#pragma unroll
                    for (int i = 0; i < DG; i++) {
                        const float4 k4 = *reinterpret_cast<const float4*>(row + i * ROWLEN + 2 * NP + m0 * KP);
                        const float km[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                        for (int z = 0; z < 4; z++)
#pragma unroll
                            for (int c = 0; c < 4; c++) sreg[m0 + z][c] = fmaf(km[z], uw[i][c], sreg[m0 + z][c]);
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < (CH ? 0 : RPT); m++)
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    float x = cf[11] * sreg[m][c];
#pragma unroll
                    for (int i = 0; i < DG; i++) x = fmaf(kr[i][m], uw[i][c], x);
                    sreg[m][c] = x;
                }
        }
    }
#pragma unroll
    for (int m = 0; m < RPT; m++) {
        const int n = (m / 4) * 4 * KP + kp * 4 + m % 4;
        if (n >= d) continue;
        if (vec_state && col < dv) {
            *reinterpret_cast<float4*>(S + (size_t)n * dv + col) = make_float4(sreg[m][0], sreg[m][1], sreg[m][2], sreg[m][3]);
        } else {
#pragma unroll
            for (int c = 0; c < 4; c++)
                if (col + c < dv) S[(size_t)n * dv + col + c] = sreg[m][c];
        }
    }
}

bool aligned16(const void* p) { return (uintptr_t)p % 16 == 0; }

}  // namespace

// proj: [T, ld] 32-bit: q (G * d columns), k (G * d), v (H * dv), b and a (a column a value head) from b_at and
// a_at; taps_w: [taps, channels]; state: (taps - 1) * channels floats a slot from the pointer given; out: [T, channels]
// 32-bit; step: [T, 2 H] 32-bit (beta, then the decay's logarithm).  `shift`: the step brings one token a sequence and the state moves on here.
// With `decay` not null there is a decay a channel: a_rows [T, lda] holds a (H * d columns), dt_bias [H * d], and decay
// [T, H * d] receives the decays (a_at is not read then).
MOE_API int moe_delta_prepare(const float* proj, long long ld, int b_at, int a_at, const float* taps_w, int taps,
                              float* state, long long state_pitch, const float* a_log, const float* dt_bias,
                              const int* seq_of_token, const int* cu_seqlens, const int* slots, int num_tokens, int H,
                              int G, int d, int dv, float eps, float q_scale, int shift, float* out, float* step,
                              const float* a_rows, long long lda, float* decay, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    const long long channels = 2LL * G * d + (long long)H * dv;
    if (!proj || !taps_w || !a_log || !dt_bias || !seq_of_token || !cu_seqlens || !slots || !out || !step || H <= 0 || G <= 0 ||
        H % G || d <= 0 || d > DP_MAX_D || dv <= 0 || taps < 1 || taps > 16 || (taps > 1 && !state) || ld < channels ||
        b_at < 0 || b_at + H > ld || (decay ? !a_rows || lda < (long long)H * d : a_at < 0 || a_at + H > ld) || (taps > 1 && state_pitch < (taps - 1) * channels))
        return (int)cudaErrorInvalidValue;
    const DeltaPrep p{proj, ld, b_at, a_at, taps_w, state, state_pitch, a_log, dt_bias, seq_of_token, cu_seqlens, slots,
                      num_tokens, taps, H, G, d, dv, shift, eps, q_scale, out, step, a_rows, lda, decay};
    const bool vec = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && state_pitch % 4 == 0 && aligned16(proj) && aligned16(taps_w) &&
                     aligned16(state) && aligned16(out) &&
                     (!decay || (lda % 4 == 0 && aligned16(a_rows) && aligned16(decay) && aligned16(dt_bias)));
    const int per = vec ? 128 : 32;
    const int items = 2 * G + (H * dv + per - 1) / per + 1 + (decay ? (H * d + per - 1) / per : 0);
    // few tokens: a warp an item; many: a block a token
    const dim3 grid(num_tokens, num_tokens >= 128 ? 1 : (items + DP_WARPS - 1) / DP_WARPS);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
#define PREP(W_, T_) return launch_pdl(delta_prepare_kernel<W_, T_>, grid, dim3(DP_WARPS * 32), 0, stream, p)
    if (vec) {
        if (taps == 2) PREP(4, 2);
        if (taps == 3) PREP(4, 3);
        if (taps == 4) PREP(4, 4);
        PREP(4, 0);
    }
    if (taps == 4) PREP(1, 4);
    PREP(1, 0);
#undef PREP
}

// One token a sequence.  qkv, step: as moe_delta_prepare leaves them; state: H * d * dv floats a slot from the pointer
// given; decay: [T, H * d] or null; gate: [T, H * dv] 32-bit logits, rows of ldg, through gate_fn (GATE_*); norm_w: [H * dv]; out: [T, H * dv] in out_dt (rows of no
// sequence become zeros).  Returns -1, with nothing launched, for sizes it does not take.
MOE_API int moe_delta_step(const float* qkv, const float* step, float* state, long long state_pitch, const float* gate,
                           long long ldg, const float* norm_w, float norm_eps, const int* seq_of_token,
                           const int* cu_seqlens, const int* slots, int num_tokens, int num_seqs, int H, int G, int d,
                           int dv, const float* decay, int gate_fn, void* out, int out_dt, cudaStream_t stream) {
    if (num_seqs <= 0 || num_tokens <= 0) return 0;
    if (!qkv || !step || !state || !gate || !norm_w || !seq_of_token || !cu_seqlens || !slots || !out || H <= 0 || G <= 0 ||
        H % G || d <= 0 || dv <= 0 || ldg < (long long)H * dv || state_pitch < (long long)H * d * dv || num_seqs > 65535)
        return (int)cudaErrorInvalidValue;
    if (dv % 4 || dv > 512 || d > 256 || state_pitch % 4 || !aligned16(state)) return -1;
    const int cg = dv / 4, kp = 256 / cg, units = (d + kp - 1) / kp;
    const size_t smem = ((size_t)2 * ((d + 1) / 2 * 2) + dv + (size_t)kp * dv + (decay ? d : 0)) * sizeof(float);
    if (units > 32 || smem > 48 * 1024 || d % 2) return -1;
    const DeltaSeq p{qkv, step, state, state_pitch, cu_seqlens, slots, H, G, d, dv, decay};
#define STEP_C(OT_, U_, C_)                                                                                            \
    return launch_pdl(delta_step_kernel<OT_, U_, C_>, dim3(H, num_seqs), dim3(256), smem, stream, p, gate, ldg, norm_w, norm_eps, \
                      seq_of_token, num_tokens, gate_fn, (OT_*)out)
#define STEP(OT_, U_)                                                                                                  \
    do {                                                                                                               \
        if (decay) STEP_C(OT_, U_, true);                                                                              \
        STEP_C(OT_, U_, false);                                                                                        \
    } while (0)
#define STEP_U(OT_)                                                                                                    \
    do {                                                                                                               \
        if (units <= 4) STEP(OT_, 4);                                                                                  \
        if (units <= 8) STEP(OT_, 8);                                                                                  \
        if (units <= 16) STEP(OT_, 16);                                                                                \
        STEP(OT_, 32);                                                                                                 \
    } while (0)
    if (out_dt == DT_F32) STEP_U(float);
    STEP_U(__nv_bfloat16);
#undef STEP_U
#undef STEP
#undef STEP_C
}

// Several tokens a sequence; o: [T, H * dv] 32-bit (rows of no sequence are left alone).
MOE_API int moe_delta_scan(const float* qkv, const float* step, float* state, long long state_pitch, const int* cu_seqlens,
                           const int* slots, int num_seqs, int H, int G, int d, int dv, const float* decay, float* o,
                           cudaStream_t stream) {
    if (num_seqs <= 0) return 0;
    if (!qkv || !step || !state || !cu_seqlens || !slots || !o || H <= 0 || G <= 0 || H % G || d <= 0 || d > 256 || dv <= 0 ||
        state_pitch < (long long)H * d * dv || H > 65535 || num_seqs > 65535)
        return (int)cudaErrorInvalidValue;
    const DeltaSeq p{qkv, step, state, state_pitch, cu_seqlens, slots, H, G, d, dv, decay};
    // few blocks: the narrow form puts twice as many on the SMs
    const bool narrow = d > 64 && (long long)((dv + dcols(16) - 1) / dcols(16)) * H * num_seqs * 2 <= scan_sms();
    const int cols = dcols(narrow ? 32 : 16);
    const dim3 grid((dv + cols - 1) / cols, H, num_seqs);
    const bool vec = d % 4 == 0 && dv % 4 == 0 && aligned16(qkv) && aligned16(decay);
    // An ordinary launch: blocks that are placed while the kernel before still occupies some SMs end up several to
    // an SM beside empty ones, and a scan is as slow as its most crowded SM.
#define SCAN_V(RPT_, KP_, V_, C_)                                                                                      \
    do {                                                                                                               \
        const size_t smem = scan_smem(delta_scan_floats<RPT_, KP_, C_>() * sizeof(float), (long long)grid.x * grid.y * grid.z); \
        if (smem > 48 * 1024) {                                                                                        \
            cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<RPT_, KP_, V_, C_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                       \
        }                                                                                                              \
        delta_scan_kernel<RPT_, KP_, V_, C_><<<grid, DTHREADS, smem, stream>>>(p, o);                                  \
        return launch_status();                                                                                        \
    } while (0)
#define SCAN(RPT_, KP_)                                                                                                \
    do {                                                                                                               \
        if (decay) {                                                                                                   \
            if (vec) SCAN_V(RPT_, KP_, true, true);                                                                    \
            SCAN_V(RPT_, KP_, false, true);                                                                            \
        }                                                                                                              \
        if (vec) SCAN_V(RPT_, KP_, true, false);                                                                       \
        SCAN_V(RPT_, KP_, false, false);                                                                               \
    } while (0)
    if (d <= 64) SCAN(4, 16);
    if (narrow) {
        if (d <= 128) SCAN(4, 32);
        SCAN(8, 32);
    }
    if (d <= 128) SCAN(8, 16);
    SCAN(16, 16);
#undef SCAN
#undef SCAN_V
}
