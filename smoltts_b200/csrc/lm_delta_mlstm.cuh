// Two further recurrences of the hybrid language-model engine (included by lm_kernels.cu after lm_sigmoid_linear.cuh):
//   - the gated delta rule (short convolutions in front, one decay and one step size per head and token, unit queries and
//     keys, state [dim, vdim] per head),
//   - the mLSTM's gates (exponential input gate, sigmoid forget gate, running maximum); its matrix memory runs on the gated
//     linear recurrence's scan with the unit column, its end on gla_out_kernel.
// Everything here is fp32.
#pragma once

namespace smol {
namespace lm {

// ---------------------------------------------------------------------------------------------------------------------
// Gated delta rule.  proj row layout: q | k [G*d each] | v | gate [H*dv each] | step [H] | decay [H]; G key heads serve H / G heads each.
//   q, k, v: short convolution and silu;  q <- q / sqrt(sum q^2 + unit_eps) * q_scale,  k <- k / sqrt(sum k^2 + unit_eps)
//   b = sigmoid(step),  w = exp(-exp(a_log) * softplus(decay + dt_bias))
//   S <- w S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q
struct GatedDeltaArgs {
    const float* proj;
    int n_in, H, G, d, dv, n_tokens;
    float q_scale, unit_eps;
    const float *a_log, *dt_bias;
    const int32_t* tok_seq;
    ConvIo conv;                       // channels q | k | v; its sequences and slots are the recurrence's
    size_t state_off;
    int32_t* err;
};

// Blocks (token, group of 4 warps).  The first G warps of a token take a key head each: convolved q and k, their lengths and
// their product; the others take 64 value channels each.  qkv [T][2 G d + H dv]: unit q (scaled) | unit k | v;
// head: decay [T][H], step [T][H], then k.q [T][G].
constexpr int kGatedDeltaCols = 64;
__global__ void __launch_bounds__(128) gated_delta_prep_kernel(const GatedDeltaArgs A, const float* __restrict__ slots, float* __restrict__ qkv,
                                                               float* __restrict__ head) {
    const int t = blockIdx.x, warp = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    const ConvIo& C = A.conv;
    const int s = A.tok_seq[t], r = t - C.seq_start[s], pos0 = C.seq_pos0[s], slot = C.seq_slot[s];
    if (slot < 0 || slot >= C.n_slots) {
        if (threadIdx.x == 0) atomicExch(A.err, 2);
        return;
    }
    const float* before = slots + (size_t)slot * C.slot_floats + C.conv_off;
    const int gd = A.G * A.d;
    float* row = qkv + (size_t)t * C.ch;
    for (int h = threadIdx.x; blockIdx.y == 0 && h < A.H; h += blockDim.x) {
        const float* p = A.proj + (size_t)t * A.n_in + C.ch + A.H * A.dv + h;
        head[(size_t)t * A.H + h] = expf(-expf(A.a_log[h]) * softplus_(p[A.H] + A.dt_bias[h]));
        head[(size_t)(A.n_tokens + t) * A.H + h] = sigmoidf_(p[0]);
    }
    if (warp < A.G) {
        constexpr int R = 8;               // key sizes up to 256
        float q[R], k[R];
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
        for (int e = 0; e < R; ++e) {
            const int c = lane + 32 * e;
            q[e] = k[e] = 0.0f;
            if (c < A.d) {
                q[e] = conv_channel(C, before, t, r, pos0, warp * A.d + c);
                k[e] = conv_channel(C, before, t, r, pos0, gd + warp * A.d + c);
            }
            qq = fmaf(q[e], q[e], qq);
            kk = fmaf(k[e], k[e], kk);
            qk = fmaf(q[e], k[e], qk);
        }
#pragma unroll
        for (int x = 16; x > 0; x >>= 1) {
            qq += __shfl_xor_sync(0xffffffffu, qq, x);
            kk += __shfl_xor_sync(0xffffffffu, kk, x);
            qk += __shfl_xor_sync(0xffffffffu, qk, x);
        }
        const float rq = A.q_scale / sqrtf(qq + A.unit_eps), rk = 1.0f / sqrtf(kk + A.unit_eps);
#pragma unroll
        for (int e = 0; e < R; ++e) {
            const int c = lane + 32 * e;
            if (c < A.d) {
                row[warp * A.d + c] = q[e] * rq;
                row[gd + warp * A.d + c] = k[e] * rk;
            }
        }
        if (lane == 0) head[(size_t)2 * A.n_tokens * A.H + (size_t)t * A.G + warp] = qk * rq * rk;
        return;
    }
    const int c0 = (warp - A.G) * kGatedDeltaCols;
#pragma unroll
    for (int e = 0; e < kGatedDeltaCols / 32; ++e) {
        const int c = c0 + lane + 32 * e;
        if (c < A.H * A.dv) row[2 * gd + c] = conv_channel(C, before, t, r, pos0, 2 * gd + c);
    }
}

// The scan, organised like gla_scan_kernel: a head's value columns cut into groups, one block per (sequence, head, group), L
// lanes per column with the state's rows in registers, q | k | v and the scalars staged kDeltaChunk tokens at a time by cp.async.
// With S the state before the token, both sums over the key rows are taken from S at once -- seen = S^T k and S^T q -- and
//   u = b (v - w seen),   o = w (S^T q) + u (k.q),   S <- w S + k u^T,
// which is the rule above with the read-out of the new state written out: one reduction per token instead of two in a row.
// The blocks of a sequence also bring the slot's convolution inputs up to date.
__host__ __device__ constexpr int gated_delta_buf_floats(int DK) { return kDeltaChunk * (2 * DK + gla_block_cols(DK) + 4); }

template <int DK, int VEC>
__device__ __forceinline__ void gated_delta_stage(const GatedDeltaArgs& A, const float* __restrict__ qkv, const float* __restrict__ head, float* buf, int c0,
                                                  int n, int h, int j0, int nc) {
    constexpr int CB = gla_block_cols(DK), PL = kDeltaChunk * DK;
    const int d = A.d, dq = d / VEC, ncq = (nc + VEC - 1) / VEC, hs = h / (A.H / A.G), ch = A.conv.ch;
    for (int idx = threadIdx.x; idx < n * dq; idx += blockDim.x) {
        const int tt = idx / dq, i = (idx - tt * dq) * VEC;
        const float* src = qkv + (size_t)(c0 + tt) * ch + hs * d + i;
        cp_async_f<VEC>(buf + tt * DK + i, src);
        cp_async_f<VEC>(buf + PL + tt * DK + i, src + A.G * d);
    }
    for (int idx = threadIdx.x; idx < n * ncq; idx += blockDim.x) {
        const int tt = idx / ncq, j = (idx - tt * ncq) * VEC;
        cp_async_f<VEC>(buf + 2 * PL + tt * CB + j, qkv + (size_t)(c0 + tt) * ch + 2 * A.G * d + h * A.dv + j0 + j);
    }
    float* sc = buf + 2 * PL + kDeltaChunk * CB;        // per token: decay, step, k.q, unused
    for (int idx = threadIdx.x; idx < 3 * n; idx += blockDim.x) {
        const int tt = idx / 3, what = idx - tt * 3;
        const float* src = what < 2 ? head + (size_t)(what * A.n_tokens + c0 + tt) * A.H + h
                                    : head + (size_t)2 * A.n_tokens * A.H + (size_t)(c0 + tt) * A.G + hs;
        cp_async_f<1>(sc + tt * 4 + what, src);
    }
}

template <int DK>
__global__ void __launch_bounds__(gla_block_cols(DK) * gla_lanes(DK)) gated_delta_scan_kernel(const GatedDeltaArgs A, const float* __restrict__ qkv,
                                                                                              const float* __restrict__ head, float* state_pool,
                                                                                              float* __restrict__ o_raw) {
    constexpr int L = gla_lanes(DK), CB = gla_block_cols(DK), RV = DK / L / 4, PL = kDeltaChunk * DK;
    constexpr int kBuf = gated_delta_buf_floats(DK);
    extern __shared__ __align__(16) float sh[];
    const ConvIo& C = A.conv;
    const int d = A.d, dv = A.dv, NS = (dv + CB - 1) / CB;
    const int part = blockIdx.x % (A.H * NS), seq = blockIdx.x / (A.H * NS);
    const int h = part / NS, j0 = (part % NS) * CB;
    const int nc = min(CB, dv - j0);
    const int col = threadIdx.x / L, q = threadIdx.x % L, j = j0 + col;
    const int t0 = C.seq_start[seq], t1 = C.seq_start[seq + 1];
    const int slot = C.seq_slot[seq];
    if (slot < 0 || slot >= C.n_slots) {
        if (threadIdx.x == 0) atomicExch(A.err, 2);
        return;
    }
    const bool vec = d % 4 == 0 && dv % 4 == 0 && reinterpret_cast<uintptr_t>(qkv) % 16 == 0;
    for (int i = threadIdx.x; i < 2 * kBuf; i += blockDim.x) sh[i] = 0.0f;      // padded channels and columns stay zero for good
    __syncthreads();
    if (vec) gated_delta_stage<DK, 4>(A, qkv, head, sh, t0, min(kDeltaChunk, t1 - t0), h, j0, nc);
    else gated_delta_stage<DK, 1>(A, qkv, head, sh, t0, min(kDeltaChunk, t1 - t0), h, j0, nc);
    cp_async_commit();
    float* st = state_pool + (size_t)slot * C.slot_floats + A.state_off + (size_t)h * d * dv;
    float S[RV][4];
    const bool fresh = C.seq_pos0[seq] == 0;
#pragma unroll
    for (int e = 0; e < RV; ++e)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = 4 * (e * L + q) + x;
            S[e][x] = (!fresh && i < d && j < dv) ? st[(size_t)i * dv + j] : 0.0f;
        }
    if (C.taps > 1)
        for (int c = part * blockDim.x + threadIdx.x; c < C.ch; c += A.H * NS * blockDim.x) conv_state_update(C, state_pool, seq, c);
    int cur = 0;
    for (int c0 = t0; c0 < t1; c0 += kDeltaChunk, cur ^= 1) {
        const int n = min(kDeltaChunk, t1 - c0);
        cp_async_wait<0>();
        __syncthreads();                          // this chunk has landed; every thread is done with the other buffer
        if (c0 + kDeltaChunk < t1) {
            const int nn = min(kDeltaChunk, t1 - c0 - kDeltaChunk);
            if (vec) gated_delta_stage<DK, 4>(A, qkv, head, sh + (cur ^ 1) * kBuf, c0 + kDeltaChunk, nn, h, j0, nc);
            else gated_delta_stage<DK, 1>(A, qkv, head, sh + (cur ^ 1) * kBuf, c0 + kDeltaChunk, nn, h, j0, nc);
            cp_async_commit();
        }
        const float* b = sh + cur * kBuf;
        const float4* s4 = reinterpret_cast<const float4*>(b) + q;      // piece e of q of token tt: s4[(tt*DK)/4 + e*L]; k: PL / 4 further on
        const float* s_v = b + 2 * PL + col;
        const float4* s_sc = reinterpret_cast<const float4*>(b + 2 * PL + kDeltaChunk * CB);
        auto token = [&](int tt) {
            const float v = s_v[tt * CB];
            const float4 sc = s_sc[tt];                                 // decay, step, k.q
            float4 qv[RV], kv[RV];
            float ka = 0.0f, kb = 0.0f, qa = 0.0f, qb = 0.0f;
#pragma unroll
            for (int e = 0; e < RV; ++e) {
                qv[e] = s4[tt * (DK / 4) + e * L];
                kv[e] = s4[PL / 4 + tt * (DK / 4) + e * L];
                ka = fmaf(kv[e].x, S[e][0], ka); qa = fmaf(qv[e].x, S[e][0], qa);
                kb = fmaf(kv[e].y, S[e][1], kb); qb = fmaf(qv[e].y, S[e][1], qb);
                ka = fmaf(kv[e].z, S[e][2], ka); qa = fmaf(qv[e].z, S[e][2], qa);
                kb = fmaf(kv[e].w, S[e][3], kb); qb = fmaf(qv[e].w, S[e][3], qb);
            }
            float seen = ka + kb, read = qa + qb;
#pragma unroll
            for (int x = 1; x < L; x <<= 1) {
                const float y = __shfl_xor_sync(0xffffffffu, seen, x), z = __shfl_xor_sync(0xffffffffu, read, x);
                seen += y;
                read += z;
            }
            const float u = sc.y * fmaf(-sc.x, seen, v);
            if (q == 0 && j < dv) o_raw[(size_t)(c0 + tt) * A.H * dv + h * dv + j] = fmaf(sc.x, read, u * sc.z);
#pragma unroll
            for (int e = 0; e < RV; ++e) {
                S[e][0] = fmaf(sc.x, S[e][0], kv[e].x * u);
                S[e][1] = fmaf(sc.x, S[e][1], kv[e].y * u);
                S[e][2] = fmaf(sc.x, S[e][2], kv[e].z * u);
                S[e][3] = fmaf(sc.x, S[e][3], kv[e].w * u);
            }
        };
        if (n == kDeltaChunk) {
#pragma unroll 8
            for (int tt = 0; tt < kDeltaChunk; ++tt) token(tt);         // unrolled: the next tokens' vectors are read ahead
        } else {
            for (int tt = 0; tt < n; ++tt) token(tt);
        }
    }
#pragma unroll
    for (int e = 0; e < RV; ++e)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = 4 * (e * L + q) + x;
            if (i < d && j < dv) st[(size_t)i * dv + j] = S[e][x];
        }
}

// ---------------------------------------------------------------------------------------------------------------------
// mLSTM gates.  Per head, with i = cap tanh((input row + bias) / cap) and f = ln sigmoid(cap tanh((forget row + bias) / cap)):
//   m_t = max(f_t + m_(t-1), i_t),  the memory's decay exp(f_t + m_(t-1) - m_t) and write weight exp(i_t - m_t), and the
//   denominator's floor exp(-m_t).  m starts at 0 and lives in the slot ([H] at m_off).
// A token acts on m as m -> max(F + m, I) with (F, I) = (f, i); two tokens one after the other as (F1 + F2, max(I1 + F2, I2)),
// so the maxima of a whole tile of tokens come from a parallel scan.  One block per (sequence, head).  Rounding in m is harmless:
// decay, weight and floor are all formed from the same m, which only scales numerator and denominator.
struct MlstmArgs {
    const float* proj;
    int n_in, H, n_tokens;
    size_t gate_off;                   // column of the input rows; the forget rows follow
    float cap;
    const float *i_bias, *f_bias;      // [H]
    const int32_t *seq_start, *seq_pos0, *seq_slot;
    size_t slot_floats, m_off;
    int n_slots;
    int32_t* err;
};
constexpr int kMlstmTile = 256;

// head: decay [T][H], write weight [T][H], floor [T][H]
__global__ void __launch_bounds__(kMlstmTile) mlstm_gate_kernel(const MlstmArgs A, float* __restrict__ slots, float* __restrict__ head) {
    __shared__ float wf[kMlstmTile / 32], wi[kMlstmTile / 32], ms[kMlstmTile + 1];
    const int s = blockIdx.x / A.H, h = blockIdx.x % A.H, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t0 = A.seq_start[s], t1 = A.seq_start[s + 1], slot = A.seq_slot[s];
    if (slot < 0 || slot >= A.n_slots) {
        if (threadIdx.x == 0) atomicExch(A.err, 2);
        return;
    }
    float* m_at = slots + (size_t)slot * A.slot_floats + A.m_off + h;
    float m = A.seq_pos0[s] == 0 ? 0.0f : *m_at;
    const float ib = A.i_bias[h], fb = A.f_bias[h];
    const size_t TH = (size_t)A.n_tokens * A.H;
    for (int base = t0; base < t1; base += blockDim.x) {
        const int t = base + threadIdx.x;
        const bool in = t < t1;
        float f = 0.0f, i = -INFINITY;                 // beyond the last token: leaves m as it is
        if (in) {
            const float* p = A.proj + (size_t)t * A.n_in + A.gate_off + h;
            i = A.cap * tanhf((p[0] + ib) / A.cap);
            f = log_sigmoid_(A.cap * tanhf((p[A.H] + fb) / A.cap));
        }
        float F = f, I = i;                            // this token and those before it in the warp
#pragma unroll
        for (int x = 1; x < 32; x <<= 1) {
            const float f0 = __shfl_up_sync(0xffffffffu, F, x), i0 = __shfl_up_sync(0xffffffffu, I, x);
            if (lane >= x) {
                I = fmaxf(i0 + F, I);
                F += f0;
            }
        }
        __syncthreads();                               // the previous tile's shared values have been read
        if (lane == 31) { wf[warp] = F; wi[warp] = I; }
        __syncthreads();
        float mw = m;                                  // the maximum as this warp's first token finds it
        for (int w = 0; w < warp; ++w) mw = fmaxf(wf[w] + mw, wi[w]);
        const float mt = fmaxf(F + mw, I);
        ms[threadIdx.x + 1] = mt;
        if (threadIdx.x == 0) ms[0] = m;
        __syncthreads();
        const float before = ms[threadIdx.x];
        if (in) {
            head[(size_t)t * A.H + h] = expf(f + before - mt);
            head[TH + (size_t)t * A.H + h] = expf(i - mt);
            head[2 * TH + (size_t)t * A.H + h] = expf(-mt);
        }
        m = ms[min((int)blockDim.x, t1 - base)];
    }
    if (threadIdx.x == 0 && t1 > t0) *m_at = m;
}

}  // namespace lm
}  // namespace smol
