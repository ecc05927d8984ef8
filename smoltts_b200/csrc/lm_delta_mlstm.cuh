// Two further recurrences of the hybrid language-model engine (included by lm_kernels.cu after lm_sigmoid_linear.cuh):
//   - the gated delta rule (short convolutions in front, one decay and one step size per head and token, unit queries and
//     keys, state [dim, vdim] per head),
//   - the mLSTM (matrix memory with exponential input gate, sigmoid forget gate, running maximum; state [dim, vdim] and a key
//     sum per head),
// both on a scan that takes four tokens at a time.  Their ends run on gla_out_kernel.  Everything here is fp32.
#pragma once

namespace smol {
namespace lm {

// ---------------------------------------------------------------------------------------------------------------------
// The scan of a recurrence with one decay w and one step b per head and token,
//   S <- w S;  u = b (v - S^T k)  [DELTA]  or  u = b v;  S <- S + k u^T;  o = S^T q,
// four tokens at a time.  With S the state before the group, e_j the u of token j decayed up to the current one and P the product of
// the decays so far, token i of the group follows from sums over the key rows that all read the same S:
//   S^T k_i before its write = P_i (S^T k_i) + sum_(j<i) (k_j.k_i) e_j,    o_i = P_i (S^T q_i) + sum_(j<=i) (k_j.q_i) e_j,
// and the group leaves  S <- P_3 S + sum_j k_j e_j^T.  So the eight sums of a group are reduced across lanes side by side (a
// chain of single tokens pays that latency every token), and only the small triangle above is sequential.  Groups count from
// the sequence's first token of the step; a group's missing tokens have decay 1 and step 0.
// Organised like gla_scan_kernel: a head's value columns cut into parts, one block per (sequence, head, part), L lanes per
// column with the state's rows in registers; q | k | v and the scalars come by cp.async, the next chunk while the current one
// is computed.
constexpr int kScanGroup = 4;
constexpr int kPairFloats = 2 * kScanGroup;     // per token and key head: k_j.k_i of the group's earlier tokens j, then k_j.q_i up to its own
struct GroupScanArgs {
    int H, G, d, dv;                   // H value heads over G query / key heads
    const float *q_src, *k_src, *v_src;         // token t: q_src + t * q_ld + g * d, k likewise, v_src + t * v_ld + h * dv
    int q_ld, k_ld, v_ld;
    const float *head, *pairs;         // [T][H][2] decay and step, [T][G][kPairFloats]
    float q_scale;
    const int32_t *seq_start, *seq_pos0, *seq_slot;
    size_t slot_floats, state_off;
    int n_slots;
    int32_t* err;
    // A further state column per head whose value is 1 for every token (the sum of the written keys): its rows live at unit_off
    // inside the slot ([H][d]), its product with the query goes to unit_out[t * H + h].  nullptr: none.
    float* unit_out;
    size_t unit_off;
    ConvIo conv;                       // taps > 1: the blocks of a sequence also bring these inputs in the slot up to date
};
__host__ __device__ constexpr int group_scan_chunk(int DK) { return DK <= 128 ? 32 : 16; }      // tokens per buffer
__host__ __device__ constexpr int group_scan_buf_floats(int DK) { return group_scan_chunk(DK) * (2 * DK + gla_block_cols(DK) + 2 + kPairFloats); }

// The products between a group's queries and keys.  One warp per (group, sequence, key head); sequences of one token are left out
// (their only product is made by the kernel in front).  DELTA: keys with keys too, and the own products are there already.
template <bool DELTA>
__global__ void __launch_bounds__(128) scan_pairs_kernel(const GroupScanArgs A, float* __restrict__ pairs) {
    const int g = blockIdx.z * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    const int t0 = A.seq_start[blockIdx.y], n_all = A.seq_start[blockIdx.y + 1] - t0, r0 = blockIdx.x * kScanGroup;
    if (g >= A.G || n_all <= 1 || r0 >= n_all) return;
    const int n = min(kScanGroup, n_all - r0);
    float kk[kScanGroup][kScanGroup], qk[kScanGroup][kScanGroup];
#pragma unroll
    for (int i = 0; i < kScanGroup; ++i)
#pragma unroll
        for (int j = 0; j < kScanGroup; ++j) kk[i][j] = qk[i][j] = 0.0f;
    for (int c = lane; c < A.d; c += 32) {
        float q[kScanGroup], k[kScanGroup];
#pragma unroll
        for (int i = 0; i < kScanGroup; ++i) {
            const size_t t = t0 + r0 + i;
            q[i] = i < n ? A.q_src[t * A.q_ld + g * A.d + c] : 0.0f;
            k[i] = i < n ? A.k_src[t * A.k_ld + g * A.d + c] : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < kScanGroup; ++i)
#pragma unroll
            for (int j = 0; j <= i; ++j) {
                if (DELTA && j < i) kk[i][j] = fmaf(k[i], k[j], kk[i][j]);
                if (!DELTA || j < i) qk[i][j] = fmaf(q[i], k[j], qk[i][j]);
            }
    }
#pragma unroll
    for (int i = 0; i < kScanGroup; ++i)
#pragma unroll
        for (int j = 0; j <= i; ++j) {
            if (DELTA && j < i) kk[i][j] = warp_sum(kk[i][j]);
            if (!DELTA || j < i) qk[i][j] = warp_sum(qk[i][j]);
            if (lane == 0 && i < n) {
                float* row = pairs + ((size_t)(t0 + r0 + i) * A.G + g) * kPairFloats;
                if (DELTA && j < i) row[j] = kk[i][j];
                if (!DELTA || j < i) row[kScanGroup + j] = qk[i][j];
            }
        }
}

template <int DK, int VEC>
__device__ __forceinline__ void group_scan_stage(const GroupScanArgs& A, float* buf, int c0, int n, int h, int j0, int nc) {
    constexpr int CB = gla_block_cols(DK), CH = group_scan_chunk(DK), PL = CH * DK;
    const int d = A.d, dq = d / VEC, ncq = (nc + VEC - 1) / VEC, g = h / (A.H / A.G);
    for (int idx = threadIdx.x; idx < n * dq; idx += blockDim.x) {
        const int tt = idx / dq, i = (idx - tt * dq) * VEC;
        cp_async_f<VEC>(buf + tt * DK + i, A.q_src + (size_t)(c0 + tt) * A.q_ld + g * d + i);
        cp_async_f<VEC>(buf + PL + tt * DK + i, A.k_src + (size_t)(c0 + tt) * A.k_ld + g * d + i);
    }
    for (int idx = threadIdx.x; idx < n * ncq; idx += blockDim.x) {
        const int tt = idx / ncq, j = (idx - tt * ncq) * VEC;
        cp_async_f<VEC>(buf + 2 * PL + tt * CB + j, A.v_src + (size_t)(c0 + tt) * A.v_ld + h * A.dv + j0 + j);
    }
    float* sc = buf + 2 * PL + CH * CB;                 // pair products [chunk][kPairFloats], then decay and step [chunk][2]
    for (int idx = threadIdx.x; idx < n * (kPairFloats / 4); idx += blockDim.x) {
        const int tt = idx / (kPairFloats / 4), x = idx % (kPairFloats / 4) * 4;
        cp_async_f<4>(sc + tt * kPairFloats + x, A.pairs + ((size_t)(c0 + tt) * A.G + g) * kPairFloats + x);
    }
    for (int idx = threadIdx.x; idx < 2 * n; idx += blockDim.x)
        cp_async_f<1>(sc + CH * kPairFloats + idx, A.head + ((size_t)(c0 + idx / 2) * A.H + h) * 2 + idx % 2);
}

template <int DK, bool DELTA>
__global__ void __launch_bounds__(gla_block_cols(DK) * gla_lanes(DK)) group_scan_kernel(const GroupScanArgs A, float* state_pool, float* __restrict__ o_raw) {
    constexpr int L = gla_lanes(DK), CB = gla_block_cols(DK), RV = DK / L / 4, CH = group_scan_chunk(DK), PL = CH * DK;
    constexpr int kBuf = group_scan_buf_floats(DK), GS = kScanGroup;
    static_assert(L >= GS && kBuf % 4 == 0, "a lane per token of a group stores its result; 16-byte buffers");
    extern __shared__ __align__(16) float sh[];
    const int d = A.d, dv = A.dv, dvs = dv + (A.unit_out ? 1 : 0), NS = (dvs + CB - 1) / CB;      // dvs: state columns
    const int part = blockIdx.x % (A.H * NS), seq = blockIdx.x / (A.H * NS);
    const int h = part / NS, j0 = (part % NS) * CB;
    const int nc = max(0, min(CB, dv - j0));
    const int col = threadIdx.x / L, q = threadIdx.x % L, j = j0 + col;
    const int t0 = A.seq_start[seq], t1 = A.seq_start[seq + 1];
    const int slot = A.seq_slot[seq];
    if (slot < 0 || slot >= A.n_slots) {
        if (threadIdx.x == 0) atomicExch(A.err, 2);
        return;
    }
    // 16-byte copies need every source to start on a 16-byte boundary: d, dv and the row lengths multiples of 4
    const bool vec = (d % 4 == 0) && (dv % 4 == 0) && (A.q_ld % 4 == 0) && (A.k_ld % 4 == 0) && (A.v_ld % 4 == 0) &&
                     ((reinterpret_cast<uintptr_t>(A.q_src) | reinterpret_cast<uintptr_t>(A.k_src) | reinterpret_cast<uintptr_t>(A.v_src)) % 16 == 0);
    for (int i = threadIdx.x; i < 2 * kBuf; i += blockDim.x) sh[i] = 0.0f;      // padded channels and columns stay zero for good
    if (dvs > dv && dv >= j0 && dv < j0 + CB) {                                 // ... and the unit column one
        __syncthreads();
        for (int i = threadIdx.x; i < 2 * CH; i += blockDim.x) sh[(i / CH) * kBuf + 2 * PL + (i % CH) * CB + dv - j0] = 1.0f;
    }
    __syncthreads();
    if (vec) group_scan_stage<DK, 4>(A, sh, t0, min(CH, t1 - t0), h, j0, nc);
    else group_scan_stage<DK, 1>(A, sh, t0, min(CH, t1 - t0), h, j0, nc);
    cp_async_commit();
    // element i of this thread's column: st[i * st_ld]
    const bool unit = j == dv && dvs > dv;
    float* st = state_pool + (size_t)slot * A.slot_floats + (unit ? A.unit_off + (size_t)h * d : A.state_off + (size_t)h * d * dv + j);
    const int st_ld = unit ? 1 : dv;
    float S[RV][4];
    const bool fresh = A.seq_pos0[seq] == 0;
#pragma unroll
    for (int e = 0; e < RV; ++e)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = 4 * (e * L + q) + x;
            S[e][x] = (!fresh && i < d && j < dvs) ? st[(size_t)i * st_ld] : 0.0f;
        }
    if (A.conv.taps > 1)
        for (int c = part * blockDim.x + threadIdx.x; c < A.conv.ch; c += A.H * NS * blockDim.x) conv_state_update(A.conv, state_pool, seq, c);
    // this lane's output: token q of a group (q < GS)
    float* out = unit ? A.unit_out + h : o_raw + (size_t)h * dv + j;
    const size_t out_ld = unit ? A.H : (size_t)A.H * dv;
    int cur = 0;
    for (int c0 = t0; c0 < t1; c0 += CH, cur ^= 1) {
        const int n = min(CH, t1 - c0);
        cp_async_wait<0>();
        __syncthreads();                          // this chunk has landed; every thread is done with the other buffer
        if (c0 + CH < t1) {
            const int nn = min(CH, t1 - c0 - CH);
            if (vec) group_scan_stage<DK, 4>(A, sh + (cur ^ 1) * kBuf, c0 + CH, nn, h, j0, nc);
            else group_scan_stage<DK, 1>(A, sh + (cur ^ 1) * kBuf, c0 + CH, nn, h, j0, nc);
            cp_async_commit();
        }
        const float* b = sh + cur * kBuf;
        const float4* s4 = reinterpret_cast<const float4*>(b) + q;      // piece e of q of token tt: s4[(tt*DK)/4 + e*L]; k: PL / 4 further on
        const float* s_v = b + 2 * PL + col;
        const float4* s_p = reinterpret_cast<const float4*>(b + 2 * PL + CH * CB);
        const float2* s_h = reinterpret_cast<const float2*>(b + 2 * PL + CH * CB + CH * kPairFloats);
        auto group = [&](const int tt, auto full) {
            constexpr bool FULL = decltype(full)::value;
            float4 k[GS][RV];
            float seen[GS], read[GS];
#pragma unroll
            for (int u = 0; u < GS; ++u) {
                float ka = 0.0f, kb = 0.0f, qa = 0.0f, qb = 0.0f;
#pragma unroll
                for (int e = 0; e < RV; ++e) {
                    const float4 qv = s4[(tt + u) * (DK / 4) + e * L];
                    k[u][e] = s4[PL / 4 + (tt + u) * (DK / 4) + e * L];
                    if (DELTA) {
                        ka = fmaf(k[u][e].x, S[e][0], ka); kb = fmaf(k[u][e].y, S[e][1], kb);
                        ka = fmaf(k[u][e].z, S[e][2], ka); kb = fmaf(k[u][e].w, S[e][3], kb);
                    }
                    qa = fmaf(qv.x, S[e][0], qa); qb = fmaf(qv.y, S[e][1], qb);
                    qa = fmaf(qv.z, S[e][2], qa); qb = fmaf(qv.w, S[e][3], qb);
                }
                seen[u] = ka + kb;
                read[u] = qa + qb;
            }
#pragma unroll
            for (int x = 1; x < L; x <<= 1)
#pragma unroll
                for (int u = 0; u < GS; ++u) {
                    if (DELTA) seen[u] += __shfl_xor_sync(0xffffffffu, seen[u], x);
                    read[u] += __shfl_xor_sync(0xffffffffu, read[u], x);
                }
            float e[GS], P = 1.0f, mine = 0.0f;
#pragma unroll
            for (int i = 0; i < GS; ++i) {
                const bool on = FULL || tt + i < n;
                const float2 wb = s_h[tt + i];
                const float w = on ? wb.x : 1.0f, step = on ? wb.y : 0.0f;
                float kk[4], qk[4];
                *reinterpret_cast<float4*>(qk) = s_p[(tt + i) * 2 + 1];
                P *= w;
#pragma unroll
                for (int m = 0; m < i; ++m) e[m] *= w;
                float u = s_v[(tt + i) * CB];
                if (DELTA) {
                    *reinterpret_cast<float4*>(kk) = s_p[(tt + i) * 2];
                    float sn = P * seen[i];
#pragma unroll
                    for (int m = 0; m < i; ++m) sn = fmaf(kk[m], e[m], sn);
                    u -= sn;
                }
                e[i] = step * u;
                float o = P * read[i];
#pragma unroll
                for (int m = 0; m <= i; ++m) o = fmaf(qk[m], e[m], o);
                if (q == i) mine = o;
            }
            if (q < GS && j < dvs && (FULL || tt + q < n)) out[(size_t)(c0 + tt + q) * out_ld] = mine * A.q_scale;
#pragma unroll
            for (int r = 0; r < RV; ++r) {
                float a0 = P * S[r][0], a1 = P * S[r][1], a2 = P * S[r][2], a3 = P * S[r][3];
#pragma unroll
                for (int u = 0; u < GS; ++u) {
                    a0 = fmaf(k[u][r].x, e[u], a0); a1 = fmaf(k[u][r].y, e[u], a1);
                    a2 = fmaf(k[u][r].z, e[u], a2); a3 = fmaf(k[u][r].w, e[u], a3);
                }
                S[r][0] = a0; S[r][1] = a1; S[r][2] = a2; S[r][3] = a3;
            }
        };
        if (n == CH) {
#pragma unroll 4
            for (int tt = 0; tt < CH; tt += GS) group(tt, TrueType{});
        } else {
            for (int tt = 0; tt < n; tt += GS) group(tt, FalseType{});
        }
    }
#pragma unroll
    for (int e = 0; e < RV; ++e)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = 4 * (e * L + q) + x;
            if (i < d && j < dvs) st[(size_t)i * st_ld] = S[e][x];
        }
}

// ---------------------------------------------------------------------------------------------------------------------
// Gated delta rule.  proj row layout: q | k [G*d each] | v | gate [H*dv each] | step [H] | decay [H]; G key heads serve H / G heads each.
//   q, k, v: short convolution and silu;  q <- q / sqrt(sum q^2 + unit_eps) * q_scale,  k <- k / sqrt(sum k^2 + unit_eps)
//   b = sigmoid(step),  w = exp(-exp(a_log) * softplus(decay + dt_bias))
//   S <- w S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q
struct GatedDeltaArgs {
    const float* proj;
    int n_in, H, G, d, dv;
    float q_scale, unit_eps;
    const float *a_log, *dt_bias;
    const int32_t* tok_seq;
    ConvIo conv;                       // channels q | k | v; its sequences and slots are the recurrence's
    int32_t* err;
};

// Blocks (token, group of 4 warps).  The first G warps of a token take a key head each: convolved q and k, their lengths and
// their product; the others take 64 value channels each.  qkv [T][2 G d + H dv]: unit q (scaled) | unit k | v;
// head: (decay, step) [T][H]; pairs: the token's own k.q where group_scan_kernel expects it.
constexpr int kGatedDeltaCols = 64;
__global__ void __launch_bounds__(128) gated_delta_prep_kernel(const GatedDeltaArgs A, const float* __restrict__ slots, float* __restrict__ qkv,
                                                               float* __restrict__ head, float* __restrict__ pairs) {
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
        head[((size_t)t * A.H + h) * 2] = expf(-expf(A.a_log[h]) * softplus_(p[A.H] + A.dt_bias[h]));
        head[((size_t)t * A.H + h) * 2 + 1] = sigmoidf_(p[0]);
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
        if (lane == 0) pairs[((size_t)t * A.G + warp) * kPairFloats + kScanGroup + r % kScanGroup] = qk * rq * rk;
        return;
    }
    const int c0 = (warp - A.G) * kGatedDeltaCols;
#pragma unroll
    for (int e = 0; e < kGatedDeltaCols / 32; ++e) {
        const int c = c0 + lane + 32 * e;
        if (c < A.H * A.dv) row[2 * gd + c] = conv_channel(C, before, t, r, pos0, 2 * gd + c);
    }
}

// ---------------------------------------------------------------------------------------------------------------------
// mLSTM gates.  Per head, with i = cap tanh((input row + bias) / cap) and f = ln sigmoid(cap tanh((forget row + bias) / cap)):
//   m_t = max(f_t + m_(t-1), i_t),  the memory's decay exp(f_t + m_(t-1) - m_t) and write weight exp(i_t - m_t), and the
//   denominator's floor exp(-m_t).  m starts at 0 and lives in the slot ([H] at m_off).
// A token acts on m as m -> max(F + m, I) with (F, I) = (f, i); two tokens one after the other as (F1 + F2, max(I1 + F2, I2)),
// so the maxima of a whole tile of tokens come from a parallel scan.  One block per (sequence, head).  Rounding in m is harmless:
// decay, weight and floor are all formed from the same m, which only scales numerator and denominator.  A sequence of one token
// also gets its k.q here (pairs, see group_scan_kernel).
struct MlstmArgs {
    const float* proj;
    int n_in, H;
    size_t gate_off;                   // column of the input rows; the forget rows follow
    int d;                             // q rows [H*d] first, k rows behind them
    float cap;
    const float *i_bias, *f_bias;      // [H]
    const int32_t *seq_start, *seq_pos0, *seq_slot;
    size_t slot_floats, m_off;
    int n_slots;
    int32_t* err;
};
constexpr int kMlstmTile = 1024;

// head: (decay, write weight) [T][H]; floor [T][H]
__global__ void __launch_bounds__(kMlstmTile) mlstm_gate_kernel(const MlstmArgs A, float* __restrict__ slots, float* __restrict__ head, float* __restrict__ floor_,
                                                              float* __restrict__ pairs) {
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
    if (t1 - t0 == 1 && warp == 0) {
        const float *q = A.proj + (size_t)t0 * A.n_in + h * A.d, *k = q + A.H * A.d;
        float qk = 0.0f;
        for (int c = lane; c < A.d; c += 32) qk = fmaf(q[c], k[c], qk);
        qk = warp_sum(qk);
        if (lane == 0) pairs[((size_t)t0 * A.H + h) * kPairFloats + kScanGroup] = qk;
    }
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
            head[((size_t)t * A.H + h) * 2] = expf(f + before - mt);
            head[((size_t)t * A.H + h) * 2 + 1] = expf(i - mt);
            floor_[(size_t)t * A.H + h] = expf(-mt);
        }
        m = ms[min((int)blockDim.x, t1 - base)];
    }
    if (threadIdx.x == 0 && t1 > t0) *m_at = m;
}

}  // namespace lm
}  // namespace smol
