// Two more recurrences over a state of fixed size per request, and the small kernels around them.  Conventions as in
// recurrence.cu: one flat batch of tokens, request s owns rows q_start[s] .. q_start[s+1]-1, its state lives in row
// slots[s] of a float32 table [slots, state_stride], rows whose tok_seq is negative are padding of a fixed-shape step.
//
//   cw_unit_heads          every head of a row divided by sqrt(sum of squares + eps), times a scale (one scale for the
//                          leading heads, another for the rest), in place
//   cw_delta_coefficients  a[t, h, i] = exp(-exp(A[h]) softplus(pre[t, h, i] + dt[h, i])) and beta[t, h] = sigmoid(.), in place
//   cw_delta_prepare       everything between a delta layer's joint product and its scan in one kernel: short convolutions and
//                          SiLU on q, k, v, unit vectors per q and k head, one decay and one write strength per head
//   cw_delta_scan          the gated delta rule with a decay per key channel, or one per head:
//                              S <- diag(a_t) S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  y_t = S^T q_t
//                          and, if asked, the convolutions' last inputs kept for the next step
//   cw_gate_scan           the scalar part of a matrix memory with exponential gates, per request and head in token order:
//                              li = cap tanh((zi + bi)/cap), lf = log sigmoid(cap tanh((zf + bf)/cap)),
//                              m_t = max(lf + m_(t-1), li);  keep = exp(lf + m_(t-1) - m_t), take = exp(li - m_t), floor = exp(-m_t)
//                          written as [keep | take | floor] per token: the coefficients of cw_recurrence_scan's form 4
//   cw_memory_norm         what form 4 leaves per head, [S^T q (dv) | n . q], divided by max(|n . q|, floor) + 1e-6, each
//                          head divided by its root mean square, times a weight, times sigmoid(gate)
//
// Everything here is float32 in both run precisions.
#include "common.cuh"

// ---- unit vectors per head ------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
unit_heads_kernel(float* __restrict__ x, int ld, int N, int heads, int dim, float eps, int heads_a, float scale_a, float scale_b) {
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);  // a warp per (row, head)
    if (item >= (long long)N * heads) return;
    const int row = (int)(item / heads), h = (int)(item - (long long)row * heads);
    float* at = x + (size_t)row * ld + (size_t)h * dim;
    float ss = 0.f;
    for (int i = lane; i < dim; i += 32) ss = fmaf(at[i], at[i], ss);
    ss = warp_sum(ss);
    const float f = (h < heads_a ? scale_a : scale_b) / sqrtf(ss + eps);
    for (int i = lane; i < dim; i += 32) at[i] *= f;
}

extern "C" int cw_unit_heads(float* x, int ld, int N, int heads, int dim, float eps, int heads_a, float scale_a, float scale_b,
                             cudaStream_t stream) {
    if (N == 0) return CW_OK;
    if (N < 0 || heads <= 0 || dim <= 0 || ld < heads * dim) return CW_ERR_BAD_SIZE;
    const long long items = (long long)N * heads;
    return cw_launch_ordered(unit_heads_kernel, dim3((unsigned)((items + 7) / 8)), dim3(256), 0, stream, x, ld, N, heads, dim, eps, heads_a,
                             scale_a, scale_b);
}

// ---- decays and write strengths of the delta rule ----------------------------------------------------------
__global__ void __launch_bounds__(256)
delta_coefficients_kernel(float* __restrict__ pre, int ldp, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                          float* __restrict__ beta, int ldb, int N, int H, int Dk) {
    pdl_wait();
    const int C = H * Dk;
    const long long total = (long long)N * (C + H);
    for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
        const int t = (int)(idx / (C + H)), c = (int)(idx - (long long)t * (C + H));
        if (c < C) {
            float* at = pre + (size_t)t * ldp + c;
            const float x = *at + dt_bias[c];
            const float step = fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
            *at = expf(-expf(a_log[c / Dk]) * step);
        } else {
            float* at = beta + (size_t)t * ldb + (c - C);
            *at = 1.f / (1.f + expf(-*at));
        }
    }
}

extern "C" int cw_delta_coefficients(float* pre, int ldp, const float* dt_bias, const float* a_log, float* beta, int ldb, int N, int H,
                                     int Dk, cudaStream_t stream) {
    if (N == 0) return CW_OK;
    if (N < 0 || H <= 0 || Dk <= 0 || ldp < H * Dk || ldb < H) return CW_ERR_BAD_SIZE;
    const long long total = (long long)N * (H * Dk + H);
    const int blocks = (int)min((long long)148 * 8, (total + 255) / 256);
    return cw_launch_ordered(delta_coefficients_kernel, dim3(blocks), dim3(256), 0, stream, pre, ldp, dt_bias, a_log, beta, ldb, N, H, Dk);
}

// ---- from the joint product to the scan's operands ----------------------------------------------------------
// x [N, ldx] float32: a token's product row [q (groups*dk) | k (groups*dk) | v (H*dv) | ..], C = 2*groups*dk + H*dv columns
// that pass a causal convolution of `taps` taps per channel (weight [C, taps], the current token's last; inputs before a
// portion's first row are the rows kept in the request's state) and SiLU; then every q and k head is divided by
// sqrt(sum of squares + eps), q heads times q_scale.  out [N, C].  beta [N, ldb] and decay [N, lda] hold the pre-activations of a
// number per head: coef [N, 2H] = [exp(-exp(A[h]) softplus(decay + dt[h])) | sigmoid(beta)].  Blocks: (token, share of its heads
// and channels); a warp per q or k head, its channels in registers between the sum and the division.  VEC: four taps, four
// neighbouring channels a lane in 16-byte accesses (heads of a multiple of four channels at 16-byte addresses).
#define DP_CH 8  // channels of a head per lane (heads up to 256 wide)
struct DeltaPrepareArgs {
    const float* x;
    int ldx;
    const float* weight;
    int taps;
    const float* state;
    long long state_stride, conv_off;
    const long long* slots;
    const int* tok_seq;
    const int* q_start;
    int groups, Dk, H, Dv;
    float eps, q_scale;
    const float* beta;
    int ldb;
    const float* decay;
    int lda;
    const float* dt_bias;
    const float* a_log;
    float* out;
    float* coef;
};

template <bool VEC>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const DeltaPrepareArgs a) {
    pdl_wait();
    const int row = blockIdx.x, tid = threadIdx.x, share = blockIdx.y, shares = gridDim.y;
    const int Dk = a.Dk, qk = a.groups * Dk, C = 2 * qk + a.H * a.Dv, R = a.taps - 1;
    const int at = share * blockDim.x + tid, step = shares * blockDim.x;  // this thread's first channel (or four) and the stride
    float* o = a.out + (size_t)row * C;
    float* cf = a.coef + (size_t)row * 2 * a.H;
    const int seq = a.tok_seq[row];
    if (seq < 0) {  // padding of a fixed-shape step
        for (int c = at; c < C; c += step) o[c] = 0.f;
        for (int h = at; h < 2 * a.H; h += step) cf[h] = 0.f;
        return;
    }
    const int start = a.q_start[seq];
    const float* kept = a.state + a.slots[seq] * a.state_stride + a.conv_off;
    auto source = [&](int j) {  // the row that tap j reads
        const int src = row - (R - j);
        return src >= start ? a.x + (size_t)src * a.ldx : kept + (size_t)(R - (start - src)) * C;
    };
    auto silu = [](float z) { return z / (1.f + expf(-z)); };
    auto conv = [&](int c) {
        float acc = 0.f;
        for (int j = 0; j < a.taps; ++j) acc = fmaf(a.weight[(size_t)c * a.taps + j], source(j)[c], acc);
        return silu(acc);
    };
    const float* rows4[4];
    if (VEC) {
#pragma unroll
        for (int j = 0; j < 4; ++j) rows4[j] = source(j);
    }
    auto conv4 = [&](int c) {  // channels c .. c + 3
        float4 x[4], w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] = *(const float4*)(rows4[j] + c);
#pragma unroll
        for (int i = 0; i < 4; ++i) w[i] = *(const float4*)(a.weight + (size_t)(c + i) * 4);
        float4 y;
        y.x = silu(fmaf(w[0].w, x[3].x, fmaf(w[0].z, x[2].x, fmaf(w[0].y, x[1].x, w[0].x * x[0].x))));
        y.y = silu(fmaf(w[1].w, x[3].y, fmaf(w[1].z, x[2].y, fmaf(w[1].y, x[1].y, w[1].x * x[0].y))));
        y.z = silu(fmaf(w[2].w, x[3].z, fmaf(w[2].z, x[2].z, fmaf(w[2].y, x[1].z, w[2].x * x[0].z))));
        y.w = silu(fmaf(w[3].w, x[3].w, fmaf(w[3].z, x[2].w, fmaf(w[3].y, x[1].w, w[3].x * x[0].w))));
        return y;
    };
    const int lane = tid & 31, nwarps = blockDim.x >> 5;
    for (int head = share * nwarps + (tid >> 5); head < 2 * a.groups; head += shares * nwarps) {
        float ss = 0.f;
        const float scale = head < a.groups ? a.q_scale : 1.f;
        if (VEC) {
            float4 u[DP_CH / 4];
#pragma unroll
            for (int r = 0; r < DP_CH / 4; ++r) {
                const int i = (lane + 32 * r) * 4;
                u[r] = i < Dk ? conv4(head * Dk + i) : make_float4(0.f, 0.f, 0.f, 0.f);
                ss = fmaf(u[r].x, u[r].x, fmaf(u[r].y, u[r].y, fmaf(u[r].z, u[r].z, fmaf(u[r].w, u[r].w, ss))));
            }
            const float f = scale / sqrtf(warp_sum(ss) + a.eps);
#pragma unroll
            for (int r = 0; r < DP_CH / 4; ++r) {
                const int i = (lane + 32 * r) * 4;
                if (i < Dk) *(float4*)(o + head * Dk + i) = make_float4(u[r].x * f, u[r].y * f, u[r].z * f, u[r].w * f);
            }
        } else {
            float u[DP_CH];
#pragma unroll
            for (int r = 0; r < DP_CH; ++r) {
                const int i = lane + 32 * r;
                u[r] = i < Dk ? conv(head * Dk + i) : 0.f;
                ss = fmaf(u[r], u[r], ss);
            }
            const float f = scale / sqrtf(warp_sum(ss) + a.eps);
#pragma unroll
            for (int r = 0; r < DP_CH; ++r) {
                const int i = lane + 32 * r;
                if (i < Dk) o[head * Dk + i] = u[r] * f;
            }
        }
    }
    if (VEC) {
        for (int c = 2 * qk + 4 * at; c < C; c += 4 * step) *(float4*)(o + c) = conv4(c);
    } else {
        for (int c = 2 * qk + at; c < C; c += step) o[c] = conv(c);
    }
    for (int h = at; h < a.H; h += step) {
        const float z = a.decay[(size_t)row * a.lda + h] + a.dt_bias[h];
        const float softplus = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
        cf[h] = expf(-expf(a.a_log[h]) * softplus);
        cf[a.H + h] = 1.f / (1.f + expf(-a.beta[(size_t)row * a.ldb + h]));
    }
}

extern "C" int cw_delta_prepare(const float* x, int ldx, const float* weight, int taps, const float* state, long long state_stride,
                                long long conv_off, const long long* slots, const int* tok_seq, const int* q_start, int groups, int Dk,
                                int H, int Dv, float eps, float q_scale, const float* beta, int ldb, const float* decay, int lda,
                                const float* dt_bias, const float* a_log, int N, float* out, float* coef, cudaStream_t stream) {
    if (N == 0) return CW_OK;
    if (N < 0 || groups <= 0 || Dk <= 0 || H <= 0 || Dv <= 0 || taps <= 0 || ldx < 2 * groups * Dk + H * Dv || ldb < H || lda < H)
        return CW_ERR_BAD_SIZE;
    if (Dk > 32 * DP_CH) return CW_ERR_UNSUPPORTED;
    const int C = 2 * groups * Dk + H * Dv;
    auto whole = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = taps == 4 && Dk % 4 == 0 && C % 4 == 0 && ldx % 4 == 0 && state_stride % 4 == 0 && conv_off % 4 == 0 && whole(x) &&
                     whole(weight) && whole(state) && whole(out);
    int threads = 64;
    while (threads < 256 && threads * 4 < C) threads *= 2;
    // few tokens: a token's channels over several blocks, as many as have work and fill the GPU once
    int shares = 1;
    while (shares < 32 && (long long)N * shares < 148 && shares * threads * 4 < C) shares *= 2;
    const DeltaPrepareArgs args = {x, ldx, weight, taps, state, state_stride, conv_off, slots, tok_seq, q_start, groups, Dk, H, Dv, eps,
                                   q_scale, beta, ldb, decay, lda, dt_bias, a_log, out, coef};
    return cw_launch_ordered(vec ? delta_prepare_kernel<true> : delta_prepare_kernel<false>, dim3(N, shares), dim3(threads), 0, stream, args);
}

// ---- the delta rule ---------------------------------------------------------------------------------------
// State per request and head: S [Dk, Dv] stored value-column-major (element (i, j) of head h at (h*Dv + j)*Dk + i).
// Blocks: (request, head, slice of JB value columns); IP threads share a value column.  The operands of DC tokens at a time
// are staged in shared memory by cp.async (the next chunk while the current one runs).  Per token the column's S^T k is
// summed over the IP lanes by shuffles (the update needs it); the read-out sums wait until the chunk is through.  Every sum
// has a fixed order, so a row's result does not depend on how the request's tokens were cut into steps or on what else the
// step holds.
// IPT > 0: IP known at compile time and heads of whole groups of eight channels at 16-byte addresses: a thread owns channels
// 4 ipart .. 4 ipart + 3 and the same four in the upper half of the head (two 16-byte words per operand and token), and the
// read-out sums of the chunk's tokens are added up over the lanes with the tokens spread over them.  IPT = 0: any head size,
// channels ipart, ipart + IP, .. one word at a time.
// HEAD: one decay per head and token (a [N, H]) instead of one per key channel (a [N, H*Dk]); S^T k of the decayed state is then
// the decay times S^T k of the state before.
#define DS 8    // key channels per thread
#define DC 16   // tokens per staged chunk

__device__ __forceinline__ void dcp4(float* smem, const float* gmem) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(gmem) : "memory");
}
__device__ __forceinline__ void dcp16(float* smem, const float* gmem) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(gmem) : "memory");
}

struct DeltaScanArgs {
    const float* q;  // [N, ldq]: head h reads columns (h / heads_per_group) * Dk ..
    int ldq;
    const float* k;
    int ldk;
    const float* v;  // [N, ldv]: head h's columns h*Dv ..
    int ldv;
    const float* a;  // decays
    int lda;
    const float* beta;  // [N, ldb]
    int ldb;
    float* state;
    long long state_stride, state_off;
    const long long* slots;
    const int* tok_seq;
    const int* q_start;
    int Dk, Dv, heads_per_group, IP, wide;
    float* out;  // [N, ldo]
    int ldo;
    // the rows of `carry` [N, ldc] (C columns) that the next step's convolutions read again: the last R of each portion go to
    // the request's state at carry_off (null: none; the convolutions of this step have run)
    const float* carry;
    int ldc, C, R;
    long long carry_off;
};

template <int IPT, bool HEAD>
__global__ void __launch_bounds__(256)
delta_scan_kernel(const DeltaScanArgs g) {
    extern __shared__ __align__(16) float ds_smem[];
    __shared__ __align__(16) float nothing[4];  // zeros: what lanes without channels read
    if (threadIdx.x < 4) nothing[threadIdx.x] = 0.f;
    pdl_wait();
    // (the request is the slowest index: the blocks of a request that brings tokens then start side by side on as many SMs,
    // however many requests of a fixed-shape step bring none)
    const int seq = blockIdx.z, h = blockIdx.y, tid = threadIdx.x;
    const int start = g.q_start[seq], end = g.q_start[seq + 1];
    if (end <= start) return;
    constexpr bool VEC = IPT > 0;
    const int IP = VEC ? IPT : g.IP, Dk = g.Dk, Dv = g.Dv;
    const int ipart = tid % IP, jl = tid / IP, JB = blockDim.x / IP;
    const int j0 = blockIdx.x * JB, j = j0 + jl;
    const bool live = j < Dv;
    if (g.tok_seq[start] < 0) {  // padding rows of a fixed-shape step: no request, no state
        if (live && ipart == 0)
            for (int t = start; t < end; ++t) g.out[(size_t)t * g.ldo + (size_t)h * Dv + j] = 0.f;
        return;
    }
    // one buffer: q [DC][Dk], k [DC][Dk], a [DC][Dk] or [DC], v [DC][JB], beta [DC]
    const int a_words = HEAD ? DC : DC * Dk;
    const int buf_words = 2 * DC * Dk + a_words + DC * JB + DC;
    const int group = h / g.heads_per_group;
    float* row_state = g.state + g.slots[seq] * g.state_stride;
    float* S_mem = row_state + g.state_off + ((size_t)h * Dv + (live ? j : 0)) * Dk;
    const int half = Dk >> 1;
    const bool mine = ipart * DS < Dk;  // (VEC: the thread owns channels at all)
    const int token_step = mine ? Dk : 0, upper = mine ? half : 0;
    auto channel = [&](int r) { return VEC ? (r < 4 ? 0 : half) + ipart * 4 + (r & 3) : ipart + r * IP; };
    auto owns = [&](int r) { return VEC ? mine : ipart + r * IP < Dk; };
    float S[DS];
#pragma unroll
    for (int r = 0; r < DS; ++r) S[r] = (owns(r) && live) ? S_mem[channel(r)] : 0.f;
    const float* qp = g.q + (size_t)group * Dk;
    const float* kp = g.k + (size_t)group * Dk;
    const float* ap = g.a + (HEAD ? (size_t)h : (size_t)h * Dk);
    const float* vp = g.v + (size_t)h * Dv + j0;
    const float* bp = g.beta + h;
    const int nv = min(JB, Dv - j0);
    auto fetch = [&](int t0, float* buf) {
        const int n = min(DC, end - t0);
        float* qs = buf;
        float* ks = buf + DC * Dk;
        float* as = buf + 2 * DC * Dk;
        float* vs = as + a_words;
        float* bs = vs + DC * JB;
        if (VEC || g.wide) {  // rows of whole 16-byte pieces at 16-byte addresses
            const int pieces = Dk >> 2;
            for (int idx = tid; idx < n * pieces; idx += blockDim.x) {
                const int t = idx / pieces, i = (idx - t * pieces) << 2;
                dcp16(qs + t * Dk + i, qp + (size_t)(t0 + t) * g.ldq + i);
                dcp16(ks + t * Dk + i, kp + (size_t)(t0 + t) * g.ldk + i);
                if (!HEAD) dcp16(as + t * Dk + i, ap + (size_t)(t0 + t) * g.lda + i);
            }
        } else {
            for (int idx = tid; idx < n * Dk; idx += blockDim.x) {
                const int t = idx / Dk, i = idx - t * Dk;
                dcp4(qs + idx, qp + (size_t)(t0 + t) * g.ldq + i);
                dcp4(ks + idx, kp + (size_t)(t0 + t) * g.ldk + i);
                if (!HEAD) dcp4(as + idx, ap + (size_t)(t0 + t) * g.lda + i);
            }
        }
        for (int idx = tid; idx < n * nv; idx += blockDim.x) {
            const int t = idx / nv, c = idx - t * nv;
            dcp4(vs + t * JB + c, vp + (size_t)(t0 + t) * g.ldv + c);
        }
        for (int t = tid; t < n; t += blockDim.x) {
            dcp4(bs + t, bp + (size_t)(t0 + t) * g.ldb);
            if (HEAD) dcp4(as + t, ap + (size_t)(t0 + t) * g.lda);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(start, ds_smem);
    if (g.carry != nullptr) {  // the blocks of the request share its channels out
        const int n = end - start, block = blockIdx.y * gridDim.x + blockIdx.x, blocks = gridDim.y * gridDim.x;
        float* kept = row_state + g.carry_off;
        for (int c = block * blockDim.x + tid; c < g.C; c += blocks * blockDim.x)
            for (int d = g.R; d >= 1; --d)  // ascending writes; what is read lies ahead of what was written
                kept[(size_t)(g.R - d) * g.C + c] =
                    d <= n ? g.carry[(size_t)(end - d) * g.ldc + c] : kept[(size_t)(g.R - (d - n)) * g.C + c];
    }
    int which = 0;
    for (int t0 = start; t0 < end; t0 += DC, which ^= 1) {
        const int n = min(DC, end - t0);
        float* buf = ds_smem + which * buf_words;
        const float* qs = buf;
        const float* ks = buf + DC * Dk;
        const float* as = buf + 2 * DC * Dk;
        const float* vs = as + a_words;
        const float* bs = vs + DC * JB;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // this chunk has landed; everyone has left the other buffer
        if (t0 + DC < end) fetch(t0 + DC, ds_smem + (which ^ 1) * buf_words);
        float part[DC];
        const float* q0 = mine ? qs + ipart * 4 : nothing;
        const float* k0 = mine ? ks + ipart * 4 : nothing;
        const float* a0 = mine ? as + ipart * 4 : nothing;
        auto token = [&](int t) {  // the thread's share of token t's output; its column of the state moves on by the token
            float kc[DS], qc[DS], ac[DS];
            if (VEC) {
                const int at = t * token_step;
                *(float4*)&kc[0] = *(const float4*)(k0 + at);
                *(float4*)&kc[4] = *(const float4*)(k0 + at + upper);
                *(float4*)&qc[0] = *(const float4*)(q0 + at);
                *(float4*)&qc[4] = *(const float4*)(q0 + at + upper);
                if (!HEAD) {
                    *(float4*)&ac[0] = *(const float4*)(a0 + at);
                    *(float4*)&ac[4] = *(const float4*)(a0 + at + upper);
                }
            } else {
#pragma unroll
                for (int r = 0; r < DS; ++r) {
                    const int i = ipart + r * IP;
                    const bool on = i < Dk;
                    kc[r] = on ? ks[t * Dk + i] : 0.f;
                    qc[r] = on ? qs[t * Dk + i] : 0.f;
                    if (!HEAD) ac[r] = on ? as[t * Dk + i] : 0.f;
                }
            }
            const float decay = HEAD ? as[t] : 0.f;
            float aS[DS];
            float dot0 = 0.f, dot1 = 0.f;  // two chains, added at the end: the same order for every token and batch
#pragma unroll
            for (int r = 0; r < DS; ++r) {
                aS[r] = (HEAD ? decay : ac[r]) * S[r];
                if (r & 1) dot1 = fmaf(HEAD ? S[r] : aS[r], kc[r], dot1);
                else dot0 = fmaf(HEAD ? S[r] : aS[r], kc[r], dot0);
            }
            float dot = dot0 + dot1;
            if (VEC) {
#pragma unroll
                for (int o = 1; o < (VEC ? IPT : 1); o <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
            } else {
                for (int o = 1; o < IP; o <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
            }
            if (HEAD) dot *= decay;
            const float u = live ? bs[t] * (vs[t * JB + jl] - dot) : 0.f;
            float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
            for (int r = 0; r < DS; ++r) {
                S[r] = fmaf(kc[r], u, aS[r]);
                if (r & 1) sum1 = fmaf(qc[r], S[r], sum1);
                else sum0 = fmaf(qc[r], S[r], sum0);
            }
            return sum0 + sum1;
        };
        if (n == DC) {
#pragma unroll
            for (int t = 0; t < DC; ++t) part[t] = token(t);
        } else {
#pragma unroll
            for (int t = 0; t < DC; ++t) part[t] = t < n ? token(t) : 0.f;
        }
        if (VEC) {
            const int first = sum_tokens_over_lanes<VEC ? IPT : 1, DC>(part, ipart);
            if (live && first >= 0) {
#pragma unroll
                for (int i = 0; i < (IPT > DC ? 1 : DC / (VEC ? IPT : 1)); ++i)
                    if (first + i < n) g.out[(size_t)(t0 + first + i) * g.ldo + (size_t)h * Dv + j] = part[i];
            }
        } else {
#pragma unroll
            for (int t = 0; t < DC; ++t)
                for (int o = 1; o < IP; o <<= 1) part[t] += __shfl_xor_sync(0xffffffffu, part[t], o);
            if (live && ipart == 0) {
#pragma unroll
                for (int t = 0; t < DC; ++t)
                    if (t < n) g.out[(size_t)(t0 + t) * g.ldo + (size_t)h * Dv + j] = part[t];
            }
        }
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < DS; ++r)
            if (owns(r)) S_mem[channel(r)] = S[r];
    }
}

// q, k [N, groups*Dk] (head h reads group h / heads_per_group), v [N, H*Dv], beta [N, H], decays a [N, H*Dk] or, with
// head_decay, [N, H]: float32, unit column stride, any row stride.  out [N, H*Dv].  rows: N, which only sizes the blocks.
extern "C" int cw_delta_scan(const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, const float* a, int lda,
                             int head_decay, const float* beta, int ldb, float* state, long long state_stride, long long state_off,
                             const long long* slots, const int* tok_seq, const int* q_start, int S, int H, int Dk, int Dv,
                             int heads_per_group, float* out, int ldo, const float* carry, int ldc, int C, int R, long long carry_off,
                             int rows, cudaStream_t stream) {
    if (S == 0) return CW_OK;
    if (S < 0 || H <= 0 || Dk <= 0 || Dv <= 0 || heads_per_group <= 0 || H % heads_per_group) return CW_ERR_BAD_SIZE;
    if (carry != nullptr && (C <= 0 || R < 0 || ldc < C)) return CW_ERR_BAD_SIZE;
    if (Dk > 32 * DS || H > 65535 || S > 65535) return CW_ERR_UNSUPPORTED;
    int IP = 1, log_ip = 0;
    while (IP * DS < Dk) {
        IP *= 2;
        ++log_ip;
    }
    int threads = 256;  // more value columns per block share the staged q, k and decays; fewer when a head has few columns
    while (threads > 32 && threads / IP >= 2 * Dv) threads /= 2;
    const int JB = threads / IP;
    dim3 grid((Dv + JB - 1) / JB, H, S);
    const int wide = Dk % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && ((uintptr_t)q & 15) == 0 && ((uintptr_t)k & 15) == 0 &&
                     (head_decay || (lda % 4 == 0 && ((uintptr_t)a & 15) == 0));
    const bool vec = wide && Dk % DS == 0;
    const size_t smem = cw_scan_smem(2 * sizeof(float) * (size_t)((head_decay ? 2 : 3) * DC * Dk + DC * JB + (head_decay ? 2 : 1) * DC), rows);
    using Kernel = void (*)(const DeltaScanArgs);
    static const Kernel kernels[2][7] = {
        {delta_scan_kernel<1, false>, delta_scan_kernel<2, false>, delta_scan_kernel<4, false>, delta_scan_kernel<8, false>,
         delta_scan_kernel<16, false>, delta_scan_kernel<32, false>, delta_scan_kernel<0, false>},
        {delta_scan_kernel<1, true>, delta_scan_kernel<2, true>, delta_scan_kernel<4, true>, delta_scan_kernel<8, true>,
         delta_scan_kernel<16, true>, delta_scan_kernel<32, true>, delta_scan_kernel<0, true>}};
    static size_t allowed[2][7] = {};
    const int by_head = head_decay ? 1 : 0, which = vec ? log_ip : 6;
    if (smem > (48u << 10) && smem > allowed[by_head][which]) {
        const cudaError_t e = cudaFuncSetAttribute(kernels[by_head][which], cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        allowed[by_head][which] = smem;
    }
    const DeltaScanArgs args = {q, ldq, k, ldk, v, ldv, a, lda, beta, ldb, state, state_stride, state_off, slots, tok_seq, q_start, Dk, Dv,
                                heads_per_group, IP, wide, out, ldo, R > 0 ? carry : nullptr, ldc, C, R, carry_off};
    return cw_launch_ordered(kernels[by_head][which], grid, dim3(threads), smem, stream, args);
}

// ---- the gates of a matrix memory -----------------------------------------------------------------------
// zi, zf [N, ld*] float32 pre-activations of the input and forget gates (a column per head); the running maximum m of
// every head is one float of the request's state (at state_off + h; 0 when a request starts).  coef [N, 3H].
// A block per request, GS_WORDS / H tokens at a time through shared memory, in three passes: every (token, head) pair's
// two logarithms side by side; a thread per head walks the tokens in order (a chain of one addition and one maximum
// per token, its operands already on chip, so a token costs a few cycles); every pair's three exponentials side by
// side.  The chain's order is the tokens' order whatever the cut, so a request's coefficients do not depend on how
// its tokens came in steps.
#define GS_WORDS 2048
__global__ void __launch_bounds__(1024)
gate_scan_kernel(const float* __restrict__ zi, int ldi, const float* __restrict__ zf, int ldf, const float* __restrict__ bias_i,
                 const float* __restrict__ bias_f, float cap, float* __restrict__ state, long long state_stride, long long state_off,
                 const long long* __restrict__ slots, const int* __restrict__ tok_seq, const int* __restrict__ q_start, int H,
                 float* __restrict__ coef) {
    __shared__ float s_li[GS_WORDS], s_lf[GS_WORDS], s_m[2 * GS_WORDS];  // s_m: the maximum before token t at [t][h], after it at [t+1][h]
    pdl_wait();
    const int seq = blockIdx.x;
    const int start = q_start[seq], end = q_start[seq + 1];
    if (end <= start) return;
    const size_t ldc = 3 * (size_t)H;
    if (tok_seq[start] < 0) {  // padding rows: coefficients that leave a zero state at zero
        const int n = end - start;
        for (int idx = threadIdx.x; idx < n * 3 * H; idx += blockDim.x) coef[(size_t)start * ldc + idx] = idx % (3 * H) < 2 * H ? 0.f : 1.f;
        return;
    }
    float* m_mem = state + slots[seq] * state_stride + state_off;
    const int TC = GS_WORDS / H;  // (the launcher refuses more heads than GS_WORDS)
    for (int c0 = start; c0 < end; c0 += TC) {
        const int n = min(TC, end - c0);
        for (int idx = threadIdx.x; idx < n * H; idx += blockDim.x) {
            const int t = c0 + idx / H, h = idx % H;
            const float li = cap * tanhf((zi[(size_t)t * ldi + h] + (bias_i != nullptr ? bias_i[h] : 0.f)) / cap);
            const float c = cap * tanhf((zf[(size_t)t * ldf + h] + (bias_f != nullptr ? bias_f[h] : 0.f)) / cap);
            s_li[idx] = li;
            s_lf[idx] = fminf(c, 0.f) - log1pf(expf(-fabsf(c)));
        }
        __syncthreads();
        for (int h = threadIdx.x; h < H; h += blockDim.x) {
            float m = m_mem[h];
            s_m[h] = m;
            for (int t0 = 0; t0 < n; t0 += 8) {  // eight tokens' operands fetched side by side, then the chain through them
                float li[8], lf[8];
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const int at = min(t0 + j, n - 1) * H + h;
                    li[j] = s_li[at];
                    lf[j] = s_lf[at];
                }
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    if (t0 + j < n) {
                        m = fmaxf(lf[j] + m, li[j]);
                        s_m[(t0 + j + 1) * H + h] = m;
                    }
                }
            }
            m_mem[h] = m;
        }
        __syncthreads();
        for (int idx = threadIdx.x; idx < n * H; idx += blockDim.x) {
            const int t = idx / H, h = idx - t * H;
            const float before = s_m[idx], after = s_m[idx + H];
            float* c = coef + (size_t)(c0 + t) * ldc;
            c[h] = expf(s_lf[idx] + before - after);
            c[H + h] = expf(s_li[idx] - after);
            c[2 * H + h] = expf(-after);
        }
        __syncthreads();  // the next chunk writes the same shared memory
    }
}

// N: the rows of the step (all requests'), which only sizes the blocks.
extern "C" int cw_gate_scan(const float* zi, int ldi, const float* zf, int ldf, const float* bias_i, const float* bias_f, float cap,
                            float* state, long long state_stride, long long state_off, const long long* slots, const int* tok_seq,
                            const int* q_start, int S, int H, int N, float* coef, cudaStream_t stream) {
    if (S == 0) return CW_OK;
    if (S < 0 || H <= 0 || ldi < H || ldf < H || !(cap > 0.f)) return CW_ERR_BAD_SIZE;
    if (H > GS_WORDS) return CW_ERR_UNSUPPORTED;
    const long long per_request = (long long)(N > 0 ? N : S) * H / S;  // pairs of a request, if the rows were spread evenly
    const int threads = per_request >= 8192 ? 1024 : per_request >= 1024 ? 256 : 128;
    return cw_launch_ordered(gate_scan_kernel, dim3(S), dim3(threads), 0, stream, zi, ldi, zf, ldf, bias_i, bias_f, cap, state, state_stride,
                             state_off, slots, tok_seq, q_start, H, coef);
}

// ---- read-out of the matrix memory ------------------------------------------------------------------------
// y [N, H*(dv+1)] float32: per head [S^T q (dv) | n . q];  floor_ [N, ldfl] (a column per head);  gate z [N, ldz];
// weight [H*dv].  out[row, h*dv + c] = rmsnorm_head(y_c / (max(|n . q|, floor) + 1e-6)) * weight * sigmoid(z).
// A warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256)
memory_norm_kernel(const float* __restrict__ y, const float* __restrict__ floor_, int ldfl, const float* __restrict__ z, int ldz,
                   const float* __restrict__ weight, T* __restrict__ out, int N, int H, int dv, float eps) {
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= (long long)N * H) return;
    const int row = (int)(item / H), h = (int)(item - (long long)row * H);
    const float* yr = y + ((size_t)row * H + h) * (dv + 1);
    const float inv_d = 1.f / (fmaxf(fabsf(yr[dv]), floor_[(size_t)row * ldfl + h]) + 1e-6f);
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) {
        const float u = yr[c] * inv_d;
        ss = fmaf(u, u, ss);
    }
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
    const float* zr = z + (size_t)row * ldz + (size_t)h * dv;
    const float* wr = weight + (size_t)h * dv;
    T* o = out + ((size_t)row * H + h) * dv;
    for (int c = lane; c < dv; c += 32) o[c] = from_f<T>(yr[c] * inv_d * inv * wr[c] / (1.f + expf(-zr[c])));
}

extern "C" int cw_memory_norm(const float* y, const float* floor_, int ldfl, const float* z, int ldz, const float* weight, void* out,
                              int N, int H, int dv, float eps, int dtype, cudaStream_t stream) {
    if (N == 0) return CW_OK;
    if (N < 0 || H <= 0 || dv <= 0 || ldfl < H || ldz < H * dv) return CW_ERR_BAD_SIZE;
    const long long items = (long long)N * H;
    const dim3 grid((unsigned)((items + 7) / 8));
    if (dtype == 0)
        return cw_launch_ordered(memory_norm_kernel<float>, grid, dim3(256), 0, stream, y, floor_, ldfl, z, ldz, weight, (float*)out, N, H,
                                 dv, eps);
    if (dtype == 1)
        return cw_launch_ordered(memory_norm_kernel<bf16>, grid, dim3(256), 0, stream, y, floor_, ldfl, z, ldz, weight, (bf16*)out, N, H, dv,
                                 eps);
    return CW_ERR_BAD_DTYPE;
}

CW_TRACE_TU(recurrence_gated)
