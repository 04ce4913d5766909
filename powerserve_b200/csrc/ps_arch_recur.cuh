// ps_arch_recur.cuh - device code of the layer-list executor's recurrent token mixers and short convolutions (ps_arch.cu).
//
// Everything here works on a batch of consecutive tokens of ONE sequence and reads the first token's position from device memory,
// so the same launches serve prompt portions and the replayed single-token step.  A sequence at position 0 starts from zero state
// whatever the state buffers hold (a cache set that is used again needs no clearing).
//
//   pa_k_short_conv      causal convolution over time on every channel, taps newest last, inputs before the batch from the `tail`
//                        (the last taps - 1 inputs of the sequence; as a ring of `taps` rows, position p in row p mod taps, for the rg-lru),
//                        zeros before position 0; optional bias and silu
//   pa_k_conv_tail       the tail after the batch
//   pa_k_conv_step       both for a single token
//   pa_k_qkv_whole_norm  q (all heads) and k RMS-normed as one vector each with weights; K row and V^T column into the cache
//   pa_k_rope_heads      rotate-half rotation of the first dims of every head, in place, with a scale for the heads from `h_scaled` on
//   pa_k_token_shift     h + (h' - h) mu_s for the five inputs of a time mixing (h' the token before)
//   pa_k_decay           low-rank decays per key channel and token; keeps a time mixing's last input
//   pa_k_scan            S_t = a_t S_(t-1) + k_t (c_t v_t)^T, o_t = S_t^T q_t (+ D v_t): retention (a fixed per head, c = 1) and the
//                        state-space recurrence (a_t = exp(-exp(A_log) dt_t), c_t = dt_t, dt = softplus(raw + bias)); fp32 state,
//                        16 entries of a value column per lane in registers, tokens strictly in order (the result does not
//                        depend on how a prompt was cut)
//                        MODE 1: a decay per key channel and token (gated linear attention); MODE 2: the same, and the current token counts
//                        with a bonus u per channel before it joins the state (time mixing)
//   pa_k_dec_recur       one token of the MODE 1 / 2 recurrences with everything around them: the decay's low-rank product, state, output,
//                        the head's RMS norm over a thread-block cluster, weight and silu gate in one launch
//   pa_k_gate_gru        after an attention: the heads' outputs times their sigmoid gate, and the minGRU beside the attention
//                        (S_t = (1 - z) S_(t-1) + z cand per channel, rounds of 32 tokens, gates formed ahead of the dependent steps)
//   pa_k_rglru_scan      real-gated linear recurrence of a batch: S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a_t = -rate r_t
//                        softplus(lam), times gelu(y); rounds of 32 tokens like the minGRU; leaves the convolution's ring for the next batch
//   pa_k_dec_rglru       convolution, both gates' block rows, recurrence and output product of a single token in one launch
//   pa_k_gate_norm_warp  the same for parts of at most 256 entries, a warp per part
//   pa_k_gate_norm       RMS norm in equal parts around a silu gate: (y silu(g)) normed times w, or normed y times silu(g)
//   pa_k_moe_sum         sum of a token's expert slots (fixed order) plus the gated shared expert
#pragma once

__device__ __forceinline__ float pa_silu(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float pa_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// grid (channels / 256, tokens)
__global__ void __launch_bounds__(256) pa_k_short_conv(const float *__restrict__ u, int ldu, const float *__restrict__ w, const float *__restrict__ b, int C, int T,
                                                       const float *__restrict__ tail, int act_silu, float *__restrict__ y, int ldy, const int32_t *__restrict__ pos, int ring) {
    const int t = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    if (c >= C) return;
    const int p0 = pos[0];
    float acc = b ? b[c] : 0.f;
    for (int j = 0; j < T; j++) {
        const int s = t - (T - 1) + j; // token of the batch this tap meets (negative: before the batch)
        float v = 0.f;
        if (s >= 0) v = u[(int64_t)s * ldu + c];
        else if (p0 + s >= 0) v = tail[(int64_t)(ring ? (p0 + s) % T : T - 1 + s) * C + c];
        acc = fmaf(w[(int64_t)c * T + j], v, acc);
    }
    y[(int64_t)t * ldy + c] = act_silu ? pa_silu(acc) : acc;
}

// a thread per channel; the tail is shifted in place oldest first (entry j takes what lay bs entries later)
__global__ void __launch_bounds__(256) pa_k_conv_tail(const float *__restrict__ u, int ldu, int C, int T, float *__restrict__ tail, const int32_t *__restrict__ pos, int bs) {
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c >= C) return;
    const int p0 = pos[0];
    for (int j = 0; j < T - 1; j++) {
        const int s = bs - (T - 1) + j;
        float v = 0.f;
        if (s >= 0) v = u[(int64_t)s * ldu + c];
        else if (p0 + s >= 0) v = tail[(int64_t)(T - 1 + s) * C + c];
        tail[(int64_t)j * C + c] = v;
    }
}

// single token: convolution and tail in one launch, a thread per channel (it alone touches its channel's tail)
__global__ void __launch_bounds__(256) pa_k_conv_step(const float *__restrict__ u, const float *__restrict__ w, const float *__restrict__ b, int C, int T,
                                                      float *__restrict__ tail, int act_silu, float *__restrict__ y, const int32_t *__restrict__ pos) {
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c >= C) return;
    const int p0 = pos[0];
    const float cur = u[c];
    float acc = b ? b[c] : 0.f;
    for (int j = 0; j < T - 1; j++) {
        const float v = p0 - (T - 1) + j >= 0 ? tail[(int64_t)j * C + c] : 0.f;
        acc = fmaf(w[(int64_t)c * T + j], v, acc);
        if (j > 0) tail[(int64_t)(j - 1) * C + c] = v;
    }
    acc = fmaf(w[(int64_t)c * T + T - 1], cur, acc);
    if (T > 1) tail[(int64_t)(T - 2) * C + c] = cur;
    y[c] = act_silu ? pa_silu(acc) : acc;
}

// one CTA per token; row = [q (qd) | k (kd) | ...], the value rows from v_off on (at the keys when the values are the un-normed keys)
__global__ void __launch_bounds__(256) pa_k_qkv_whole_norm(float *__restrict__ qkv, int ld, int qd, int kd, int vd, const float *__restrict__ wq, const float *__restrict__ wk,
                                                           float eps, float *__restrict__ kc, float *__restrict__ vct, int n_ctx, const int32_t *__restrict__ pos, int v_off) {
    __shared__ float red[8];
    const int t = blockIdx.x, p = pos[t];
    float *row = qkv + (int64_t)t * ld;
    float s = 0.f;
    for (int c = threadIdx.x; c < qd; c += 256) s = fmaf(row[c], row[c], s);
    const float iq = 1.0f / sqrtf(pa_block_sum(s, red) / (float)qd + eps);
    for (int c = threadIdx.x; c < qd; c += 256) row[c] = row[c] * iq * wq[c];
    s = 0.f;
    for (int c = threadIdx.x; c < kd; c += 256) s = fmaf(row[qd + c], row[qd + c], s);
    const float ik = 1.0f / sqrtf(pa_block_sum(s, red) / (float)kd + eps);
    for (int c = threadIdx.x; c < kd; c += 256) kc[(int64_t)p * kd + c] = row[qd + c] * ik * wk[c];
    for (int c = threadIdx.x; c < vd; c += 256) vct[(int64_t)c * n_ctx + p] = row[v_off + c];
}

// grid (entries / 256, tokens); n_heads heads of hd entries from v[t * ld] on; heads h >= h_scaled are multiplied by `scale` after the rotation
__global__ void __launch_bounds__(256) pa_k_rope_heads(float *__restrict__ v, int ld, int n_heads, int hd, PaRope rope, int h_scaled, float scale, const int32_t *__restrict__ pos) {
    const int t = blockIdx.y, p = pos[t], half = rope.dims >> 1;
    float *row = v + (int64_t)t * ld;
    for (int e = blockIdx.x * 256 + threadIdx.x; e < n_heads * hd; e += gridDim.x * 256) {
        const int hh = e / hd, c = e % hd;
        const float sc = hh >= h_scaled ? scale : 1.0f;
        float *x = row + hh * hd;
        if (c >= rope.dims) { x[c] *= sc; continue; }
        if (c >= half) continue; // written by its partner
        const double turns = (double)p * rope.freq[c];
        const float ang = (float)fma(-rint(turns * 0.15915494309189535), 6.283185307179586, turns);
        const float cs = cosf(ang) * rope.mscale, sn = sinf(ang) * rope.mscale;
        const float a = x[c], b = x[c + half];
        x[c] = (a * cs - b * sn) * sc;
        x[c + half] = (b * cs + a * sn) * sc;
    }
}

#define PA_GG_THREADS 128
#define PA_GG_TOK 32      // tokens per round of the side mixer's scan
// What follows an attention that has an output gate and / or a minGRU beside it, on the rows of the first projection
// [.. | gate (od) | z (W) | u (W) | side gate (W)]:
//   CTAs below gate_ctas (grid.y walks the tokens): att[t][c] <- att[t][c] * sigmoid(gate[t][c]) * mix_scale
//   the others (blockIdx.y = 0 only; 32 channels each), tokens strictly in order:  z = sigmoid(z_raw + bz), u = u_raw + bx,
//   cand = u + 1/2 (u >= 0) or sigmoid(u) (u < 0), S <- (1 - z) S + z cand  (S = 0 at position 0 whatever the buffer holds),
//   att[t][od + c] = S * silu(side gate) * side_scale.
// The next product reads att rows of od + W entries against [W_o | W_side_o].
__global__ void __launch_bounds__(PA_GG_THREADS) pa_k_gate_gru(float *__restrict__ att, int ldo, const float *__restrict__ proj, int ld, int od, int g_off, float mix_scale, int gate_ctas,
                                                     int W, int z_off, const float *__restrict__ bz, const float *__restrict__ bx, float side_scale,
                                                     float *__restrict__ state, const int32_t *__restrict__ pos, int bs) {
    if ((int)blockIdx.x < gate_ctas) {
        const int c = blockIdx.x * 128 + threadIdx.x;
        if (c >= od) return;
        for (int t = blockIdx.y; t < bs; t += gridDim.y) {
            const float g = g_off >= 0 ? 1.0f / (1.0f + expf(-proj[(int64_t)t * ld + g_off + c])) : 1.0f;
            att[(int64_t)t * ldo + c] *= g * mix_scale;
        }
        return;
    }
    // 32 channels per CTA, rounds of 32 tokens: the four warps take eight tokens each, fetch their operands and form the gates side by
    // side into shared memory (nothing there depends on S); then warp 0 walks the 32 steps in order, a lane per channel - the same
    // operations per step whatever the round, so the result does not depend on how the prompt was cut
    __shared__ float za[PA_GG_TOK][32], ca[PA_GG_TOK][32], ga[PA_GG_TOK][32];
    if (blockIdx.y != 0) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = ((int)blockIdx.x - gate_ctas) * 32 + lane;
    const bool live = c < W;
    float S = (live && pos[0] > 0) ? state[c] : 0.f;
    const float b0 = live ? bz[c] : 0.f, b1 = live ? bx[c] : 0.f;
    constexpr int PER = PA_GG_TOK / (PA_GG_THREADS / 32);
    for (int t0 = 0; t0 < bs; t0 += PA_GG_TOK) {
        float zr[PER], ur[PER], gr[PER];
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const int t = t0 + warp * PER + i;
            const float *row = proj + (int64_t)min(t, bs - 1) * ld + z_off;
            zr[i] = live ? row[c] : 0.f; ur[i] = live ? row[W + c] : 0.f; gr[i] = live ? row[2 * W + c] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const float u = ur[i] + b1;
            za[warp * PER + i][lane] = 1.0f / (1.0f + expf(-(zr[i] + b0)));
            ca[warp * PER + i][lane] = u >= 0.f ? u + 0.5f : 1.0f / (1.0f + expf(-u));
            ga[warp * PER + i][lane] = pa_silu(gr[i]) * side_scale;
        }
        __syncthreads();
        if (warp == 0 && live) {
            const int n = min(PA_GG_TOK, bs - t0);
#pragma unroll 8
            for (int i = 0; i < n; i++) {
                const float z = za[i][lane];
                S = (1.0f - z) * S + z * ca[i][lane];
                att[(int64_t)(t0 + i) * ldo + od + c] = S * ga[i][lane];
            }
        }
        __syncthreads();
    }
    if (warp == 0 && live) state[c] = S;
}

struct PaRglru {
    const float *y, *x;        // rows of the first projection: the gelu branch and the convolution's input, W channels each (row stride ld)
    int ld;
    const float *u, *g;        // batch: convolved inputs [t][W]; gate logits [t][block][r part | i part] without their biases
    const float *rb, *ib, *sp; // [W]: gate biases, rate * softplus(lam)
    int W, bsz, taps;          // channels, channels per block of the gates' matrices
    const float *conv_w, *conv_b; // [W][taps], [W]
    const bf16 *wri;           // [block][r rows | i rows][bsz]
    float *S, *ring;           // [W]; [taps][W], the convolution's input of position p in row p mod taps
    float *o;                  // S gelu(y), row stride ldo
    int ldo;
    const int32_t *pos;
    int bs;
};
// one step's coefficients from the gate logits: a = exp(-sp r), b = sqrt(1 - a^2) i u (1 - a^2 without cancellation)
__device__ __forceinline__ void pa_rglru_coef(float gr, float gi, float sp, float u, float &a, float &b) {
    const float la = -sp * pa_sigmoid(gr);
    a = expf(la);
    b = sqrtf(-expm1f(2.0f * la)) * pa_sigmoid(gi) * u;
}
__device__ __forceinline__ float pa_gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

// 32 channels per CTA, rounds of 32 tokens: the four warps form the coefficients of eight tokens each (nothing there depends on S), warp
// 0 walks the 32 steps in order, a lane per channel - the same operations per step whatever the round and the cut of the prompt
__global__ void __launch_bounds__(PA_GG_THREADS) pa_k_rglru_scan(const PaRglru a) {
    __shared__ float aa[PA_GG_TOK][32], ba[PA_GG_TOK][32], ya[PA_GG_TOK][32];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane, W = a.W;
    const bool live = c < W;
    const int cc = live ? c : W - 1, blk = cc / a.bsz, gc = blk * 2 * a.bsz + cc % a.bsz;
    const int p0 = a.pos[0];
    float S = p0 > 0 ? a.S[cc] : 0.f;
    const float rb = a.rb[cc], ib = a.ib[cc], sp = a.sp[cc];
    constexpr int PER = PA_GG_TOK / (PA_GG_THREADS / 32);
    for (int t0 = 0; t0 < a.bs; t0 += PA_GG_TOK) {
        float gr[PER], gi[PER], ur[PER], yr[PER];
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const int64_t t = min(t0 + warp * PER + i, a.bs - 1);
            gr[i] = a.g[t * 2 * W + gc]; gi[i] = a.g[t * 2 * W + gc + a.bsz]; ur[i] = a.u[t * W + cc]; yr[i] = a.y[t * a.ld + cc];
        }
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const int s = warp * PER + i;
            pa_rglru_coef(gr[i] + rb, gi[i] + ib, sp, ur[i], aa[s][lane], ba[s][lane]);
            ya[s][lane] = pa_gelu_tanh(yr[i]);
        }
        __syncthreads();
        if (warp == 0 && live) {
            const int n = min(PA_GG_TOK, a.bs - t0);
#pragma unroll 8
            for (int i = 0; i < n; i++) {
                S = fmaf(aa[i][lane], S, ba[i][lane]);
                a.o[(int64_t)(t0 + i) * a.ldo + c] = S * ya[i][lane];
            }
        }
        __syncthreads();
    }
    if (warp == 0 && live) a.S[c] = S;
    // the last taps - 1 inputs of the sequence (older ones than this batch's are in the ring already)
    if (warp == 1 && live)
        for (int t = max(0, a.bs - (a.taps - 1)); t < a.bs; t++) a.ring[(int64_t)((p0 + t) % a.taps) * W + c] = a.x[(int64_t)t * a.ld + c];
}

// grid (channels per block / 8, blocks): a CTA convolves the block's inputs into shared memory, then a warp takes one channel - its r and i
// rows are the pair of dot products (fp32 inputs, never rounded).  The ring has `taps` rows, so the row this token writes (by the channel's
// own CTA) is none of those that the other CTAs read.
__global__ void __launch_bounds__(256) pa_k_dec_rglru(const PaRglru a) {
    extern __shared__ __align__(16) float pa_us[]; // [bsz]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, bsz = a.bsz, blk = blockIdx.y, n = blockIdx.x * 8 + warp;
    const bf16 *wr = a.wri + ((int64_t)blk * 2 * bsz + min(n, bsz - 1)) * bsz, *wi = wr + (int64_t)bsz * bsz;
    pa_prefetch2(wr, wi, 0, bsz, lane);
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    const int p = a.pos[0], T = a.taps;
    for (int c = threadIdx.x; c < bsz; c += 256) {
        const int ch = blk * bsz + c;
        const float cur = a.x[ch];
        float acc = a.conv_b[ch];
        for (int j = 0; j < T - 1; j++) {
            const int q = p - (T - 1) + j;
            acc = fmaf(a.conv_w[(int64_t)ch * T + j], q >= 0 ? a.ring[(int64_t)(q % T) * a.W + ch] : 0.f, acc);
        }
        pa_us[c] = fmaf(a.conv_w[(int64_t)ch * T + T - 1], cur, acc);
        if (c >= blockIdx.x * 8 && c < blockIdx.x * 8 + 8) a.ring[(int64_t)(p % T) * a.W + ch] = cur;
    }
    __syncthreads();
    if (n >= bsz) return;
    float gr, gi;
    pa_dot2<false>(wr, wi, pa_us, bsz, 1.0f, lane, gr, gi);
    if (lane == 0) {
        const int ch = blk * bsz + n;
        float ca, cb;
        pa_rglru_coef(gr + a.rb[ch], gi + a.ib[ch], a.sp[ch], pa_us[n], ca, cb);
        const float S = fmaf(ca, p > 0 ? a.S[ch] : 0.f, cb);
        a.S[ch] = S;
        a.o[ch] = S * pa_gelu_tanh(a.y[ch]);
    }
}

// out[s][t][c] = h[t][c] + (h[t - 1][c] - h[t][c]) mu[s][c]; the row before the batch's first is row (pos - 1) & 1 of `ring` (zeros at
// position 0).  Grid (channels / 256, tokens, sets).
__global__ void __launch_bounds__(256) pa_k_token_shift(const float *__restrict__ h, int dim, const float *__restrict__ mu, const float *__restrict__ ring, const int32_t *__restrict__ pos,
                                                        float *__restrict__ out, int64_t set_stride) {
    const int c = blockIdx.x * 256 + threadIdx.x, t = blockIdx.y;
    if (c >= dim) return;
    const int p0 = pos[0];
    const float v = h[(int64_t)t * dim + c];
    const float b = t > 0 ? h[(int64_t)(t - 1) * dim + c] : p0 > 0 ? ring[(int64_t)((p0 - 1) & 1) * dim + c] : 0.f;
    out[blockIdx.z * set_stride + (int64_t)t * dim + c] = fmaf(b - v, mu[(int64_t)blockIdx.z * dim + c], v);
}
// The decays of a batch, dec[t][n] = act(W2[n] . a1[t] + b[n]): fp32 inputs, never rounded, one chain of FMAs in the order of the single-token
// step's.  Grid (channels / 256, tokens / PA_DC_TOK); a thread takes one channel of PA_DC_TOK tokens.  With `ring` given (a time mixing) the
// launch also leaves the batch's last input h in row (last position) & 1 of the ring - nothing behind the first projection reads the old row.
#define PA_DC_TOK 8
__global__ void __launch_bounds__(256) pa_k_decay(const float *__restrict__ a1, int lda, int rank, const bf16 *__restrict__ w2, const float *__restrict__ b, int n, PaAct act,
                                                  float *__restrict__ dec, int bs, const float *__restrict__ h, int dim, float *__restrict__ ring, const int32_t *__restrict__ pos) {
    extern __shared__ __align__(16) float ls[]; // [rank][PA_DC_TOK]
    const int t0 = blockIdx.y * PA_DC_TOK, c = blockIdx.x * 256 + threadIdx.x;
    if (ring)
        for (int e = (blockIdx.y * gridDim.x + blockIdx.x) * 256 + threadIdx.x; e < dim; e += gridDim.x * gridDim.y * 256)
            ring[(int64_t)((pos[0] + bs - 1) & 1) * dim + e] = h[(int64_t)(bs - 1) * dim + e];
    for (int e = threadIdx.x; e < rank * PA_DC_TOK; e += 256) {
        const int r = e % rank, t = e / rank;
        ls[r * PA_DC_TOK + t] = t0 + t < bs ? a1[(int64_t)(t0 + t) * lda + r] : 0.f;
    }
    __syncthreads();
    if (c >= n) return;
    const bf16 *w = w2 + (int64_t)c * rank;
    float z[PA_DC_TOK] = {};
    auto add = [&](int r, float wv) {
        const float4 u = *reinterpret_cast<const float4 *>(ls + r * PA_DC_TOK), v = *reinterpret_cast<const float4 *>(ls + r * PA_DC_TOK + 4);
        const float x[PA_DC_TOK] = {u.x, u.y, u.z, u.w, v.x, v.y, v.z, v.w};
#pragma unroll
        for (int t = 0; t < PA_DC_TOK; t++) z[t] = fmaf(wv, x[t], z[t]);
    };
    if ((rank & 7) == 0) {
        for (int r = 0; r < rank; r += 8) {
            const uint4 v = __ldg(reinterpret_cast<const uint4 *>(w + r));
            const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int e = 0; e < 4; e++) { add(r + 2 * e, __uint_as_float(u[e] << 16)); add(r + 2 * e + 1, __uint_as_float(u[e] & 0xffff0000u)); }
        }
    } else {
        for (int r = 0; r < rank; r++) add(r, pa_ld(w + r));
    }
    const float bias = b[c];
#pragma unroll
    for (int t = 0; t < PA_DC_TOK; t++)
        if (t0 + t < bs) dec[(int64_t)(t0 + t) * n + c] = pa_act1(z[t] + bias, act);
}

#define PA_SC_TOK 32    // tokens staged per round (half as many for the widest states)
#define PA_SC_FLIGHT 4  // tokens whose outputs are reduced together
#define PA_SC_WARPS 4
#define PA_SC_REGS 16   // state entries per lane
struct PaScan {
    const float *q, *k, *v;   // q[t * ldq + g * q_gs + i], k likewise (i < dk, g = the head's group), v[t * ldv + h * dv + j]
    int ldq, ldk, ldv, q_gs, k_gs;
    int H, G, dk, dv;
    const float *decay;       // [H]: a_t = decay[h], c_t = 1 (dt null)
    const float *dt;          // dt[t * lddt + h] raw step sizes: c_t = softplus(dt + dt_bias[h]), a_t = exp(-exp(a_log[h]) c_t)
    int lddt;
    const float *dt_bias, *a_log, *d_skip; // [H]; d_skip null: no skip term
    const float *dec;         // MODE 1, 2: decays dec[t * lddec + h * dk + i]
    int lddec;
    const float *bonus;       // MODE 2: u [H][dk]
    float o_scale;            // MODE 1, 2: factor on the output
    float *S;                 // [H][dv][dkp]: a value column's state entries lie together, dkp = 16 * pa_scan_il(dk)
    float *o;                 // o[t * ldo + h * dv + j]
    int ldo;
    const int32_t *pos;
    int bs;
};
// lanes that share a value column: every lane holds PA_SC_REGS state entries of it, so dk <= 16 * IL (IL a power of two, at most 16)
static inline int pa_scan_il(int dk) { int il = 1; while (il * PA_SC_REGS < dk) il *= 2; return il; }
static inline int pa_scan_dkp(int dk) { return PA_SC_REGS * pa_scan_il(dk); }
static inline int pa_scan_cols(int dk, int nc) { return 32 / pa_scan_il(dk) * PA_SC_WARPS * nc; } // value columns per CTA, nc per lane
static inline int pa_scan_tok(int dk) { return pa_scan_il(dk) <= 8 ? PA_SC_TOK : PA_SC_TOK / 2; } // tokens staged per round
static inline size_t pa_scan_smem(int dk, int nc, int mode) {
    return 4 * (size_t)pa_scan_tok(dk) * (2 * ((mode ? 3 : 2) * (size_t)pa_scan_dkp(dk) + pa_scan_cols(dk, nc) + 1) + pa_scan_cols(dk, nc) + 2);
}

__device__ __forceinline__ void pa_cp_async4(float *dst_smem, const float *src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst_smem)), "l"(src) : "memory");
}

__device__ __forceinline__ void pa_cp_async16(float *dst_smem, const float *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst_smem)), "l"(src) : "memory");
}

// grid (dv / columns per CTA, H).  A lane owns entries i = (m * IL + li) * 4 + e (m, e < 4) of NC columns: k and q come out of shared
// memory as float4 (lanes of a column read neighbouring float4s, lanes of different columns the same ones) and serve the lane's NC
// columns from registers; the output is reduced over the IL lanes of a column by log2(IL) shuffles, always in the same order (the
// result does not depend on NC).  The q / k / v rows (and raw step sizes) of a round of tokens arrive by asynchronous copies (16 bytes where rows and sizes allow)
// into one of two buffers while the round before is computed.
template <int IL, int NC, int MODE>
__global__ void __launch_bounds__(32 * PA_SC_WARPS) pa_k_scan(const PaScan a) {
    extern __shared__ __align__(16) float sm[];
    constexpr int CW = 32 / IL, CC = CW * PA_SC_WARPS * NC, DKP = PA_SC_REGS * IL, NT = 32 * PA_SC_WARPS, TOK = IL <= 8 ? PA_SC_TOK : PA_SC_TOK / 2;
    constexpr int BUF = TOK * ((MODE ? 3 : 2) * DKP + CC + 1); // floats of one input buffer: q rows, k rows, v entries, raw step sizes (MODE 1, 2: decay rows)
    const int dk = a.dk, dv = a.dv;
    float *os = sm + 2 * BUF, *as = os + TOK * CC, *cs = as + TOK;
    const int h = blockIdx.y, g = h / (a.H / a.G), j0 = blockIdx.x * CC, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int li = lane % IL, col0 = (warp * NC) * CW + lane / IL; // the lane's columns: col0 + c * CW
    const bool fresh = a.pos[0] == 0;
    float S[NC][PA_SC_REGS];
#pragma unroll
    for (int c = 0; c < NC; c++) {
        const int j = j0 + col0 + c * CW;
        const float4 *Sg = reinterpret_cast<const float4 *>(a.S + ((int64_t)h * dv + min(j, dv - 1)) * DKP) + li;
#pragma unroll
        for (int m = 0; m < 4; m++) {
            const float4 v = (!fresh && j < dv) ? Sg[m * IL] : make_float4(0.f, 0.f, 0.f, 0.f);
            S[c][4 * m] = v.x; S[c][4 * m + 1] = v.y; S[c][4 * m + 2] = v.z; S[c][4 * m + 3] = v.w;
        }
    }
    float u[MODE == 2 ? PA_SC_REGS : 1];
    if (MODE == 2) {
#pragma unroll
        for (int e = 0; e < PA_SC_REGS; e++) { // entry (m * IL + li) * 4 + e % 4, m = e / 4
            const int i = ((e >> 2) * IL + li) * 4 + (e & 3);
            u[MODE == 2 ? e : 0] = i < dk ? a.bonus[(int64_t)h * dk + i] : 0.f;
        }
    }
    const float rate = a.dt ? expf(a.a_log[h]) : 0.f, bias = a.dt ? a.dt_bias[h] : 0.f, fixed = (MODE || a.dt) ? 0.f : a.decay[h], skip = a.d_skip ? a.d_skip[h] : 0.f;
    for (int e = tid; e < 2 * BUF; e += NT) sm[e] = 0.f; // what the copies never write (entries beyond dk, columns beyond dv) stays zero
    __syncthreads();
    auto al = [](const float *p, int ld, int n) { return ((reinterpret_cast<uintptr_t>(p) & 15) | ((ld | n) & 3)) == 0; };
    const bool wide = al(a.q, a.ldq, a.q_gs | dk) && al(a.k, a.ldk, a.k_gs) && al(a.v, a.ldv, dv) && (!MODE || al(a.dec, a.lddec, dk));
    auto fetch = [&](int t0, int buf) {
        float *qs = sm + buf * BUF, *ks = qs + TOK * DKP, *vs = ks + TOK * DKP, *ds = vs + TOK * CC;
        const int nt = min(TOK, a.bs - t0);
        for (int tt = warp; tt < nt; tt += PA_SC_WARPS) {
            const float *qr = a.q + (int64_t)(t0 + tt) * a.ldq + g * a.q_gs, *kr = a.k + (int64_t)(t0 + tt) * a.ldk + g * a.k_gs;
            if (wide) {
                for (int i = lane * 4; i < dk; i += 128) {
                    pa_cp_async16(qs + tt * DKP + i, qr + i);
                    pa_cp_async16(ks + tt * DKP + i, kr + i);
                    if (MODE) pa_cp_async16(ds + TOK + tt * DKP + i, a.dec + (int64_t)(t0 + tt) * a.lddec + h * dk + i);
                }
                const float *vr = a.v + (int64_t)(t0 + tt) * a.ldv + h * dv + j0;
                for (int c = lane * 4; c < CC && j0 + c < dv; c += 128) pa_cp_async16(vs + tt * CC + c, vr + c);
                continue;
            }
            for (int i = lane; i < dk; i += 32) {
                pa_cp_async4(qs + tt * DKP + i, qr + i);
                pa_cp_async4(ks + tt * DKP + i, kr + i);
            }
            if (MODE) {
                const float *dr = a.dec + (int64_t)(t0 + tt) * a.lddec + h * dk;
                for (int i = lane; i < dk; i += 32) pa_cp_async4(ds + TOK + tt * DKP + i, dr + i);
            }
            const float *vr = a.v + (int64_t)(t0 + tt) * a.ldv + h * dv + j0;
            for (int c = lane; c < CC && j0 + c < dv; c += 32) pa_cp_async4(vs + tt * CC + c, vr + c);
        }
        if (a.dt)
            for (int tt = tid; tt < nt; tt += NT) pa_cp_async4(ds + tt, a.dt + (int64_t)(t0 + tt) * a.lddt + h);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    for (int t0 = 0, buf = 0; t0 < a.bs; t0 += TOK, buf ^= 1) {
        const int nt = min(TOK, a.bs - t0);
        const float *qs = sm + buf * BUF, *ks = qs + TOK * DKP, *vs = ks + TOK * DKP, *ds = vs + TOK * CC;
        if (t0 + TOK < a.bs) {
            fetch(t0 + TOK, buf ^ 1); // (every thread left that buffer's round behind the barrier that ended it)
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        for (int tt = tid; MODE == 0 && tt < nt; tt += NT) {
            if (a.dt) {
                const float d = pa_softplus(ds[tt] + bias);
                cs[tt] = d;
                as[tt] = expf(-rate * d);
            } else {
                cs[tt] = 1.0f;
                as[tt] = fixed;
            }
        }
        if (MODE == 0) __syncthreads();
        // one token: the state, and the lane's part of the output of its columns
        auto step = [&](int tt, float (&part)[NC]) {
            const float aa = MODE ? 0.f : as[tt], ct = MODE ? 1.0f : cs[tt];
            float x[NC], vv[NC], acc[NC][4];
#pragma unroll
            for (int c = 0; c < NC; c++) {
                x[c] = vs[tt * CC + col0 + c * CW];
                vv[c] = x[c] * ct;
                acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
            }
            const float4 *k4 = reinterpret_cast<const float4 *>(ks + tt * DKP) + li, *q4 = reinterpret_cast<const float4 *>(qs + tt * DKP) + li;
#pragma unroll
            for (int m = 0; m < 4; m++) {
                const float4 kk = k4[m * IL], qq = q4[m * IL];
                if (MODE) {
                    const float4 dd = (reinterpret_cast<const float4 *>(ds + TOK + tt * DKP) + li)[m * IL];
                    const float ke[4] = {kk.x, kk.y, kk.z, kk.w}, qe[4] = {qq.x, qq.y, qq.z, qq.w}, de[4] = {dd.x, dd.y, dd.z, dd.w};
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const float uk = MODE == 2 ? u[MODE == 2 ? 4 * m + e : 0] * ke[e] : 0.f;
#pragma unroll
                        for (int c = 0; c < NC; c++) {
                            float &s = S[c][4 * m + e];
                            if (MODE == 2) acc[c][e] = fmaf(fmaf(uk, vv[c], s), qe[e], acc[c][e]); // the state before, and the bonus
                            s = fmaf(de[e], s, ke[e] * vv[c]);
                            if (MODE == 1) acc[c][e] = fmaf(s, qe[e], acc[c][e]);
                        }
                    }
                    continue;
                }
#pragma unroll
                for (int c = 0; c < NC; c++) {
                    S[c][4 * m] = fmaf(aa, S[c][4 * m], kk.x * vv[c]);         acc[c][0] = fmaf(S[c][4 * m], qq.x, acc[c][0]);
                    S[c][4 * m + 1] = fmaf(aa, S[c][4 * m + 1], kk.y * vv[c]); acc[c][1] = fmaf(S[c][4 * m + 1], qq.y, acc[c][1]);
                    S[c][4 * m + 2] = fmaf(aa, S[c][4 * m + 2], kk.z * vv[c]); acc[c][2] = fmaf(S[c][4 * m + 2], qq.z, acc[c][2]);
                    S[c][4 * m + 3] = fmaf(aa, S[c][4 * m + 3], kk.w * vv[c]); acc[c][3] = fmaf(S[c][4 * m + 3], qq.w, acc[c][3]);
                }
            }
#pragma unroll
            for (int c = 0; c < NC; c++) part[c] = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
        };
        // ... reduced over the column's lanes in the same order for every token
        auto finish = [&](int tt, float (&part)[NC]) {
#pragma unroll
            for (int c = 0; c < NC; c++)
                if (li == 0) os[tt * CC + col0 + c * CW] = MODE ? part[c] * a.o_scale : fmaf(skip, vs[tt * CC + col0 + c * CW], part[c]);
        };
        int tt = 0;
        for (; tt + PA_SC_FLIGHT <= nt; tt += PA_SC_FLIGHT) { // several tokens in flight: nothing is stored between their loads
            float part[PA_SC_FLIGHT][NC];
#pragma unroll
            for (int f = 0; f < PA_SC_FLIGHT; f++) step(tt + f, part[f]);
#pragma unroll
            for (int o = IL / 2; o; o >>= 1)
#pragma unroll
                for (int f = 0; f < PA_SC_FLIGHT; f++)
#pragma unroll
                    for (int c = 0; c < NC; c++) part[f][c] += __shfl_xor_sync(0xffffffffu, part[f][c], o);
#pragma unroll
            for (int f = 0; f < PA_SC_FLIGHT; f++) finish(tt + f, part[f]);
        }
        for (; tt < nt; tt++) {
            float part[NC];
            step(tt, part);
#pragma unroll
            for (int o = IL / 2; o; o >>= 1)
#pragma unroll
                for (int c = 0; c < NC; c++) part[c] += __shfl_xor_sync(0xffffffffu, part[c], o);
            finish(tt, part);
        }
        __syncthreads();
        for (int tt = warp; tt < nt; tt += PA_SC_WARPS) {
            float *orow = a.o + (int64_t)(t0 + tt) * a.ldo + h * dv + j0;
            for (int c = lane; c < CC; c += 32)
                if (j0 + c < dv) orow[c] = os[tt * CC + c];
        }
    }
#pragma unroll
    for (int c = 0; c < NC; c++) {
        const int j = j0 + col0 + c * CW;
        if (j >= dv) continue;
        float4 *Sg = reinterpret_cast<float4 *>(a.S + ((int64_t)h * dv + j) * DKP) + li;
#pragma unroll
        for (int m = 0; m < 4; m++) Sg[m * IL] = make_float4(S[c][4 * m], S[c][4 * m + 1], S[c][4 * m + 2], S[c][4 * m + 3]);
    }
}

// One token of a recurrence with a decay per key channel, and what stands around it.  A cluster of gridDim.x CTAs takes head blockIdx.y, each
// CTA an equal share of its value columns:
//   decay_i = dact(W_a2[h dk + i] . a1 + b)   (fp32 inputs, never rounded; every CTA of the head forms all dk of them)
//   bonus null:  S <- diag(decay) S + k v^T, o = S^T q o_scale;   bonus given:  o = (S + diag(u) k v^T)^T q o_scale, then the same update
//   out = o / sqrt(mean(o^2) + eps) * norm_w * silu(g)   with the mean over the head's dv columns (partial sums through distributed shared memory)
struct PaRecStep {
    const float *q, *k, *v, *g, *a1;
    const bf16 *a2;
    const float *a2b;
    int rank;
    PaAct dact;
    const float *bonus;   // [H][dk]
    float o_scale;
    float *S;             // [H][dv][dkp]
    const float *norm_w;  // [H * dv]
    float eps;
    float *out;
    const int32_t *pos;
    int dk, dv, dkp, lg;  // lg: log2 of the lanes that share a value column (dkp / 16)
};
static inline size_t pa_rec_step_smem(int dkp, int cols, int rank) { return 4 * ((size_t)4 * dkp + 3 * (size_t)cols + rank); }

__global__ void __launch_bounds__(256) pa_k_dec_recur(const PaRecStep a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[8], part_s;
    cg::cluster_group cl = cg::this_cluster();
    const int n_cl = gridDim.x, h = blockIdx.y, cols = (a.dv + n_cl - 1) / n_cl, j0 = blockIdx.x * cols, nc = max(0, min(cols, a.dv - j0)), dk = a.dk, dkp = a.dkp;
    float *qs = sm, *ks = qs + dkp, *ds = ks + dkp, *us = ds + dkp, *vs = us + dkp, *gs = vs + cols, *os = gs + cols, *ls = os + cols;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float *Sh = a.S + ((int64_t)h * a.dv + j0) * dkp;
    // neither a weight nor the state's address depends on the kernel before: on their way to L2 (the state is read behind the wait)
    for (int e = tid * 32; e < nc * dkp; e += 256 * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(Sh + e));
    for (int e = tid * 64; e < dk * a.rank; e += 256 * 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.a2 + (int64_t)h * dk * a.rank + e));
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    const bool fresh = a.pos[0] == 0;
    for (int i = tid; i < dkp; i += 256) {
        const bool in = i < dk;
        qs[i] = in ? a.q[h * dk + i] : 0.f;
        ks[i] = in ? a.k[h * dk + i] : 0.f;
        us[i] = in && a.bonus ? a.bonus[h * dk + i] : 0.f;
    }
    for (int j = tid; j < nc; j += 256) { vs[j] = a.v[h * a.dv + j0 + j]; gs[j] = pa_silu(a.g[h * a.dv + j0 + j]); }
    for (int r = tid; r < a.rank; r += 256) ls[r] = a.a1[r];
    __syncthreads();
    for (int i = tid; i < dkp; i += 256) {
        float d = 0.f;
        if (i < dk) {
            const bf16 *w = a.a2 + ((int64_t)h * dk + i) * a.rank;
            float z = 0.f;
            if ((a.rank & 7) == 0) {
                for (int r = 0; r < a.rank; r += 8) {
                    const uint4 v = __ldg(reinterpret_cast<const uint4 *>(w + r));
                    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                    for (int t = 0; t < 4; t++) {
                        z = fmaf(__uint_as_float(u[t] << 16), ls[r + 2 * t], z);
                        z = fmaf(__uint_as_float(u[t] & 0xffff0000u), ls[r + 2 * t + 1], z);
                    }
                }
            } else {
                for (int r = 0; r < a.rank; r++) z = fmaf(pa_ld(w + r), ls[r], z);
            }
            d = pa_act1(z + a.a2b[h * dk + i], a.dact);
        }
        ds[i] = d;
    }
    __syncthreads();
    // 2^lg lanes share a value column, 16 state entries each (the layout of pa_k_scan); entries beyond dk are zero and stay zero
    const int il = 1 << a.lg, li = lane & (il - 1), per_warp = 32 >> a.lg;
    float ss = 0.f;
    for (int jb = warp * per_warp; jb < nc; jb += 8 * per_warp) {
        const int j = jb + (lane >> a.lg), jj = min(j, nc - 1);
        float4 *Sg = reinterpret_cast<float4 *>(Sh + (int64_t)jj * dkp) + li;
        const float v = vs[jj];
        float4 s[4];
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int m = 0; m < 4; m++) s[m] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : Sg[m * il];
#pragma unroll
        for (int m = 0; m < 4; m++) {
            const float4 kk = (reinterpret_cast<const float4 *>(ks) + li)[m * il], qq = (reinterpret_cast<const float4 *>(qs) + li)[m * il], dd = (reinterpret_cast<const float4 *>(ds) + li)[m * il],
                         uu = (reinterpret_cast<const float4 *>(us) + li)[m * il];
            const float ke[4] = {kk.x, kk.y, kk.z, kk.w}, qe[4] = {qq.x, qq.y, qq.z, qq.w}, de[4] = {dd.x, dd.y, dd.z, dd.w}, ue[4] = {uu.x, uu.y, uu.z, uu.w};
            float se[4] = {s[m].x, s[m].y, s[m].z, s[m].w};
#pragma unroll
            for (int e = 0; e < 4; e++) {
                if (a.bonus) acc[e] = fmaf(fmaf(ue[e] * ke[e], v, se[e]), qe[e], acc[e]);
                se[e] = fmaf(de[e], se[e], ke[e] * v);
                if (!a.bonus) acc[e] = fmaf(se[e], qe[e], acc[e]);
            }
            s[m] = make_float4(se[0], se[1], se[2], se[3]);
        }
        float r = (acc[0] + acc[1]) + (acc[2] + acc[3]);
        for (int o = il / 2; o; o >>= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
        if (j < nc) {
#pragma unroll
            for (int m = 0; m < 4; m++) Sg[m * il] = s[m];
            if (li == 0) { r *= a.o_scale; os[j] = r; ss = fmaf(r, r, ss); }
        }
    }
    const float mine = pa_block_sum(ss, red);
    if (tid == 0) part_s = mine;
    cl.sync();
    float t = 0.f;
    for (int c = 0; c < n_cl; c++) t += *cl.map_shared_rank(&part_s, c);
    const float inv = 1.0f / sqrtf(t / (float)a.dv + a.eps);
    for (int j = tid; j < nc; j += 256) a.out[h * a.dv + j0 + j] = os[j] * inv * a.norm_w[h * a.dv + j0 + j] * gs[j];
    cl.sync(); // no CTA leaves while another reads its partial sum
}

// one CTA per (part, token); `width` entries in `parts` equal parts.  gate_first: out = N(y silu(g)) * w; else out = N(y) * silu(g) (w null: 1)
__global__ void __launch_bounds__(256) pa_k_gate_norm(const float *__restrict__ y, int ldy, const float *__restrict__ gate, int ldg, int width, int parts,
                                                      const float *__restrict__ w, int gate_first, float eps, float *__restrict__ out, int ldo) {
    __shared__ float red[8];
    const int t = blockIdx.y, ps = width / parts;
    const float *yr = y + (int64_t)t * ldy, *gr = gate + (int64_t)t * ldg;
    float *orow = out + (int64_t)t * ldo;
    {
        const int c0 = blockIdx.x * ps;
        float s = 0.f;
        for (int c = threadIdx.x; c < ps; c += 256) {
            const float v = gate_first ? yr[c0 + c] * pa_silu(gr[c0 + c]) : yr[c0 + c];
            s = fmaf(v, v, s);
        }
        const float inv = 1.0f / sqrtf(pa_block_sum(s, red) / (float)ps + eps);
        for (int c = threadIdx.x; c < ps; c += 256) {
            const float gsl = pa_silu(gr[c0 + c]), wv = w ? w[c0 + c] : 1.0f;
            orow[c0 + c] = gate_first ? yr[c0 + c] * gsl * inv * wv : yr[c0 + c] * inv * wv * gsl;
        }
    }
}

// norm first (out = N(y) w silu(g)), parts of at most 256 entries: a warp per part, eight parts per CTA.  Grid (parts / 8, tokens)
__global__ void __launch_bounds__(256) pa_k_gate_norm_warp(const float *__restrict__ y, int ldy, const float *__restrict__ gate, int ldg, int ps, int parts, const float *__restrict__ w, float eps,
                                                           float *__restrict__ out, int ldo) {
    const int t = blockIdx.y, part = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (part >= parts) return;
    const float *yr = y + (int64_t)t * ldy + part * ps, *gr = gate + (int64_t)t * ldg + part * ps;
    float v[8], g[8], s = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const int c = lane + 32 * i;
        v[i] = c < ps ? yr[c] : 0.f;
        g[i] = c < ps ? gr[c] : 0.f;
        s = fmaf(v[i], v[i], s);
    }
#pragma unroll
    for (int o = 16; o; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    const float inv = 1.0f / sqrtf(s / (float)ps + eps);
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const int c = lane + 32 * i;
        if (c < ps) out[(int64_t)t * ldo + part * ps + c] = v[i] * inv * (w ? w[part * ps + c] : 1.0f) * pa_silu(g[i]);
    }
}

// out[t][c] = sum_r slot[t][r][c] + sgate[t] * shared[t][c]   (shared null: no shared expert; sgate null: 1); a choice sel_e[t][r] >= E
// stands for the input itself: sel_w[t][r] * x[t][c]
__global__ void __launch_bounds__(256) pa_k_moe_sum(float *__restrict__ out, const float *__restrict__ slot, int top, const float *__restrict__ shared,
                                                    const float *__restrict__ sgate, int dim, const int *__restrict__ sel_e = nullptr, const float *__restrict__ sel_w = nullptr,
                                                    const float *__restrict__ x = nullptr, int E = 0) {
    const int t = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    if (c >= dim) return;
    float y = 0.f;
    for (int r = 0; r < top; r++) {
        if (x && sel_e[t * top + r] >= E) y = fmaf(sel_w[t * top + r], x[(int64_t)t * dim + c], y);
        else y += slot[((int64_t)t * top + r) * dim + c];
    }
    if (shared) y += (sgate ? sgate[t] : 1.0f) * shared[(int64_t)t * dim + c];
    out[(int64_t)t * dim + c] = y;
}
