// ps_arch_decode.cuh - single-token (bs == 1) kernels of the layer-list executor: six launches per parallel block (seven per
// sequential block with windowed attention, eleven with latent attention; three to six per general parallel block), every one independent of the position except through
// device memory, so the step is captured once and replayed as a CUDA graph.
//
//   pa_k_dec_mv          weight-streaming mat-vec (bfloat16 rows, 16-byte loads, two rows per warp) with fused prologue / epilogue:
//                          norm of the residual stream in the prologue (q|k|v + router rows, lm_head),
//                          bias, K row / V^T column straight into the cache, router logits from the UNROUNDED fp32 input,
//                          residual add (output projection of a layer without a feed-forward);
//                          sequential blocks: the seam in the prologue (the pending sublayer output joins the residual stream through
//                          its group norm, the sum is group-normed for this product; CTA 0 stores the sum to the second residual buffer),
//                          per-head products (a row reads its head's slice of the input);
//                          general parallel blocks: one range of rows leaves through the feed-forward's activation; a pass projection
//                          appends the embedding output to the seam's sum;
//                          time mixing: ranges of rows read different mixtures of the normed input with the token before's
//   pa_k_dec_scores      scores of all heads for 16 keys per CTA (thread per key and head out of shared memory), distance bias (table,
//                        logarithmic or linear), head mixing, norms and rotation of q and of the token's own key per head, rotation of its value, per-block soft-max statistics; with a window the grid starts at the first
//                        key in sight; pooled windows: further CTAs take 16 block means each, and the last CTA forms the mean of the
//                        block that the token completes
//   pa_k_dec_pv          soft-max statistics (+ sink logit) per head, weights staged once per CTA, P.V along contiguous V^T rows; many
//                        heads over one kv head are split over blockIdx.z
//   pa_k_dec_dense_up    seam in the prologue, gate | up rows of a dense feed-forward (or of a shared expert, then with the router's
//                        logits as further rows), activation; without a gate a warp's pair is two neighbouring up rows
//   pa_k_dec_latent_q    latent attention with queries from the input: W_uk folded into the query, both rotations, latent and rotated key
//                        part into the cache
//   pa_k_dec_token_input per-layer token input: seam, gate rows, the token's table row and the projection in one cluster
//   pa_k_dec_expert_up   norm + top-k of the router scores in the prologue, gate | up rows of the chosen experts, activation
//   pa_k_dec_expert_down down rows of the chosen experts summed over the slots + mixer output + residual (or, for the next seam, + the
//                        shared expert's down rows behind its gate + the input itself for identity outputs)
#pragma once
#include "ps_ptx.cuh"

#define PA_DV_THREADS 256
#define PA_DV_ROWS 16       // output rows per mat-vec CTA: 8 warps x 2 rows
#define PA_DS_KEYS 16       // keys per CTA of the decode scores kernel
#define PA_DP_DIMS 4        // value dims per CTA of the decode P.V kernel (two warps each)
#define PA_DP_FLOATS 10240  // staged floats per CTA of the P.V kernel: (PA_DP_DIMS + heads per kv head) x chunk keys

// two rows at once: s0 += w0 . f(x), s1 += w1 . f(x) with f = bfloat16 rounding (ROUND) of x * xscale, or identity
template <bool ROUND>
__device__ __forceinline__ void pa_dot2(const bf16 *__restrict__ w0, const bf16 *__restrict__ w1, const float *x, int K, float xscale, int lane, float &s0, float &s1,
                                        int k_begin, int k_end) {
    s0 = s1 = 0.f;
    if (k_end < 0) k_end = K;
    if ((K & 7) == 0 && (k_begin & 7) == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0) { // (a head's slice of x may start anywhere)
#pragma unroll 4
        for (int k = k_begin + lane * 8; k < k_end; k += 256) {
            const uint4 a = __ldg(reinterpret_cast<const uint4 *>(w0 + k));
            const uint4 b = __ldg(reinterpret_cast<const uint4 *>(w1 + k));
            const float4 x0 = *reinterpret_cast<const float4 *>(x + k), x1 = *reinterpret_cast<const float4 *>(x + k + 4);
            const float xv[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
            const uint32_t au[4] = {a.x, a.y, a.z, a.w}, bu[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int t = 0; t < 4; t++) {
                const float xa = pa_rnd<ROUND>(xv[2 * t] * xscale), xb = pa_rnd<ROUND>(xv[2 * t + 1] * xscale);
                s0 = fmaf(__uint_as_float(au[t] << 16), xa, s0);
                s0 = fmaf(__uint_as_float(au[t] & 0xffff0000u), xb, s0);
                s1 = fmaf(__uint_as_float(bu[t] << 16), xa, s1);
                s1 = fmaf(__uint_as_float(bu[t] & 0xffff0000u), xb, s1);
            }
        }
    } else {
        for (int k = k_begin + lane; k < k_end; k += 32) {
            const float xa = pa_rnd<ROUND>(x[k] * xscale);
            s0 = fmaf(__bfloat162float(w0[k]), xa, s0);
            s1 = fmaf(__bfloat162float(w1[k]), xa, s1);
        }
    }
#pragma unroll
    for (int o = 16; o; o >>= 1) { s0 += __shfl_xor_sync(0xffffffffu, s0, o); s1 += __shfl_xor_sync(0xffffffffu, s1, o); }
}

// ask L2 for a warp's slice of two weight rows before the prologue's barriers: the stream then starts from L2
__device__ __forceinline__ void pa_prefetch2(const bf16 *w0, const bf16 *w1, int k_begin, int k_end, int lane) {
    for (int k = k_begin + lane * 64; k < k_end; k += 32 * 64) {
        asm volatile("prefetch.global.L2 [%0];" ::"l"(w0 + k));
        asm volatile("prefetch.global.L2 [%0];" ::"l"(w1 + k));
    }
}

// block-wide: hs[k] = x[k] / sqrt(mean(x^2) + eps) * w[k]  (w holds 1 + weight for unit-offset norms); 256 threads
__device__ __forceinline__ void pa_norm_to_smem(float *hs, const float *__restrict__ x, const float *__restrict__ w, int dim, float eps) {
    __shared__ float red[8];
    __shared__ float inv_s;
    float s = 0.f;
    for (int c = threadIdx.x; c < dim; c += blockDim.x) s = fmaf(x[c], x[c], s);
#pragma unroll
    for (int o = 16; o; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = s;
    __syncthreads();
    if (threadIdx.x == 0) {
        float t = 0.f;
        for (int i = 0; i < (int)(blockDim.x >> 5); i++) t += red[i];
        inv_s = 1.0f / sqrtf(t / (float)dim + eps);
    }
    __syncthreads();
    const float inv = inv_s;
    for (int c = threadIdx.x; c < dim; c += blockDim.x) hs[c] = x[c] * inv * w[c];
    __syncthreads();
}

struct PaNoHook { __device__ __forceinline__ void operator()() const {} };
// the seam below for one part whose vectors fit into registers (dim a multiple of 4, at most 16 NT): every load of a phase is in flight at
// once, the sums come out of registers.  `between` runs behind the first loads.
template <int NT, typename F>
__device__ __forceinline__ void pa_seam_regs(float *hs, const float *__restrict__ x, const float *__restrict__ y, const float *__restrict__ w_out, const float *__restrict__ w_in,
                                             float *__restrict__ x_out, int dim, float eps, int center, const float *__restrict__ add_tok, const float *__restrict__ add_vec, float y_scale, float *red,
                                             const F &between) {
    constexpr int V = 4;
    const int n4 = dim >> 2, tid = threadIdx.x;
    auto ld = [&](const float *p, int c) { return p && c < n4 ? reinterpret_cast<const float4 *>(p)[c] : make_float4(0.f, 0.f, 0.f, 0.f); };
    auto stats = [&](const float4 (&v)[V], float &mu) { // 1 / sqrt(mean((v - mu)^2) + eps)
        mu = 0.f;
        if (center) {
            float m = 0.f;
#pragma unroll
            for (int i = 0; i < V; i++) m += (v[i].x + v[i].y) + (v[i].z + v[i].w);
            mu = pa_block_sum(m, red) / (float)dim;
        }
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < V; i++) {
            if (tid + i * NT >= n4) continue;
            const float a = v[i].x - mu, b = v[i].y - mu, c = v[i].z - mu, d = v[i].w - mu;
            s = fmaf(a, a, s); s = fmaf(b, b, s); s = fmaf(c, c, s); s = fmaf(d, d, s);
        }
        return 1.0f / sqrtf(pa_block_sum(s, red) / (float)dim + eps);
    };
    float4 v[V];
    {
        float4 t[V];
#pragma unroll
        for (int i = 0; i < V; i++) { t[i] = ld(y, tid + i * NT); v[i] = ld(x, tid + i * NT); }
        between();
        if (y && w_out) {
            float4 w[V];
#pragma unroll
            for (int i = 0; i < V; i++) w[i] = ld(w_out, tid + i * NT);
            float mu;
            const float f = stats(t, mu) * y_scale;
#pragma unroll
            for (int i = 0; i < V; i++) {
                v[i].x = fmaf((t[i].x - mu) * f, w[i].x, v[i].x); v[i].y = fmaf((t[i].y - mu) * f, w[i].y, v[i].y);
                v[i].z = fmaf((t[i].z - mu) * f, w[i].z, v[i].z); v[i].w = fmaf((t[i].w - mu) * f, w[i].w, v[i].w);
            }
        } else if (y) {
#pragma unroll
            for (int i = 0; i < V; i++) { v[i].x = fmaf(y_scale, t[i].x, v[i].x); v[i].y = fmaf(y_scale, t[i].y, v[i].y); v[i].z = fmaf(y_scale, t[i].z, v[i].z); v[i].w = fmaf(y_scale, t[i].w, v[i].w); }
        }
    }
    if (add_tok || add_vec) {
#pragma unroll
        for (int i = 0; i < V; i++) {
            const float4 p = ld(add_tok, tid + i * NT), q = ld(add_vec, tid + i * NT);
            v[i].x += p.x + q.x; v[i].y += p.y + q.y; v[i].z += p.z + q.z; v[i].w += p.w + q.w;
        }
    }
    if (x_out && blockIdx.x == 0 && blockIdx.y == 0) {
#pragma unroll
        for (int i = 0; i < V; i++)
            if (tid + i * NT < n4) reinterpret_cast<float4 *>(x_out)[tid + i * NT] = v[i];
    }
    if (w_in) {
        float4 w[V];
#pragma unroll
        for (int i = 0; i < V; i++) w[i] = ld(w_in, tid + i * NT);
        float mu;
        const float f = stats(v, mu);
#pragma unroll
        for (int i = 0; i < V; i++) { v[i].x = (v[i].x - mu) * f * w[i].x; v[i].y = (v[i].y - mu) * f * w[i].y; v[i].z = (v[i].z - mu) * f * w[i].z; v[i].w = (v[i].w - mu) * f * w[i].w; }
    }
#pragma unroll
    for (int i = 0; i < V; i++)
        if (tid + i * NT < n4) reinterpret_cast<float4 *>(hs)[tid + i * NT] = v[i];
    __syncthreads();
}

// norm weights on their way to L2 before the dependency wait (a few CTAs ask for all)
__device__ __forceinline__ void pa_prefetch_norms(const float *a, const float *b, int dim) {
    if (blockIdx.x >= 2 || blockIdx.y) return;
    for (int c = threadIdx.x * 32; c < dim; c += blockDim.x * 32) {
        if (a) asm volatile("prefetch.global.L2 [%0];" ::"l"(a + c));
        if (b) asm volatile("prefetch.global.L2 [%0];" ::"l"(b + c));
    }
}

// block-wide seam between two blocks (NT threads): hs = G(x + y_scale P(y) + add_tok + add_vec; w_in) with P(y) = G(y; w_out) (w_out
// null: y itself; y / add_tok / add_vec null: nothing joins), G over `groups` equal parts, the part's mean taken off first when
// `center`.  CTA 0 also stores the updated residual to x_out - a buffer other than x, which the other CTAs are still reading.
template <int NT = 256, typename F = PaNoHook>
__device__ __forceinline__ void pa_seam_to_smem(float *hs, const float *__restrict__ x, const float *__restrict__ y, const float *__restrict__ w_out,
                                                const float *__restrict__ w_in, float *__restrict__ x_out, int dim, int groups, float eps, int center = 0,
                                                const float *__restrict__ add_tok = nullptr, const float *__restrict__ add_vec = nullptr, float y_scale = 1.0f,
                                                const F &between = F{}) {
    __shared__ float red[NT / 32];
    if (groups == 1 && (dim & 3) == 0 && dim <= 16 * NT) {
        pa_seam_regs<NT>(hs, x, y, w_out, w_in, x_out, dim, eps, center, add_tok, add_vec, y_scale, red, between);
        return;
    }
    between();
    const int gs = dim / groups;
    for (int g = 0; g < groups; g++) {
        const int c0 = g * gs;
        float inv = 1.0f, mu = 0.f;
        if (y && w_out) inv = pa_block_stats<NT>(y + c0, gs, center, eps, red, mu);
        for (int c = threadIdx.x; c < gs; c += NT) {
            float v = x[c0 + c];
            if (y) v += y_scale * (w_out ? (y[c0 + c] - mu) * inv * w_out[c0 + c] : y[c0 + c]);
            if (add_tok || add_vec) v += (add_tok ? add_tok[c0 + c] : 0.f) + (add_vec ? add_vec[c0 + c] : 0.f);
            hs[c0 + c] = v;
            if (x_out && blockIdx.x == 0 && blockIdx.y == 0) x_out[c0 + c] = v;
        }
        if (w_in) {
            float mu2;
            const float inv2 = pa_block_stats<NT>(hs + c0, gs, center, eps, red, mu2); // (a thread's own entries)
            for (int c = threadIdx.x; c < gs; c += NT) hs[c0 + c] = (hs[c0 + c] - mu2) * inv2 * w_in[c0 + c];
        }
    }
    __syncthreads();
}

struct PaMv {
    const float *x;        // input vector [K]
    const float *norm_w;   // non-null: the input is normed first (K = model width)
    float eps;
    // sequential blocks (groups > 0): the input is the seam G(x + P(seam_y; seam_w); norm_w); CTA 0 stores x + P(..) to x_out
    int groups;
    const float *seam_y, *seam_w;
    float *x_out;
    int center;            // the norms take the mean off first
    float y_scale;         // factor on seam_y's part
    float *h_out;          // non-null: CTA 0 stores the seam's result (the normed input) there as well
    const float *cat;      // non-null: the seam covers the first seam_dim inputs only, these K - seam_dim values follow
    int seam_dim;
    const float *add_tok, *add_vec; // what a new pass of a looped model adds to the stream at this seam (null: nothing)
    // per-head products (grp_rows > 0): rows [g * grp_rows, (g + 1) * grp_rows) read x + g * x_gs and write y + g * y_gs
    int grp_rows, x_gs, y_gs;
    const bf16 *W;         // [N][K]
    const float *bias;     // [N] or null
    int N, K;
    float *y;              // [N] (rows routed to the cache below are not stored here)
    float *residual;       // non-null: residual[n] += result instead of y[n] = result
    // q | k | v routing of the rows: [0, qd) -> y, [qd, qd + kd) -> K cache row `pos`, then vd rows -> V^T column `pos` (kd = vd = 0: none)
    int qd, kd, vd;
    float *kc, *vct;
    int n_ctx;
    const int32_t *pos;
    int v_is_k;            // the K rows are the value rows as well: each goes to the K cache row AND to its V^T column (vd = 0)
    // extra fp32-input rows after the N weight rows: router logits z[e] = Wr[e] . h (h unrounded)
    const bf16 *Wr;
    int E;
    float *z;
    const float *zbias;    // [E] or null
    // rows n >= act_from (> 0) leave through the one-argument activation, `gap` entries further on
    int act_from, gap;
    PaAct act;
    // rows that read different mixtures of the normed input (seg_n > 0; with groups > 0): rows below seg_end[0] read h, rows from
    // seg_end[s - 1] to seg_end[s] read h + (h' - h) mu[s - 1] with h' the token before's h: row (pos - 1) & 1 of the ring [2][K], zeros at
    // position 0; CTA 0 stores h to row pos & 1.  Every CTA takes neighbouring row groups and forms only the mixtures they read.
    int seg_n, seg_end[6];
    const float *mu;
    float *ring;
    int ksplit;            // warps of a CTA that share a row pair, each taking K / ksplit of the columns (1, 2, 4 or 8)
    int prefetch;          // 1: request the first row group into L2 before the dependency wait; 2: also every next group one ahead
};

template <bool ROUND>
__global__ void __launch_bounds__(PA_DV_THREADS, 4) pa_k_dec_mv(const PaMv a) {
    extern __shared__ __align__(16) float pa_hs[];
    __shared__ float part_s[8][2];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int ks = a.ksplit, pairs = 8 / ks, pair = warp % pairs, slice = warp / pairs;
    const int total = a.N + a.E;
    const int groups = (total + 2 * pairs - 1) / (2 * pairs); // row groups of `pairs` row pairs; the CTAs walk them with the grid's stride
    const int kc = a.K / ks, k_begin = slice * kc, k_end = slice == ks - 1 ? a.K : k_begin + kc;
    // rows of a pair: weight rows below N, router rows (fp32 input, never rounded) from N on
    auto row = [&](int n) { return n < a.N ? a.W + (int64_t)n * a.K : a.Wr + (int64_t)(n - a.N) * a.K; };
    auto prefetch = [&](int grp) {
        const int n0 = (grp * pairs + pair) * 2;
        if (a.prefetch && n0 < total) pa_prefetch2(row(n0), row(min(n0 + 1, total - 1)), k_begin, k_end, lane);
    };
    // row groups of this CTA: every gridDim.x-th, or (mixtures) a run of neighbours
    const int per_cta = (groups + (int)gridDim.x - 1) / (int)gridDim.x;
    const int g_begin = a.seg_n > 0 ? blockIdx.x * per_cta : blockIdx.x, g_end = a.seg_n > 0 ? min(groups, g_begin + per_cta) : groups, g_step = a.seg_n > 0 ? 1 : gridDim.x;
    auto segment = [&](int n) { int sg = 0; while (sg < a.seg_n - 1 && n >= a.seg_end[sg]) sg++; return sg; };
    prefetch(g_begin);
    pa_prefetch_norms(a.seam_w, a.norm_w, a.groups > 0 ? (a.cat ? a.seam_dim : a.K) : 0);
    // launched with programmatic stream serialisation: everything above touches weights only and overlaps the kernel before
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    const float *xin = a.x;
    if (a.groups > 0) {
        const int sd = a.cat ? a.seam_dim : a.K;
        pa_seam_to_smem(pa_hs, a.x, a.seam_y, a.seam_w, a.norm_w, a.x_out, sd, a.groups, a.eps, a.center, a.add_tok, a.add_vec, a.y_scale);
        if (a.cat) {
            for (int c = threadIdx.x; c < a.K - sd; c += PA_DV_THREADS) pa_hs[sd + c] = a.cat[c];
            __syncthreads();
        }
        if (a.h_out && blockIdx.x == 0)
            for (int c = threadIdx.x; c < sd; c += PA_DV_THREADS) a.h_out[c] = pa_hs[c];
        if (a.seg_n > 0) {
            const int p = a.pos[0], s_lo = segment(g_begin * 2 * pairs), s_hi = segment(min(g_end * 2 * pairs, total) - 1);
            const float *prev = a.ring + (int64_t)((p - 1) & 1) * a.K;
            float *keep = a.ring + (int64_t)(p & 1) * a.K;
            for (int c = threadIdx.x; c < a.K; c += PA_DV_THREADS) {
                const float h = pa_hs[c], d = (p > 0 ? prev[c] : 0.f) - h;
                if (blockIdx.x == 0) keep[c] = h;
                for (int sg = max(s_lo, 1); sg <= s_hi; sg++) pa_hs[sg * a.K + c] = fmaf(d, a.mu[(int64_t)(sg - 1) * a.K + c], h);
            }
            __syncthreads();
        }
        xin = pa_hs;
    } else if (a.norm_w) {
        pa_norm_to_smem(pa_hs, a.x, a.norm_w, a.K, a.eps);
        xin = pa_hs;
    }
    for (int grp = g_begin; grp < g_end; grp += g_step) {
        if (a.prefetch > 1 && grp + g_step < g_end) prefetch(grp + g_step); // opt-in: the next group's rows travel to L2 meanwhile
        const int n0 = (grp * pairs + pair) * 2, n1 = min(n0 + 1, total - 1);
        const bool live = n0 < total;
        float s0 = 0.f, s1 = 0.f;
        if (live) {
            const bf16 *w0 = row(n0), *w1 = row(n1);
            if (a.seg_n > 0) {
                const int e0 = segment(n0), e1 = segment(n1);
                if (e0 == e1) {
                    pa_dot2<ROUND>(w0, w1, xin + e0 * a.K, a.K, 1.0f, lane, s0, s1, k_begin, k_end);
                } else {
                    float t;
                    pa_dot2<ROUND>(w0, w0, xin + e0 * a.K, a.K, 1.0f, lane, s0, t, k_begin, k_end);
                    pa_dot2<ROUND>(w1, w1, xin + e1 * a.K, a.K, 1.0f, lane, s1, t, k_begin, k_end);
                }
            } else if (a.grp_rows > 0 && n0 / a.grp_rows == n1 / a.grp_rows) {
                pa_dot2<ROUND>(w0, w1, xin + (n0 / a.grp_rows) * a.x_gs, a.K, 1.0f, lane, s0, s1, k_begin, k_end);
            } else if (a.grp_rows > 0) { // every row reads its own head's slice of x
                float t;
                pa_dot2<ROUND>(w0, w0, xin + (n0 / a.grp_rows) * a.x_gs, a.K, 1.0f, lane, s0, t, k_begin, k_end);
                pa_dot2<ROUND>(w1, w1, xin + (n1 / a.grp_rows) * a.x_gs, a.K, 1.0f, lane, s1, t, k_begin, k_end);
            } else if (n0 >= a.N) {
                pa_dot2<false>(w0, w1, xin, a.K, 1.0f, lane, s0, s1, k_begin, k_end);
            } else if (n1 >= a.N) { // the pair straddles the two matrices
                float t;
                pa_dot2<ROUND>(w0, w0, xin, a.K, 1.0f, lane, s0, t, k_begin, k_end);
                pa_dot2<false>(w1, w1, xin, a.K, 1.0f, lane, s1, t, k_begin, k_end);
            } else {
                pa_dot2<ROUND>(w0, w1, xin, a.K, 1.0f, lane, s0, s1, k_begin, k_end);
            }
        }
        if (ks > 1) {
            if (lane == 0) { part_s[warp][0] = s0; part_s[warp][1] = s1; }
            __syncthreads();
            if (slice == 0) {
                s0 = s1 = 0.f;
                for (int q = 0; q < ks; q++) { s0 += part_s[q * pairs + pair][0]; s1 += part_s[q * pairs + pair][1]; }
            }
        }
        if (slice == 0 && live && lane < 2 && !(lane && n1 == n0)) {
            const int n = lane ? n1 : n0;
            float v = lane ? s1 : s0;
            if (n >= a.N) {
                a.z[n - a.N] = a.zbias ? v + a.zbias[n - a.N] : v;
            } else {
                if (a.bias) v += a.bias[n];
                if (n >= a.qd && n < a.qd + a.kd + a.vd) {
                    const int p = a.pos[0];
                    if (n < a.qd + a.kd) {
                        a.kc[(int64_t)p * a.kd + (n - a.qd)] = v;
                        if (a.v_is_k) a.vct[(int64_t)(n - a.qd) * a.n_ctx + p] = v;
                    } else {
                        a.vct[(int64_t)(n - a.qd - a.kd) * a.n_ctx + p] = v;
                    }
                } else if (a.act_from > 0 && n >= a.act_from) {
                    a.y[n + a.gap] = pa_act1(v, a.act);
                } else if (a.residual) {
                    a.residual[n] += v;
                } else if (a.grp_rows > 0) {
                    a.y[(n / a.grp_rows) * a.y_gs + n % a.grp_rows] = v;
                } else {
                    a.y[n] = v;
                }
            }
        }
        if (ks > 1) __syncthreads(); // part_s is written again by the next group
    }
}

// ---------------------------------------------------------------------------------------------------- per-layer token input
// eight rows at once (neighbours of stride K; K and the address multiples of eight): s[i] = w_i . f(x), reduced over the warp
template <bool ROUND> __device__ __forceinline__ void pa_dot8(const bf16 *__restrict__ w, const float *x, int K, int lane, float (&s)[8]) {
#pragma unroll
    for (int i = 0; i < 8; i++) s[i] = 0.f;
    for (int k = lane * 8; k < K; k += 256) {
        uint4 v[8];
#pragma unroll
        for (int i = 0; i < 8; i++) v[i] = __ldg(reinterpret_cast<const uint4 *>(w + (int64_t)i * K + k));
        const float4 x0 = *reinterpret_cast<const float4 *>(x + k), x1 = *reinterpret_cast<const float4 *>(x + k + 4);
        const float xv[8] = {pa_rnd<ROUND>(x0.x), pa_rnd<ROUND>(x0.y), pa_rnd<ROUND>(x0.z), pa_rnd<ROUND>(x0.w), pa_rnd<ROUND>(x1.x), pa_rnd<ROUND>(x1.y), pa_rnd<ROUND>(x1.z), pa_rnd<ROUND>(x1.w)};
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const uint32_t u[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
#pragma unroll
            for (int t = 0; t < 4; t++) {
                s[i] = fmaf(__uint_as_float(u[t] << 16), xv[2 * t], s[i]);
                s[i] = fmaf(__uint_as_float(u[t] & 0xffff0000u), xv[2 * t + 1], s[i]);
            }
        }
    }
#pragma unroll
    for (int o = 16; o; o >>= 1)
#pragma unroll
        for (int i = 0; i < 8; i++) s[i] += __shfl_xor_sync(0xffffffffu, s[i], o);
}

// x <- x + seam; y = W_proj (gelu(W_gate x) * e) in one launch of one cluster: each CTA forms its share of the gated vector and hands it to
// every other through distributed shared memory, then takes its share of the projection's rows.  y waits for the next seam.
#define PA_TI_THREADS 512
#define PA_TI_CLUSTER 16 // (beyond the portable size: asked for by attribute)
struct PaTokIn {
    const float *x, *seam_y, *seam_w;
    float *x_out;
    float eps, y_scale;
    const bf16 *Wg, *Wp; // [td][dim], [dim][td]
    int dim, td;
    PaRowMul e;
    float *y;
};
template <bool ROUND>
__global__ void __launch_bounds__(PA_TI_THREADS) pa_k_dec_token_input(const PaTokIn a) {
    extern __shared__ __align__(16) float pa_hs[]; // [dim] the stream, [td] the gated vector
    cg::cluster_group cl = cg::this_cluster();
    const int n_cl = gridDim.x, me = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, dim = a.dim, td = a.td;
    float *gs = pa_hs + ((dim + 3) & ~3);
    const int per_g = (td + n_cl - 1) / n_cl, g0 = min(me * per_g, td), g1 = min(g0 + per_g, td);
    const int per_p = ((dim + n_cl - 1) / n_cl + 7) & ~7, p0 = min(me * per_p, dim), p1 = min(p0 + per_p, dim);
    for (int64_t e = threadIdx.x * 64; e < (int64_t)(g1 - g0) * dim; e += PA_TI_THREADS * 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.Wg + (int64_t)g0 * dim + e));
    for (int64_t e = threadIdx.x * 64; e < (int64_t)(p1 - p0) * td; e += PA_TI_THREADS * 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.Wp + (int64_t)p0 * td + e));
    pa_prefetch_norms(a.seam_w, nullptr, dim);
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    cl.barrier_arrive(); // this CTA runs: its shared memory may be written
    const bf16 *erow = a.e.table + (int64_t)a.e.tok[0] * a.e.ld;
    if (warp == PA_TI_THREADS / 32 - 1)
        for (int n = g0 + lane * 32; n < g1; n += 32 * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(erow + n));
    pa_seam_to_smem<PA_TI_THREADS>(pa_hs, a.x, a.seam_y, a.seam_w, nullptr, a.x_out, dim, 1, a.eps, 0, nullptr, nullptr, a.y_scale);
    cl.barrier_wait();
    const PaAct gelu{0.f, 0.f, 0.f, PS_ACT_GELU_TANH};
    for (int n = g0 + 2 * warp; n < g1; n += 2 * (PA_TI_THREADS / 32)) {
        const int n1 = min(n + 1, g1 - 1);
        float s0, s1;
        const float e0 = pa_ld(erow + n), e1 = pa_ld(erow + n1);
        pa_dot2<ROUND>(a.Wg + (int64_t)n * dim, a.Wg + (int64_t)n1 * dim, pa_hs, dim, 1.0f, lane, s0, s1);
        if (lane < n_cl) { // a lane per CTA
            float *dst = cl.map_shared_rank(gs, lane);
            dst[n] = pa_act1(s0, gelu) * e0;
            dst[n1] = pa_act1(n1 == n ? s0 : s1, gelu) * e1;
        }
    }
    cl.sync();
    if ((td & 7) == 0) {
        for (int n = p0 + 8 * warp; n < p1; n += 8 * (PA_TI_THREADS / 32)) {
            if (n + 8 <= p1) {
                float s[8];
                pa_dot8<ROUND>(a.Wp + (int64_t)n * td, gs, td, lane, s);
#pragma unroll
                for (int i = 0; i < 8; i++)
                    if (lane == i) a.y[n + i] = s[i];
            } else {
                for (int m = n; m < p1; m++) {
                    float s0, s1;
                    pa_dot2<ROUND>(a.Wp + (int64_t)m * td, a.Wp + (int64_t)m * td, gs, td, 1.0f, lane, s0, s1);
                    if (lane == 0) a.y[m] = s0;
                }
            }
        }
    } else {
        for (int n = p0 + 2 * warp; n < p1; n += 2 * (PA_TI_THREADS / 32)) {
            const int n1 = min(n + 1, p1 - 1);
            float s0, s1;
            pa_dot2<ROUND>(a.Wp + (int64_t)n * td, a.Wp + (int64_t)n1 * td, gs, td, 1.0f, lane, s0, s1);
            if (lane == 0) a.y[n] = s0;
            if (lane == 1 && n1 != n) a.y[n1] = s1;
        }
    }
}

// ---------------------------------------------------------------------------------------------------- decode attention
// b[h][j] for the CTA's PA_DS_KEYS keys.  The keys' cache rows arrive in shared memory by 1-D bulk copies (one per row, the rows
// padded against bank conflicts) while the threads fetch q; then a thread per (key, head) forms the dot product with float4 reads
// and applies scale / temperature / distance bias - no shuffles, and the bias look-ups of all pairs are in flight together.
// CTAs from `tok_blocks` on take 16 pooled blocks each: the mean key rows behind the token rows, scores at pool_off, statistics at stat_off.
// With pool_v given, the last CTA also forms the means of the block that this token completes (no query sees that block before a
// later step, so nothing in this launch reads them).
__global__ void __launch_bounds__(256) pa_k_dec_scores(PaAttn at, const float *__restrict__ q, const float *kc, const int32_t *__restrict__ pos_dev,
                                                       float *__restrict__ b, int *__restrict__ err, int tok_blocks, float *pool_v) {
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(8) uint64_t bar;
    const int H = at.H, G = at.G, dq = at.dq, rep = H / G, kd = G * dq, kds = ((kd + 3) & ~3) + 4;
    float *ks = sm;                        // [PA_DS_KEYS][kds]
    float *qs = ks + PA_DS_KEYS * kds;     // [H][dq]
    float *sa = qs + H * dq;               // [H][PA_DS_KEYS + 1]
    float *Ts = sa + H * (PA_DS_KEYS + 1); // [H][H]
    const float2 *cs = at.rope.cs;
    const int tid = threadIdx.x;
    if (at.mix) for (int t = tid; t < H * H; t += 256) Ts[t] = at.mix[t]; // a weight: fetched before the dependency wait
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    const int pos = pos_dev[0];
    if (pool_v && at.pool > 0 && blockIdx.x == gridDim.x - 1 && (pos + 1) % at.pool == 0 && pos + 1 <= at.n_ctx)
        for (int c = tid; c < kd + G * at.dv; c += 256) pa_pool_block(const_cast<float *>(kc), pool_v, kd, G * at.dv, at.n_ctx, at.pool, at.n_pool, (pos + 1) / at.pool - 1, c);
    const bool pooled = (int)blockIdx.x >= tok_blocks;
    int lo = pa_first_key(at, pos);
    int blk = lo / PA_DS_KEYS + blockIdx.x, j0 = blk * PA_DS_KEYS; // the grid starts at the block of the first key in sight
    int nj = min(PA_DS_KEYS, pos + 1 - j0), s_off = 0;
    if (pooled) { // rows n_ctx + j0 .. of the K buffer; every one of the first pa_pool_vis blocks is in sight
        lo = 0;
        j0 = ((int)blockIdx.x - tok_blocks) * PA_DS_KEYS;
        nj = min(PA_DS_KEYS, pa_pool_vis(at, pos) - j0);
        blk = at.stat_off + (int)blockIdx.x - tok_blocks;
        s_off = at.pool_off;
        kc += (int64_t)at.n_ctx * kd;
    }
    if (nj <= 0) return;
    const bool bulk = (kd & 3) == 0;
    const bool own = at.k_raw && !pooled && j0 + nj == pos + 1; // the token's own key: raw in k_raw, not in the cache yet
    const int nc = own ? nj - 1 : nj;                           // rows that come from the cache
    if (bulk && tid == 0) {
        ps_mbar_init(&bar, 1);
        ps_fence_barrier_init();
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        ps_mbar_expect_tx(&bar, (uint32_t)(nc * kd * 4));
        for (int jj = 0; jj < nc; jj++) ps_bulk_g2s(ks + jj * kds, kc + (int64_t)(j0 + jj) * kd, (uint32_t)(kd * 4), &bar);
    }
    if (!bulk) for (int t = tid; t < nc * kd; t += 256) ks[(t / kd) * kds + t % kd] = kc[(int64_t)j0 * kd + t];
    if (at.k_raw) { // a warp per head: norm of q (times the position's temperature), and of the token's key on its way into the cache
        const int lane = tid & 31;
        const float qt = pa_q_temp(at.qt_coef, at.qt_every, pos);
        const int rh = at.rope.dims >> 1, vh = at.vrope.dims >> 1;
        if (own && vh > 0) // the token's value, rotated, into its V^T column
            for (int e = tid; e < G * vh; e += 256) {
                const int g = e / vh, m = e % vh;
                const float va = at.v_raw[g * at.dv + m], vb = at.v_raw[g * at.dv + m + vh];
                const float2 t = at.vrope.cs[m];
                at.vct_out[(int64_t)(g * at.dv + m) * at.n_ctx + pos] = va * t.x - vb * t.y;
                at.vct_out[(int64_t)(g * at.dv + m + vh) * at.n_ctx + pos] = vb * t.x + va * t.y;
            }
        for (int hh = tid >> 5; hh < H + (own ? G : 0); hh += 8) {
            const bool is_q = hh < H;
            const float *src = is_q ? q + hh * dq : at.k_raw + (hh - H) * dq, *w = is_q ? at.qn : at.kn;
            float *dst = is_q ? qs + hh * dq : ks + nc * kds + (hh - H) * dq;
            float s = 0.f;
#pragma unroll 4
            for (int c = lane; c < dq; c += 32) {
                const float v = src[c];
                dst[c] = w ? v * w[c] : v;
                s = fmaf(v, v, s);
            }
#pragma unroll
            for (int o = 16; o; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
            const float inv = (at.head_norm ? 1.0f / sqrtf(s / (float)dq + at.eps) : 1.0f) * (is_q ? qt : 1.0f);
            float *kout = is_q ? nullptr : at.kc_out + (int64_t)pos * kd + (hh - H) * dq;
            if (rh > 0) {
                __syncwarp();
                for (int i = lane; i < rh; i += 32) {
                    const float2 c2 = cs[i];
                    const float va = dst[i] * inv, vb = dst[i + rh] * inv, ra = va * c2.x - vb * c2.y, rb = vb * c2.x + va * c2.y;
                    dst[i] = ra;
                    dst[i + rh] = rb;
                    if (kout) { kout[i] = ra; kout[i + rh] = rb; }
                }
            }
            for (int c = 2 * rh + lane; c < dq; c += 32) { // (without a rotation: a lane's own entries)
                const float v = dst[c] * inv;
                dst[c] = v;
                if (kout) kout[c] = v;
            }
        }
    } else {
        for (int t = tid; t < H * dq; t += 256) qs[t] = q[t];
    }
    __syncthreads();
    if (bulk && !ps_tc_wait(&bar, 0)) { if (tid == 0) err[0] = 5; return; }
    for (int t = tid; t < PA_DS_KEYS * H; t += 256) {
        const int jj = t % PA_DS_KEYS, h = t / PA_DS_KEYS;
        if (jj >= nj || j0 + jj < lo) continue;
        const float *kr = ks + jj * kds + (h / rep) * dq, *qr = qs + h * dq;
        float s;
        if ((dq & 3) == 0) {
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int d = 0; d < dq; d += 4) {
                const float4 k4 = *reinterpret_cast<const float4 *>(kr + d), q4 = *reinterpret_cast<const float4 *>(qr + d);
                acc.x = fmaf(k4.x, q4.x, acc.x); acc.y = fmaf(k4.y, q4.y, acc.y); acc.z = fmaf(k4.z, q4.z, acc.z); acc.w = fmaf(k4.w, q4.w, acc.w);
            }
            s = (acc.x + acc.y) + (acc.z + acc.w);
        } else {
            s = 0.f;
            for (int d = 0; d < dq; d++) s = fmaf(kr[d], qr[d], s);
        }
        sa[h * (PA_DS_KEYS + 1) + jj] = pa_score(at, s, h, pooled ? 0 : pos - (j0 + jj));
    }
    __syncthreads();
    // mix the heads, store, and leave the block's soft-max statistics (max, sum of exponentials) for the P.V kernel:
    // the 16 keys of a head sit in 16 adjacent lanes
    const int n_t = (PA_DS_KEYS * H + 31) & ~31;
    for (int t = tid; t < n_t; t += 256) {
        const int h = t / PA_DS_KEYS, jj = t % PA_DS_KEYS;
        const bool valid = h < H && jj < nj && j0 + jj >= lo;
        float s = -INFINITY;
        if (valid) {
            if (at.mix) {
                s = 0.f;
                for (int g = 0; g < H; g++) s = fmaf(Ts[h * H + g], sa[g * (PA_DS_KEYS + 1) + jj], s);
            } else {
                s = sa[h * (PA_DS_KEYS + 1) + jj];
            }
            b[(int64_t)h * at.ldS + s_off + j0 + jj] = s;
        }
        float m = s;
#pragma unroll
        for (int o = PA_DS_KEYS / 2; o; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        float e = valid ? expf(s - m) : 0.f;
#pragma unroll
        for (int o = PA_DS_KEYS / 2; o; o >>= 1) e += __shfl_xor_sync(0xffffffffu, e, o);
        if (h < H && jj == 0) { // (every lane of the 16 holds the block's pair; the block has a key in sight)
            at.pm[(int64_t)h * at.ldP + blk] = m;
            at.pl[(int64_t)h * at.ldP + blk] = e;
        }
    }
}

// att[h][c] = sum_j p_hj V^T[g(h) dv + c][j] for one kv head g and PA_DP_DIMS value dims; p = soft-max of b[h][0 .. pos] with the
// optional sink term.  Phase 1: max and sum of every query head of the group, merged from the per-block pairs the scores kernel
// left (16 keys each).  Phase 2, per chunk of keys: the CTA's V^T rows
// arrive by 1-D bulk copies while the threads compute the chunk's weights once into shared memory; two warps per value dim
// (the halves of the chunk) then run float4 dot products out of shared memory for every head of the group.
__global__ void __launch_bounds__(256) pa_k_dec_pv(PaAttn at, const float *__restrict__ b, const float *__restrict__ vct, const int32_t *__restrict__ pos_dev,
                                                   float *__restrict__ att, int chunk, int *__restrict__ err) {
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(8) uint64_t bar;
    // blockIdx.z splits the query heads that share kv head g (many heads over one latent): this CTA takes `rep` of them from h0 on
    const int H = at.H, G = at.G, dv = at.dv, rep_all = H / G, g = blockIdx.y;
    const int rep_z = (rep_all + (int)gridDim.z - 1) / (int)gridDim.z, h0 = g * rep_all + (int)blockIdx.z * rep_z, rep = min(rep_z, rep_all - (int)blockIdx.z * rep_z);
    if (rep <= 0) return;
    float *vs = sm;                         // [PA_DP_DIMS][chunk] V^T rows of the chunk
    float *ps = vs + PA_DP_DIMS * chunk;    // [rep][chunk] soft-max weights of the chunk (un-normalised)
    float *ms = ps + rep * chunk;           // [rep] row maxima
    float *inv = ms + rep;                  // [rep] 1 / denominators
    float *acc = inv + rep;                 // [8 warps][rep]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    const int n = pos_dev[0] + 1, lo = pa_first_key(at, n - 1);
    const bool bulk = (at.n_ctx & 3) == 0;
    if (bulk && tid == 0) {
        ps_mbar_init(&bar, 1);
        ps_fence_barrier_init();
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    const int c0 = blockIdx.x * PA_DP_DIMS;
    // value dim of the CTA's cc-th row (dv or more: outside); with rotated values the CTA takes two pairs (m, m + dv / 2)
    const int vh = at.vrope.dims >> 1;
    auto col = [&](int cc) {
        if (vh == 0) return c0 + cc;
        const int m = c0 / 2 + (cc & 1);
        return m < vh ? m + (cc >= 2 ? vh : 0) : dv;
    };
    // a chunk's V^T rows: 1-D bulk copies, issued by one thread (the first chunk's travel while the statistics are merged)
    auto copy_rows = [&](const float *vbase, int ldv, int j0, int nj4) {
        int rows = 0;
        for (int cc = 0; cc < PA_DP_DIMS; cc++) rows += col(cc) < dv;
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); // the rows were read through the generic proxy
        ps_mbar_expect_tx(&bar, (uint32_t)(rows * nj4 * 4));
        for (int cc = 0; cc < PA_DP_DIMS; cc++)
            if (col(cc) < dv) ps_bulk_g2s(vs + cc * chunk, vbase + (int64_t)(g * dv + col(cc)) * ldv + j0, (uint32_t)(nj4 * 4), &bar);
    };
    if (bulk && tid == 0) copy_rows(vct, at.n_ctx, lo & ~3, (min(chunk, n - (lo & ~3)) + 3) & ~3);
    // soft-max statistics of every head of the group from the scores kernel's per-block pairs: a warp per head
    const int nb = (n + PA_DS_KEYS - 1) / PA_DS_KEYS;
    const int nv = pa_pool_vis(at, n - 1), nvb = (nv + PA_DS_KEYS - 1) / PA_DS_KEYS; // pooled blocks in sight, and their statistics
    for (int r = warp; r < rep; r += 8) {
        const float *bm = at.pm + (int64_t)(h0 + r) * at.ldP, *bl = at.pl + (int64_t)(h0 + r) * at.ldP;
        const float sk = pa_sink_logit(at, h0 + r);
        float mx = at.sink ? sk : -INFINITY;
        for (int j = lo / PA_DS_KEYS + lane; j < nb; j += 32) mx = fmaxf(mx, bm[j]);
        for (int j = lane; j < nvb; j += 32) mx = fmaxf(mx, bm[at.stat_off + j]);
#pragma unroll
        for (int o = 16; o; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        float sum = 0.f;
        for (int j = lo / PA_DS_KEYS + lane; j < nb; j += 32) sum = fmaf(bl[j], expf(bm[j] - mx), sum);
        for (int j = lane; j < nvb; j += 32) sum = fmaf(bl[at.stat_off + j], expf(bm[at.stat_off + j] - mx), sum);
#pragma unroll
        for (int o = 16; o; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if (lane == 0) {
            if (at.sink) sum += expf(sk - mx);
            ms[r] = mx;
            inv[r] = 1.0f / sum;
        }
    }
    for (int t = tid; t < 8 * rep; t += 256) acc[t] = 0.f;
    const int dim_l = warp % PA_DP_DIMS, part = warp / PA_DP_DIMS, n_part = 8 / PA_DP_DIMS;
    int it = 0;
    // two stretches of keys: the tokens in sight (V^T rows of n_ctx columns), then the pooled blocks (rows of n_pool columns behind them)
    for (int seg = 0; seg < (nv > 0 ? 2 : 1); seg++) {
    const float *vbase = seg ? vct + (int64_t)G * dv * at.n_ctx : vct;
    const int ldv = seg ? at.n_pool : at.n_ctx, s_lo = seg ? 0 : lo, s_n = seg ? nv : n, s_off = seg ? at.pool_off : 0;
    for (int j0 = s_lo & ~3; j0 < s_n; j0 += chunk, it++) { // (bulk copies start on 16-byte boundaries)
        const int nj = min(chunk, s_n - j0), nj4 = (nj + 3) & ~3;
        __syncthreads(); // the previous chunk's buffers are free
        if (bulk) {
            if (tid == 0 && it > 0) copy_rows(vbase, ldv, j0, nj4);
        } else {
            for (int t = tid; t < PA_DP_DIMS * nj4; t += 256) {
                const int cc = t / nj4, jj = t % nj4;
                vs[cc * chunk + jj] = (col(cc) < dv && jj < nj) ? vbase[(int64_t)(g * dv + col(cc)) * ldv + j0 + jj] : 0.f;
            }
        }
        for (int r = 0; r < rep; r++) {
            const float *br = b + (int64_t)(h0 + r) * at.ldS + s_off + j0;
            const float m = ms[r];
            for (int jb = tid; jb < nj4; jb += 4 * 256) { // four scores in flight per thread
                float v[4];
#pragma unroll
                for (int u = 0; u < 4; u++) v[u] = br[min(jb + 256 * u, nj - 1)];
#pragma unroll
                for (int u = 0; u < 4; u++) {
                    const int jj = jb + 256 * u;
                    if (jj < nj4) ps[r * chunk + jj] = (jj < nj && j0 + jj >= s_lo) ? expf(v[u] - m) : 0.f;
                }
            }
        }
        __syncthreads();
        if (bulk && !ps_tc_wait(&bar, it & 1)) { if (tid == 0) err[0] = 6; return; }
        if (col(dim_l) < dv) {
            const float4 *v4 = reinterpret_cast<const float4 *>(vs + dim_l * chunk);
            for (int r = 0; r < rep; r++) {
                const float4 *p4 = reinterpret_cast<const float4 *>(ps + r * chunk);
                float s = 0.f;
                for (int i = lane + 32 * part; i < nj4 / 4; i += 32 * n_part) {
                    const float4 v = v4[i], p = p4[i];
                    s = fmaf(p.x, v.x, s); s = fmaf(p.y, v.y, s); s = fmaf(p.z, v.z, s); s = fmaf(p.w, v.w, s);
                }
#pragma unroll
                for (int o = 16; o; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
                if (lane == 0) acc[warp * rep + r] += s;
            }
        }
    }
    }
    __syncthreads();
    for (int t = tid; t < PA_DP_DIMS * rep; t += 256) {
        const int cc = t / rep, r = t % rep, c = col(cc);
        if (c >= dv) continue;
        auto sum = [&](int k) {
            float s = 0.f;
            for (int pp = 0; pp < n_part; pp++) s += acc[(pp * PA_DP_DIMS + k) * rep + r];
            return s * inv[r];
        };
        float s = sum(cc);
        if (vh > 0) { // turned back by the query's position
            const float2 t2 = at.vrope.cs[c0 / 2 + (cc & 1)];
            const float o = sum(cc ^ 2);
            s = cc < 2 ? s * t2.x + o * t2.y : s * t2.x - o * t2.y;
        }
        if (at.gate) s *= pa_sigmoid(at.gate[h0 + r]);
        att[(h0 + r) * dv + c] = at.out_scale != 0.f ? s * at.out_scale : s;
    }
}

// ---------------------------------------------------------------------------------------------------- latent attention
// What lies between the first projection of a latent attention whose queries come straight from the input and its scores, in one
// launch.  row = [q: H heads of dn + dr | kv latent (rk) | rotated key part (dr)].
//   CTAs below gridDim.x - 1: W_uk folded into the query, qa[h][c] = sum_d wukt[h][c][d] round(q_h[d]); 2^lg lanes share an output row
//     (a lane takes eight columns at a time), so short rows keep every lane busy
//   the last CTA: the normed latent and the rotated key part into the cache, the rotated query parts into qa
template <bool ROUND>
__global__ void __launch_bounds__(256) pa_k_dec_latent_q(const float *__restrict__ row, int H, int dn, int dr, int rk, const bf16 *__restrict__ wukt, float *__restrict__ qa, int lg,
                                                         const float *__restrict__ wk, float eps, PaRope rope, float *__restrict__ kc, float *__restrict__ vct, int n_ctx,
                                                         const int32_t *__restrict__ pos) {
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, lqw = H * (dn + dr);
    if (blockIdx.x + 1 == gridDim.x) {
        __shared__ float red[8];
        ps_grid_dep_launch();
        ps_grid_dep_wait();
        const int p = pos[0];
        const float *c = row + lqw;
        float s = 0.f;
        for (int i = tid; i < rk; i += 256) s = fmaf(c[i], c[i], s);
        const float inv = 1.0f / sqrtf(pa_block_sum(s, red) / (float)rk + eps);
        float *krow = kc + (int64_t)p * (rk + dr);
        for (int i = tid; i < rk; i += 256) {
            const float v = c[i] * inv * wk[i];
            krow[i] = v;
            vct[(int64_t)i * n_ctx + p] = v;
        }
        for (int i = tid; i < dr; i += 256) pa_rope_store(rope, c + rk, krow + rk, dr, p, i);
        for (int e = tid; e < H * dr; e += 256) pa_rope_store(rope, row + (e / dr) * (dn + dr) + dn, qa + (e / dr) * (rk + dr) + rk, dr, p, e % dr);
        return;
    }
    const int lpr = 1 << lg, sub = lane & (lpr - 1), per_warp = 32 >> lg, rows = H * rk;
    const int stride = ((int)gridDim.x - 1) * 8 * per_warp;
    int n = (blockIdx.x * 8 + warp) * per_warp + (lane >> lg);
    if (n < rows && sub * 64 < dn) asm volatile("prefetch.global.L2 [%0];" ::"l"(wukt + (int64_t)n * dn + sub * 64));
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    for (; __any_sync(0xffffffffu, n < rows); n += stride) {
        const int nn = min(n, rows - 1), h = nn / rk;
        const bf16 *w = wukt + (int64_t)nn * dn;
        const float *x = row + h * (dn + dr);
        float s = 0.f;
        if ((dn & 7) == 0 && ((dn + dr) & 3) == 0) {
            for (int k = sub * 8; k < dn; k += lpr * 8) {
                const uint4 a = __ldg(reinterpret_cast<const uint4 *>(w + k));
                const float4 x0 = *reinterpret_cast<const float4 *>(x + k), x1 = *reinterpret_cast<const float4 *>(x + k + 4);
                const float xv[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
                const uint32_t au[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
                for (int t = 0; t < 4; t++) {
                    s = fmaf(__uint_as_float(au[t] << 16), pa_rnd<ROUND>(xv[2 * t]), s);
                    s = fmaf(__uint_as_float(au[t] & 0xffff0000u), pa_rnd<ROUND>(xv[2 * t + 1]), s);
                }
            }
        } else {
            for (int k = sub; k < dn; k += lpr) s = fmaf(__bfloat162float(w[k]), pa_rnd<ROUND>(x[k]), s);
        }
        for (int o = lpr >> 1; o; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if (sub == 0 && n < rows) qa[h * (rk + dr) + nn % rk] = s;
    }
}

// ---------------------------------------------------------------------------------------------------- routed experts
// grid (row pairs of ff, top_k): y[r][n] = act(gate_e . z, up_e . z), z = round(w_r * h) (score on the input) or round(h)
template <bool ROUND>
__global__ void __launch_bounds__(PA_DV_THREADS) pa_k_dec_expert_up(const float *__restrict__ x, const float *__restrict__ norm_w, float eps, const float *__restrict__ z, PaRoute rt,
                                                                    const bf16 *__restrict__ Wg, const bf16 *__restrict__ Wu, float *__restrict__ y,
                                                                    int ff, int dim, int on_input, PaAct act, int *__restrict__ sel_e,
                                                                    float *__restrict__ sel_w, float *__restrict__ h_out = nullptr) {
    extern __shared__ __align__(16) float pa_hs[];
    __shared__ float sc[PA_MAX_EXPERTS];
    __shared__ int se[PA_MAX_EXPERTS];
    __shared__ float sw[PA_MAX_EXPERTS];
    pa_prefetch_norms(norm_w, nullptr, norm_w ? dim : 0);
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    auto route = [&]() { // (the prologue's barriers publish se / sw)
        if (rt.act == PS_ROUTER_TOPK_SOFTMAX || (rt.act == PS_ROUTER_SOFTMAX && rt.groups <= 1)) {
            if (threadIdx.x < 32) {
                if (rt.act == PS_ROUTER_SOFTMAX) pa_route_softmax_warp(z, rt, se, sw, threadIdx.x);
                else pa_route_topk_warp(z, rt.E, rt.top, se, sw, threadIdx.x);
                __syncwarp();
                if (blockIdx.x == 0 && blockIdx.y == 0)
                    for (int r = threadIdx.x; r < rt.top; r += 32) { sel_e[r] = se[r]; sel_w[r] = sw[r]; }
            }
        } else if (threadIdx.x == 0) {
            pa_route_serial(z, rt, sc, se, sw);
            if (blockIdx.x == 0 && blockIdx.y == 0)
                for (int r = 0; r < rt.top; r++) { sel_e[r] = se[r]; sel_w[r] = sw[r]; }
        }
    };
    // the input, normed (norm_w null: as it is, the experts read the residual stream itself)
    pa_seam_to_smem(pa_hs, x, nullptr, nullptr, norm_w, nullptr, dim, 1, eps, 0, nullptr, nullptr, 1.0f, route);
    const int r = blockIdx.y, e = se[r], lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (h_out && blockIdx.x == 0 && blockIdx.y == 0) // the normed input, for the choices that stand for it
        for (int c = threadIdx.x; c < dim; c += blockDim.x) h_out[c] = pa_hs[c];
    if (e >= rt.E - rt.identity) return;
    const float w = on_input ? sw[r] : 1.0f;
    // a warp owns one ff row at a time: its gate row and its up row are the pair; the CTAs walk the row groups with the grid's stride
    const int rows = PA_DV_ROWS / 2;
    if (!Wg) { // no gate: the pair is two neighbouring up rows
        for (int n0 = (blockIdx.x * rows + warp) * 2; n0 < ff; n0 += gridDim.x * rows * 2) {
            const int n1 = min(n0 + 1, ff - 1);
            float s0, s1;
            pa_dot2<ROUND>(Wu + ((int64_t)e * ff + n0) * dim, Wu + ((int64_t)e * ff + n1) * dim, pa_hs, dim, w, lane, s0, s1);
            if (lane == 0) y[(int64_t)r * ff + n0] = pa_act1(s0, act);
            if (lane == 1 && n1 != n0) y[(int64_t)r * ff + n1] = pa_act1(s1, act);
        }
        return;
    }
    for (int n = blockIdx.x * rows + warp; n < ff; n += gridDim.x * rows) {
        const bf16 *wg = Wg + ((int64_t)e * ff + n) * dim, *wu = Wu + ((int64_t)e * ff + n) * dim;
        float gsum, usum;
        pa_dot2<ROUND>(wg, wu, pa_hs, dim, w, lane, gsum, usum);
        if (lane == 0) y[(int64_t)r * ff + n] = pa_expert_act(gsum, usum, act);
    }
}

// dense gated feed-forward of a sequential block, first half: the seam in the prologue (the mixer's output joins the residual
// stream, the result is normed), then y[n] = act(gate[n] . h, up[n] . h); a warp owns one ff row at a time, the CTAs walk the row
// groups with the grid's stride
template <bool ROUND>
__global__ void __launch_bounds__(PA_DV_THREADS) pa_k_dec_dense_up(const float *__restrict__ x, const float *__restrict__ seam_y, const float *__restrict__ seam_w,
                                                                   const float *__restrict__ norm_w, float *__restrict__ x_out, int groups, float eps, const bf16 *__restrict__ Wg,
                                                                   const bf16 *__restrict__ Wu, float *__restrict__ y, int ff, int dim, PaAct act,
                                                                   const bf16 *__restrict__ Wr = nullptr, int E = 0, float *__restrict__ z = nullptr, int center = 0, float y_scale = 1.0f) {
    extern __shared__ __align__(16) float pa_hs[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, rows = PA_DV_ROWS / 2;
    if (!Wg) { // no gate: a warp's pair is two neighbouring up rows, y[n] = act(up[n] . h)
        const int n = (blockIdx.x * rows + warp) * 2;
        if (n < ff) pa_prefetch2(Wu + (int64_t)n * dim, Wu + (int64_t)min(n + 1, ff - 1) * dim, 0, dim, lane);
        pa_prefetch_norms(seam_w, norm_w, dim);
        ps_grid_dep_launch();
        ps_grid_dep_wait();
        pa_seam_to_smem(pa_hs, x, seam_y, seam_w, norm_w, x_out, dim, groups, eps, center, nullptr, nullptr, y_scale);
        for (int n0 = (blockIdx.x * rows + warp) * 2; n0 < ff; n0 += gridDim.x * rows * 2) {
            const int n1 = min(n0 + 1, ff - 1);
            float s0, s1;
            pa_dot2<ROUND>(Wu + (int64_t)n0 * dim, Wu + (int64_t)n1 * dim, pa_hs, dim, 1.0f, lane, s0, s1);
            if (lane == 0) y[n0] = pa_act1(s0, act);
            if (lane == 1 && n1 != n0) y[n1] = pa_act1(s1, act);
        }
        return;
    }
    {
        const int n = blockIdx.x * rows + warp;
        if (n < ff) pa_prefetch2(Wg + (int64_t)n * dim, Wu + (int64_t)n * dim, 0, dim, lane);
        pa_prefetch_norms(seam_w, norm_w, dim);
    }
    ps_grid_dep_launch();
    ps_grid_dep_wait();
    pa_seam_to_smem(pa_hs, x, seam_y, seam_w, norm_w, x_out, dim, groups, eps, center, nullptr, nullptr, y_scale);
    // E more rows behind the ff rows: a router's logits z[e] = Wr[e] . h from the UNROUNDED input (a shared expert's launch carries them)
    for (int n = blockIdx.x * rows + warp; n < ff + E; n += gridDim.x * rows) {
        float gsum, usum;
        if (n >= ff) {
            const bf16 *wr = Wr + (int64_t)(n - ff) * dim;
            pa_dot2<false>(wr, wr, pa_hs, dim, 1.0f, lane, gsum, usum);
            if (lane == 0) z[n - ff] = gsum;
            continue;
        }
        pa_dot2<ROUND>(Wg + (int64_t)n * dim, Wu + (int64_t)n * dim, pa_hs, dim, 1.0f, lane, gsum, usum);
        if (lane == 0) y[n] = pa_expert_act(gsum, usum, act);
    }
}

// x[n] += ao[n] + sum_r down_{e_r}[n] . round(y_r)  (times w_r when the score weighs the output); slots in order; `ksplit`
// warps share a row pair, each taking ff / ksplit of the columns
template <bool ROUND>
__global__ void __launch_bounds__(PA_DV_THREADS) pa_k_dec_expert_down(const float *__restrict__ y, const int *__restrict__ sel_e, const float *__restrict__ sel_w, int top,
                                                                      const bf16 *__restrict__ Wd, const float *__restrict__ ao, float *__restrict__ x, int dim, int ff,
                                                                      int on_input, int ksplit, float *__restrict__ dst = nullptr, const float *__restrict__ extra = nullptr,
                                                                      const float *__restrict__ extra_logit = nullptr, int E = 1 << 30, const float *__restrict__ h = nullptr,
                                                                      const bf16 *__restrict__ Wsd = nullptr, const float *__restrict__ ysh = nullptr, int sff = 0) {
    __shared__ float part_s[8][2];
    ps_grid_dep_launch(); // the next kernel (the next layer's q|k|v rows, or the head) may start fetching its weights
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int pairs = 8 / ksplit, pair = warp % pairs, slice = warp / pairs;
    const int n0 = (blockIdx.x * pairs + pair) * 2, n1 = min(n0 + 1, dim - 1);
    const int kc = ff / ksplit, k_begin = slice * kc, k_end = slice == ksplit - 1 ? ff : k_begin + kc;
    const bool live = n0 < dim;
    float t0 = 0.f, t1 = 0.f;
    const int kcs = (sff / ksplit) & ~7, s_begin = slice * kcs, s_end = slice == ksplit - 1 ? sff : s_begin + kcs; // the shared expert's columns
    if (live && Wsd) pa_prefetch2(Wsd + (int64_t)n0 * sff, Wsd + (int64_t)n1 * sff, s_begin, s_end, lane);
    ps_grid_dep_wait();
    if (live) {
        for (int r = 0; r < top; r++) {
            const int e = sel_e[r];
            if (e >= E) continue;
            pa_prefetch2(Wd + ((int64_t)e * dim + n0) * ff, Wd + ((int64_t)e * dim + n1) * ff, k_begin, k_end, lane);
        }
        for (int r = 0; r < top; r++) {
            const int e = sel_e[r];
            if (e >= E) { // the input itself (one of the warps that share the rows adds it)
                if (slice == 0) { t0 = fmaf(sel_w[r], h[n0], t0); t1 = fmaf(sel_w[r], h[n1], t1); }
                continue;
            }
            float s0, s1;
            pa_dot2<ROUND>(Wd + ((int64_t)e * dim + n0) * ff, Wd + ((int64_t)e * dim + n1) * ff, y + (int64_t)r * ff, ff, 1.0f, lane, s0, s1, k_begin, k_end);
            const float w = on_input ? 1.0f : sel_w[r];
            t0 += s0 * w;
            t1 += s1 * w;
        }
        if (Wsd) { // the shared expert's down rows, times its gate
            float s0, s1;
            pa_dot2<ROUND>(Wsd + (int64_t)n0 * sff, Wsd + (int64_t)n1 * sff, ysh, sff, 1.0f, lane, s0, s1, s_begin, s_end);
            const float sg = extra_logit ? 1.0f / (1.0f + expf(-extra_logit[0])) : 1.0f;
            t0 = fmaf(sg, s0, t0);
            t1 = fmaf(sg, s1, t1);
        }
    }
    if (ksplit > 1) {
        if (lane == 0) { part_s[warp][0] = t0; part_s[warp][1] = t1; }
        __syncthreads();
        if (slice != 0) return;
        t0 = t1 = 0.f;
        for (int q = 0; q < ksplit; q++) { t0 += part_s[q * pairs + pair][0]; t1 += part_s[q * pairs + pair][1]; }
    }
    if (!live) return;
    if (dst) { // sequential blocks: the feed-forward's output waits for the next seam; a shared expert's output joins it here
        const float sg = extra ? (extra_logit ? 1.0f / (1.0f + expf(-extra_logit[0])) : 1.0f) : 0.f;
        if (lane == 0) dst[n0] = t0 + (extra ? sg * extra[n0] : 0.f);
        if (lane == 1 && n1 != n0) dst[n1] = t1 + (extra ? sg * extra[n1] : 0.f);
        return;
    }
    if (lane == 0) x[n0] += ao[n0] + t0;
    if (lane == 1 && n1 != n0) x[n1] += ao[n1] + t1;
}
