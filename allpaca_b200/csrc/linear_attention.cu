// Linear attention in its recurrent form: per head a state S of [D, V] 32-bit numbers that a request
// carries from step to step, written by outer products of keys and values and read by queries:
//
//   S_t = diag(a_t) S_{t-1} + k_t u_t^T        o_t = S_t^T q_t * out_scale
//
// with the variants as parameters of one kernel:
//   decay a_t   one fixed number per head (DECAY_HEAD_CONST: retention);
//               one number per head and token, exp(-exp(A_log[h]) * softplus(raw + dt_bias[h])) (DECAY_HEAD_TOKEN);
//               one number per key channel and token, sigmoid(z)^(1/tau) = exp(-softplus(-z) / tau) (DECAY_CHANNEL),
//               or exp(-exp(A_log[h]) * softplus(z + dt_bias[h, channel])) (DECAY_CHANNEL_TOKEN);
//               or one number per head and token that another kernel has worked out (DECAY_HEAD_READY)
//   write u_t   the value v_t, or b_t v_t with a number per head and token that another kernel has worked out; or, with
//               the delta rule, beta_t (v_t - S^T k_t) with S already decayed and beta_t = sigmoid(raw), so that the
//               read-out sees the corrected state
//   unit column the values may have one more column that is always 1: the state's last column then is the sum of
//               the keys themselves under the same decays and gates, and its read-out their product with the query
//   q, k        as projected (QK_PLAIN); the first rot_dims coordinates of every head turned by the step's
//               cosine/sine table, coordinate i with i + rot_dims/2 (QK_ROTATE); or made unit vectors,
//               x / sqrt(sum x^2 + unit_eps) (QK_UNIT); or, like the values, under SiLU (QKV_SILU).  Several value
//               heads may share a query/key head.
//
// and the kernel that finishes a head's read-out: RMS over the head, or over all heads together (a weight per
// coordinate or none), times silu(gate) or sigmoid(gate), times a constant, rounded to the activation type for the
// output projection.
//
// A step of single rows (decoding) runs the recurrence as written (la_scan_kernel); a step of portions runs it eight
// tokens at a time (la_blocks_kernel, la_chunk_kernel).
//
// Everything is 32-bit: inputs are 32-bit sums of the projections, decays, exponentials, the state, the
// read-out and the norm.  A sequence's rows are found through seq_start, its state row through
// state_slots; a portion whose first row has position 0 starts from zeros.  Nothing is decided on the
// host, so a step of these kernels can be replayed from a CUDA graph.
#include "common.cuh"

#define LA_PER_MAX 16            // state entries per thread at most
#define LA_CHUNK 16              // tokens staged at a time
#define DECAY_HEAD_CONST 0
#define DECAY_HEAD_TOKEN 1
#define DECAY_CHANNEL 2
#define DECAY_CHANNEL_TOKEN 3
#define DECAY_HEAD_READY 4
#define QK_PLAIN 0
#define QK_ROTATE 1
#define QK_UNIT 2
#define QKV_SILU 3

// whether every key channel has a decay of its own
__host__ __device__ constexpr bool la_per_channel(int mode) { return mode == DECAY_CHANNEL || mode == DECAY_CHANNEL_TOKEN; }

__device__ __forceinline__ float la_softplus(float v) { return v > 20.0f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float la_silu(float v) { return v / (1.0f + expf(-v)); }

__device__ __forceinline__ void la_copy4(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void la_copy16(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
struct LaScanArgs {
    float* q; long long ld_q;                  // head g of row t: q[t * ld_q + g * D + d]; made ready in place
    float* k; long long ld_k;
    float* v; long long ld_v;                  // head h of row t: v[t * ld_v + h * V + c]; QKV_SILU: in place
    float* decay_channel; long long ld_dc;     // DECAY_CHANNEL*: z[t * ld_dc + h * D + d], becomes the decay in place
    float* decay_head; long long ld_dh;        // DECAY_HEAD_TOKEN: raw[t * ld_dh + h], becomes the decay in place; DECAY_HEAD_READY: it
    const float* decay_const;                  // DECAY_HEAD_CONST: the decay [heads]; DECAY_*_TOKEN: A_log [heads]
    const float* dt_bias;                      // DECAY_HEAD_TOKEN: [heads], DECAY_CHANNEL_TOKEN: [heads * D]; or null
    float* beta; long long ld_beta;            // the write's gate [t * ld_beta + h], or null: it is 1
    int delta;                                 // the delta rule (its gate comes raw and becomes sigmoid in place)
    const float* cos_sin; int rot_dims;        // QK_ROTATE: [T, rot_dims / 2, 2]
    float* state; long long state_stride;      // [slots][heads][D][V]
    const int* seq_start; const int* positions; const int* state_slots;
    float* y; long long ld_y;                  // y[t * ld_y + h * V + c]
    int T, heads, qk_heads, D, V, NP, cols, decay_mode, qk_mode, vec;
    int VI;                                    // columns of v: V, or V - 1 where the last one is always 1
    float inv_tau, unit_eps, out_scale;
};

// What has to happen to a step's rows before the recurrence reads them, once per row and in place (the
// recurrence's CTAs share a head's queries and keys, so none of this belongs into them): one warp per
// (row, unit) with the units of a row being its query heads, its key heads (rotation, unit vectors or SiLU), its
// value heads (SiLU), its heads' channel decays and one unit for the numbers per head (decay and sigmoid(beta)).
__global__ void __launch_bounds__(128) la_prepare_kernel(const LaScanArgs A) {
    ap_pdl_trigger();
    ap_pdl_wait();
    const int lane = threadIdx.x & 31;
    const int G = A.qk_heads, H = A.heads, D = A.D;
    const int qk_units = A.qk_mode == QK_PLAIN ? 0 : 2 * G;
    const int v_units = A.qk_mode == QKV_SILU ? H : 0;
    const int ch_units = la_per_channel(A.decay_mode) ? H : 0;
    const int sc_units = (A.decay_mode == DECAY_HEAD_TOKEN || A.delta) ? 1 : 0;
    const int units = qk_units + v_units + ch_units + sc_units;
    const long long unit = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (unit >= (long long)A.T * units) return;
    const int t = (int)(unit / units);
    int u = (int)(unit % units);
    if (u < qk_units) {
        float* p = u < G ? A.q + (size_t)t * A.ld_q + (size_t)u * D : A.k + (size_t)t * A.ld_k + (size_t)(u - G) * D;
        if (A.qk_mode == QK_ROTATE) {
            const int half = A.rot_dims / 2;
            for (int j = lane; j < half; j += 32) {
                const float2 cs = *reinterpret_cast<const float2*>(A.cos_sin + ((size_t)t * half + j) * 2);
                const float a = p[j], b = p[j + half];
                p[j] = a * cs.x - b * cs.y;
                p[j + half] = b * cs.x + a * cs.y;
            }
        } else if (A.qk_mode == QKV_SILU) {
            for (int d = lane; d < D; d += 32) p[d] = la_silu(p[d]);
        } else {
            float ss = 0.f;
            for (int d = lane; d < D; d += 32) ss = fmaf(p[d], p[d], ss);
            ss = ap_warp_sum(ss);
            const float f = 1.0f / sqrtf(ss + A.unit_eps);
            for (int d = lane; d < D; d += 32) p[d] *= f;
        }
        return;
    }
    u -= qk_units;
    if (u < v_units) {
        float* p = A.v + (size_t)t * A.ld_v + (size_t)u * A.V;
        for (int d = lane; d < A.V; d += 32) p[d] = la_silu(p[d]);
        return;
    }
    u -= v_units;
    if (u < ch_units) {
        float* z = A.decay_channel + (size_t)t * A.ld_dc + (size_t)u * D;
        if (A.decay_mode == DECAY_CHANNEL) {
            for (int d = lane; d < D; d += 32) z[d] = expf(-la_softplus(-z[d]) * A.inv_tau);
        } else {
            const float rate = expf(A.decay_const[u]);
            const float* b = A.dt_bias ? A.dt_bias + (size_t)u * D : nullptr;
            for (int d = lane; d < D; d += 32) z[d] = expf(-rate * la_softplus(z[d] + (b ? b[d] : 0.f)));
        }
        return;
    }
    for (int h = lane; h < H; h += 32) {
        if (A.decay_mode == DECAY_HEAD_TOKEN) {
            float* a = A.decay_head + (size_t)t * A.ld_dh + h;
            *a = expf(-expf(A.decay_const[h]) * la_softplus(*a + (A.dt_bias ? A.dt_bias[h] : 0.f)));
        }
        if (A.delta) {
            float* b = A.beta + (size_t)t * A.ld_beta + h;
            *b = 1.0f / (1.0f + expf(-*b));
        }
    }
}

// One CTA per (sequence, head, block of value columns).  A thread holds PER state entries of one value
// column: the column's D entries are dealt to NP neighbouring lanes (a power of two up to 32) in runs of four
// (entry i of lane p is row (i / 4) * 4 NP + 4 p + i % 4, so that the lanes' 16-byte reads of a key lie side by
// side in shared memory), and the lanes' partial sums meet by shuffles.  Few lanes with many entries each keep the
// instructions per state entry low: a row costs a thread three operations per entry and one short reduction
// (two with the delta rule).  Tokens come LA_CHUNK at a time through two shared-memory buffers filled by
// asynchronous copies while the chunk before is computed.
template <int PER, int NP>
__global__ void __launch_bounds__(128) la_scan_kernel(const LaScanArgs A) {
    extern __shared__ __align__(16) float sm[];
    ap_pdl_trigger();
    ap_pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y;
    const int a = A.seq_start[s], n = A.seq_start[s + 1] - a;
    if (n <= 0) return;
    const int D = A.D, V = A.V, cols = A.cols;
    const int g = h / (A.heads / A.qk_heads);
    const int col0 = blockIdx.z * cols;
    const int ncols = min(cols, V - col0);
    const int vl = threadIdx.x / NP, part = threadIdx.x % NP;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    const int vcol = col0 + vl;
    const bool live = vl < ncols;
    const bool channel = la_per_channel(A.decay_mode), delta = A.delta != 0, gated = A.beta != nullptr;
    const bool token_decay = A.decay_mode == DECAY_HEAD_TOKEN || A.decay_mode == DECAY_HEAD_READY;
    const int vcols = min(ncols, A.VI - col0);               // columns that v brings; the unit column (if it lies here) follows
    const int XS = (cols + 3) / 4 * 4, DS = PER * NP;        // a row of keys in shared memory is padded with zeros
    // one buffer: v [CHUNK][XS], k [CHUNK][DS], q [CHUNK][DS], channel decays [CHUNK][DS] (if any), decay [CHUNK], beta [CHUNK]
    const int buf_floats = LA_CHUNK * (XS + (channel ? 3 : 2) * DS) + 2 * LA_CHUNK;
    if (DS > D) {
        // the rows' tails beyond D stay zero for good (the copies write the first D numbers only)
        const int pad = DS - D, per_buf = (channel ? 3 : 2) * LA_CHUNK;
        for (int i = threadIdx.x; i < 2 * per_buf * pad; i += blockDim.x) {
            const int b = i / (per_buf * pad), j = i - b * per_buf * pad;
            sm[b * buf_floats + LA_CHUNK * XS + (j / pad) * DS + D + j % pad] = 0.f;
        }
    }
    if (vcols < ncols)                                       // no copy writes it
        for (int i = threadIdx.x; i < 2 * LA_CHUNK; i += blockDim.x)
            sm[(i / LA_CHUNK) * buf_floats + (i % LA_CHUNK) * XS + vcols] = 1.f;
    float* st = A.state + (size_t)A.state_slots[s] * A.state_stride + (size_t)h * D * V;
    const bool fresh = A.positions[a] == 0;
    float S[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int nn = (i >> 2) * 4 * NP + 4 * part + (i & 3);
        S[i] = (!fresh && live && nn < D) ? st[(size_t)nn * V + vcol] : 0.f;
    }
    const float head_decay = A.decay_mode == DECAY_HEAD_CONST ? A.decay_const[h] : 1.0f;
    const bool vec = A.vec != 0;
    __syncthreads();

    auto stage = [&](int t0, float* buf) {
        const int cnt = min(LA_CHUNK, n - t0);
        float* v_b = buf;
        float* k_b = v_b + LA_CHUNK * XS;
        float* q_b = k_b + LA_CHUNK * DS;
        float* c_b = q_b + LA_CHUNK * DS;
        float* sc_b = c_b + (channel ? LA_CHUNK * DS : 0);
        const size_t row = (size_t)(a + t0);
        // values: eight threads to a row; keys, queries and channel decays: a warp to a row, the lanes across it
        for (int r = threadIdx.x >> 3; r < cnt; r += blockDim.x >> 3) {
            const float* src = A.v + (row + r) * A.ld_v + (size_t)h * A.VI + col0;
            if (vec && vcols % 4 == 0) for (int d = (threadIdx.x & 7) * 4; d < vcols; d += 32) la_copy16(v_b + r * XS + d, src + d);
            else for (int d = threadIdx.x & 7; d < vcols; d += 8) la_copy4(v_b + r * XS + d, src + d);
        }
        for (int r = warp; r < cnt; r += nwarps) {
            const float* ks = A.k + (row + r) * A.ld_k + (size_t)g * D;
            const float* qs = A.q + (row + r) * A.ld_q + (size_t)g * D;
            const float* cs = channel ? A.decay_channel + (row + r) * A.ld_dc + (size_t)h * D : nullptr;
            if (vec) {
                for (int d = lane * 4; d < D; d += 128) {
                    la_copy16(k_b + r * DS + d, ks + d);
                    la_copy16(q_b + r * DS + d, qs + d);
                    if (channel) la_copy16(c_b + r * DS + d, cs + d);
                }
            } else {
                for (int d = lane; d < D; d += 32) {
                    la_copy4(k_b + r * DS + d, ks + d);
                    la_copy4(q_b + r * DS + d, qs + d);
                    if (channel) la_copy4(c_b + r * DS + d, cs + d);
                }
            }
        }
        if ((int)threadIdx.x < cnt) {
            if (token_decay) la_copy4(sc_b + threadIdx.x, A.decay_head + (row + threadIdx.x) * A.ld_dh + h);
            if (gated) la_copy4(sc_b + LA_CHUNK + threadIdx.x, A.beta + (row + threadIdx.x) * A.ld_beta + h);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    stage(0, sm);
    int which_buf = 0;
    for (int t0 = 0; t0 < n; t0 += LA_CHUNK, which_buf ^= 1) {
        const int cnt = min(LA_CHUNK, n - t0);
        float* buf = sm + which_buf * buf_floats;
        if (t0 + LA_CHUNK < n) {
            stage(t0 + LA_CHUNK, sm + (which_buf ^ 1) * buf_floats);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* v_s = buf;
        const float* k_s = v_s + LA_CHUNK * XS + 4 * part;
        const float* q_s = k_s + LA_CHUNK * DS;
        const float* c_s = q_s + LA_CHUNK * DS;
        const float* sc_s = buf + LA_CHUNK * (XS + (channel ? 3 : 2) * DS);
        float* yp = A.y + (size_t)(a + t0) * A.ld_y + (size_t)h * V + vcol;
#pragma unroll 2
        for (int r = 0; r < cnt; ++r, yp += A.ld_y) {
            const float vv = live ? v_s[r * XS + vl] : 0.f;
            float kk[PER], qq[PER];
#pragma unroll
            for (int j = 0; j < PER / 4; ++j) {
                *reinterpret_cast<float4*>(kk + 4 * j) = *reinterpret_cast<const float4*>(k_s + r * DS + j * 4 * NP);
                *reinterpret_cast<float4*>(qq + 4 * j) = *reinterpret_cast<const float4*>(q_s + r * DS + j * 4 * NP);
            }
            if (channel) {
#pragma unroll
                for (int j = 0; j < PER / 4; ++j) {
                    const float4 c = *reinterpret_cast<const float4*>(c_s + r * DS + j * 4 * NP);
                    S[4 * j] *= c.x; S[4 * j + 1] *= c.y; S[4 * j + 2] *= c.z; S[4 * j + 3] *= c.w;
                }
            } else {
                const float dec = token_decay ? sc_s[r] : head_decay;
#pragma unroll
                for (int i = 0; i < PER; ++i) S[i] *= dec;
            }
            float u = vv;
            if (gated && !delta) u = sc_s[LA_CHUNK + r] * vv;
            if (delta) {
                float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
#pragma unroll
                for (int j = 0; j < PER / 4; ++j) {
                    d0 = fmaf(S[4 * j], kk[4 * j], d0); d1 = fmaf(S[4 * j + 1], kk[4 * j + 1], d1);
                    d2 = fmaf(S[4 * j + 2], kk[4 * j + 2], d2); d3 = fmaf(S[4 * j + 3], kk[4 * j + 3], d3);
                }
                float dot = (d0 + d1) + (d2 + d3);
#pragma unroll
                for (int o = NP >> 1; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
                u = sc_s[LA_CHUNK + r] * (vv - dot);
            }
            float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
            for (int j = 0; j < PER / 4; ++j) {
                S[4 * j] = fmaf(kk[4 * j], u, S[4 * j]); a0 = fmaf(S[4 * j], qq[4 * j], a0);
                S[4 * j + 1] = fmaf(kk[4 * j + 1], u, S[4 * j + 1]); a1 = fmaf(S[4 * j + 1], qq[4 * j + 1], a1);
                S[4 * j + 2] = fmaf(kk[4 * j + 2], u, S[4 * j + 2]); a2 = fmaf(S[4 * j + 2], qq[4 * j + 2], a2);
                S[4 * j + 3] = fmaf(kk[4 * j + 3], u, S[4 * j + 3]); a3 = fmaf(S[4 * j + 3], qq[4 * j + 3], a3);
            }
            float acc = (a0 + a1) + (a2 + a3);
#pragma unroll
            for (int o = NP >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            if (live && part == 0) *yp = acc * A.out_scale;
        }
        __syncthreads();                                     // this buffer is filled again two chunks on
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int nn = (i >> 2) * 4 * NP + 4 * part + (i & 3);
            if (nn < D) st[(size_t)nn * V + vcol] = S[i];
        }
    }
}

// ---- the recurrence, eight tokens at a time -------------------------------------------------
// What a prompt's portion takes instead of the chain above.  Over a block of tokens the recurrence closes into sums that
// need the state only as it was before them.  With c_r the decays of token r (a vector over the key channels, or a number),
// C_r = c_0 .. c_r their running product and c(j, r) = c_{j+1} .. c_r what is left of token j's write at token r:
//
//   u_r = beta_r (v_r - S^T (C_r k_r) - sum_{j<r} [k_r . c(j, r) k_j] u_j)          (delta rule; else u_r = v_r)
//   o_r = S^T (C_r q_r) + sum_{j<=r} [q_r . c(j, r) k_j] u_j
//   S  <- C_7 S + sum_j (c(j, 7) k_j) u_j^T
//
// The bracketed numbers and the vectors with their decays do not depend on the state: la_blocks_kernel forms them once
// per (eight tokens, head), together with everything the rows need before the recurrence (rotation, unit vectors, SiLU,
// decays, gates), and leaves them in one block of scratch.  The recurrence's chain is then one step per EIGHT tokens, whose
// sums meet over the lanes in the same rounds of shuffles, and a state entry costs three multiply-adds a token, two entries
// to an instruction.  All 32-bit, products of decays included (none is ever divided by).  A block of fewer tokens is filled
// up with tokens that do nothing.
//
// A block: the numbers (REC_*), then rows C_r k_r, rows C_r q_r, for decays per channel also rows c(j, 7) k_j and the row
// C_7, each padded with zeros to DS = PER * NP numbers, then rows of values (times beta) padded to VS.  The block of
// (sequence s, rows 8i .. of its portion, head h) lies at index (seq_start[s] / 8 + i + s) * heads + h.
#define LT 8                     // tokens of a block
#define REC_BA 0                 // beta_r * C_r (C_r is 1 here where the vectors hold it)
#define REC_A (REC_BA + LT)      // rows r = 1 .. 7: beta_r [k_r . c(j, r) k_j], j < r, in runs of four
#define REC_GAMMA (REC_A + 40)   // c(r, 7)
#define REC_ALPHA (REC_GAMMA + LT)   // C_r * out_scale
#define REC_P (REC_ALPHA + LT)   // rows r = 0 .. 7: [q_r . c(j, r) k_j] * out_scale, zero for j > r
#define REC_TOTAL (REC_P + LT * LT)  // C_7
#define REC_SIZE (REC_TOTAL + 4)
#define PAIRS_BELOW (LT * (LT - 1) / 2)
__host__ __device__ constexpr int rec_a_row(int r) { return REC_A + (r <= 4 ? (r - 1) * 4 : 16 + (r - 5) * 8); }

#define LC_WARPS_WANTED 400L     // warps a step of portions should bring to the GPU's schedulers

struct LaBlocks { float* at; int DS, VS, size; };

// (first row, rows, place in the scratch) of the b-th block; false beyond the last
__device__ __forceinline__ bool lc_find(const int* seq_start, int nseq, int b, int& row, int& cnt, int& index) {
    for (int s = 0; s < nseq; ++s) {
        const int a = seq_start[s], n = seq_start[s + 1] - a, groups = (n + LT - 1) / LT;
        if (b < groups) {
            row = a + b * LT;
            cnt = min(LT, n - b * LT);
            index = a / LT + b + s;
            return true;
        }
        b -= groups;
    }
    return false;
}

// Sums over a warp's lanes of N numbers (a multiple of 32): every round halves what a lane holds; lane l ends with
// the sums of numbers l * N / 32 .. in places 0 ..
template <int N> __device__ __forceinline__ void la_scatter_sums(float (&v)[N], int lane) {
#pragma unroll
    for (int n = N / 2, o = 16; o >= 1; n >>= 1, o >>= 1) {
        const bool up = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < N / 2; ++i) {
            if (i < n) {
                const float send = up ? v[i] : v[i + n], keep = up ? v[i + n] : v[i];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        }
    }
}

// One CTA per (block of tokens, head), a channel to a thread.  CH: 0, DECAY_CHANNEL or DECAY_CHANNEL_TOKEN.
template <int CH>
__global__ void __launch_bounds__(128, 4) la_blocks_kernel(const LaScanArgs A, const LaBlocks B, int nseq) {
    __shared__ float red[4][2 * 32], numbers[2][LT], unit_s[2 * LT];
    ap_pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const int H = A.heads, D = A.D, V = A.V, DS = B.DS, VS = B.VS;
    const int h = (int)(blockIdx.x % H), g = h / (H / A.qk_heads);
    int row, cnt, index;
    if (!lc_find(A.seq_start, nseq, (int)(blockIdx.x / H), row, cnt, index)) return;
    float* rec = B.at + ((size_t)index * H + h) * B.size;
    float* kt = rec + REC_SIZE;
    float* qt = kt + LT * DS;
    float* kh = qt + LT * DS;
    float* ct = kh + LT * DS;
    float* vb = CH ? ct + DS : kh;
    const int mode = A.qk_mode, half = A.rot_dims / 2;
    const float* qp = A.q + (size_t)row * A.ld_q + (size_t)g * D;
    const float* kp = A.k + (size_t)row * A.ld_k + (size_t)g * D;
    const float* zp = CH ? A.decay_channel + (size_t)row * A.ld_dc + (size_t)h * D : nullptr;
    // the numbers of each token: gate of the write, decay of the head (1 where channels have their own)
    if (threadIdx.x < LT) {
        const int r = threadIdx.x;
        const size_t t = (size_t)row + r;
        float b = r < cnt ? 1.f : 0.f, a = 1.f;
        if (r < cnt) {
            if (A.beta) b = A.delta ? 1.0f / (1.0f + expf(-A.beta[t * A.ld_beta + h])) : A.beta[t * A.ld_beta + h];
            if (A.decay_mode == DECAY_HEAD_CONST) a = A.decay_const[h];
            if (A.decay_mode == DECAY_HEAD_READY) a = A.decay_head[t * A.ld_dh + h];
            if (A.decay_mode == DECAY_HEAD_TOKEN)
                a = expf(-expf(A.decay_const[h]) * la_softplus(A.decay_head[t * A.ld_dh + h] + (A.dt_bias ? A.dt_bias[h] : 0.f)));
        }
        numbers[0][r] = b;
        numbers[1][r] = a;
    }
    if (mode == QK_UNIT) {
        float ss[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) ss[i] = 0.f;
        for (int d = threadIdx.x; d < D; d += blockDim.x) {
#pragma unroll
            for (int r = 0; r < LT; ++r) {
                const float q = r < cnt ? qp[r * A.ld_q + d] : 0.f, k = r < cnt ? kp[r * A.ld_k + d] : 0.f;
                ss[r] = fmaf(q, q, ss[r]);
                ss[LT + r] = fmaf(k, k, ss[LT + r]);
            }
        }
        la_scatter_sums<32>(ss, lane);
        if (lane < 2 * LT) red[warp][lane] = ss[0];
        __syncthreads();
        if (threadIdx.x < 2 * LT) {
            float sum = 0.f;
            for (int w = 0; w < nwarps; ++w) sum += red[w][threadIdx.x];
            unit_s[threadIdx.x] = 1.0f / sqrtf(sum + A.unit_eps);
        }
    }
    __syncthreads();
    const float rate = CH == DECAY_CHANNEL_TOKEN ? expf(A.decay_const[h]) : 0.f;
    float acc[64];                                           // pairs j < r of keys, then pairs j <= r of queries and keys
#pragma unroll
    for (int i = 0; i < 64; ++i) acc[i] = 0.f;
    for (int d = threadIdx.x; d < DS; d += blockDim.x) {
        float q[LT], k[LT], c[LT];
#pragma unroll
        for (int r = 0; r < LT; ++r) {
            const bool in = r < cnt && d < D;
            q[r] = in ? qp[r * A.ld_q + d] : 0.f;
            k[r] = in ? kp[r * A.ld_k + d] : 0.f;
            c[r] = (CH && in) ? zp[r * A.ld_dc + d] : 0.f;
        }
        if (mode == QK_UNIT) {
#pragma unroll
            for (int r = 0; r < LT; ++r) { q[r] *= unit_s[r]; k[r] *= unit_s[LT + r]; }
        } else if (mode == QKV_SILU) {
#pragma unroll
            for (int r = 0; r < LT; ++r) { q[r] = la_silu(q[r]); k[r] = la_silu(k[r]); }
        } else if (mode == QK_ROTATE && d < A.rot_dims) {
            const int m = d < half ? d : d - half, partner = d < half ? d + half : d - half;
#pragma unroll
            for (int r = 0; r < LT; ++r) {
                if (r < cnt) {
                    const float2 cs = *reinterpret_cast<const float2*>(A.cos_sin + (((size_t)row + r) * half + m) * 2);
                    const float sn = d < half ? -cs.y : cs.y;
                    q[r] = q[r] * cs.x + qp[r * A.ld_q + partner] * sn;
                    k[r] = k[r] * cs.x + kp[r * A.ld_k + partner] * sn;
                }
            }
        }
        if (CH) {
            const float bias = (CH == DECAY_CHANNEL_TOKEN && A.dt_bias && d < D) ? A.dt_bias[(size_t)h * D + d] : 0.f;
#pragma unroll
            for (int r = 0; r < LT; ++r) {
                const float e = CH == DECAY_CHANNEL ? expf(-la_softplus(-c[r]) * A.inv_tau) : expf(-rate * la_softplus(c[r] + bias));
                c[r] = r < cnt ? e : 1.f;
            }
        }
        // kk[j] becomes c(j, r) k_j as r goes on
        float kk[LT], upto = 1.f;
        int below = 0, upon = PAIRS_BELOW;
#pragma unroll
        for (int r = 0; r < LT; ++r) {
            if (CH) {
                upto *= c[r];
#pragma unroll
                for (int j = 0; j < r; ++j) kk[j] *= c[r];
            }
            kk[r] = k[r];
#pragma unroll
            for (int j = 0; j < r; ++j) {
                acc[below + j] = fmaf(k[r], kk[j], acc[below + j]);
                acc[upon + j] = fmaf(q[r], kk[j], acc[upon + j]);
            }
            acc[upon + r] = fmaf(q[r], k[r], acc[upon + r]);
            below += r;
            upon += r + 1;
            kt[r * DS + d] = CH ? upto * k[r] : k[r];
            qt[r * DS + d] = CH ? upto * q[r] : q[r];
        }
        if (CH) {
#pragma unroll
            for (int r = 0; r < LT; ++r) kh[r * DS + d] = kk[r];
            ct[d] = d < D ? upto : 0.f;
        }
    }
    la_scatter_sums<64>(acc, lane);
    red[warp][2 * lane] = acc[0];
    red[warp][2 * lane + 1] = acc[1];
    __syncthreads();
    const float* beta = numbers[0];
    const float* a = numbers[1];
    for (int t = threadIdx.x; t < LT * LT; t += blockDim.x) {
        float sum = 0.f;
        for (int w = 0; w < nwarps; ++w) sum += red[w][t];
        // number t is (r, j): t = r (r - 1) / 2 + j below the diagonal, then r (r + 1) / 2 + j with it
        const bool keys = t < PAIRS_BELOW;
        int r = keys ? 1 : 0, j = keys ? t : t - PAIRS_BELOW;
        while (j >= (keys ? r : r + 1)) { j -= keys ? r : r + 1; ++r; }
        float left = 1.f;                                    // what the head's decays leave of token j at token r
        for (int i = j + 1; i <= r; ++i) left *= a[i];
        if (keys) rec[(r <= 4 ? REC_A + (r - 1) * 4 : REC_A + 16 + (r - 5) * 8) + j] = beta[r] * left * sum;
        else rec[REC_P + r * LT + j] = A.out_scale * left * sum;
        if ((t & (LT - 1)) > t / LT) rec[REC_P + t] = 0.f;   // a later token's write
    }
    if (threadIdx.x < LT) {
        const int r = threadIdx.x;
        float upto = 1.f, after = 1.f;
        for (int i = 0; i < LT; ++i) {
            if (i <= r) upto *= a[i];
            else after *= a[i];
        }
        rec[REC_BA + r] = beta[r] * upto;
        rec[REC_GAMMA + r] = after;
        rec[REC_ALPHA + r] = upto * A.out_scale;
        if (r == LT - 1) rec[REC_TOTAL] = upto;
    }
    for (int r = 0; r < LT; ++r) {
        const float* vp = A.v + ((size_t)row + r) * A.ld_v + (size_t)h * A.VI;
        for (int d = threadIdx.x; d < VS; d += blockDim.x) {
            float v = (r < cnt && d < A.VI) ? vp[d] : 0.f;
            if (mode == QKV_SILU) v = la_silu(v);
            if (d >= A.VI && d < V) v = 1.f;                 // (beta is 0 beyond the last token)
            vb[r * VS + d] = beta[r] * v;
        }
    }
}

// two 32-bit numbers to a register pair, multiplied and added in one instruction
typedef unsigned long long la_pair;
__device__ __forceinline__ la_pair la_fma2(la_pair a, la_pair b, la_pair c) {
    la_pair d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ la_pair la_mul2(la_pair a, la_pair b) {
    la_pair d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ la_pair la_pack(float lo, float hi) {
    la_pair d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 la_unpack(la_pair p) {
    float2 v;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(v.x), "=f"(v.y) : "l"(p));
    return v;
}
__device__ __forceinline__ float la_sum2(la_pair p) { const float2 v = la_unpack(p); return v.x + v.y; }

// One CTA per (sequence, head, block of value columns).  NP lanes share CPT columns; a lane holds PER entries of each
// (entry i of lane p is row (i / 4) * 4 NP + 4 p + i % 4), so that a vector read from shared memory serves CPT columns: what
// bounds this kernel is the width of shared memory, one 128-byte wavefront per number and warp, and repeated addresses
// within a warp do not make a 16-byte read cheaper.  A lane keeps its columns in an order of its own, column c ^ (p mod
// CPT) in place c: in the first rounds of the sums over the lanes a lane then always sends the upper half of what it holds
// and keeps the lower, without choosing, and ends with the numbers of column p mod CPT, whose writes u it works out
// together with the M = NP / CPT lanes that ended on the same column.  `stage` blocks of eight tokens at a time come
// through two shared-memory buffers.
template <int PER, int NP, int CPT, bool CHANNEL, bool DELTA>
__global__ void __launch_bounds__(128, 1) la_chunk_kernel(const LaScanArgs A, const LaBlocks B, int stage) {
    extern __shared__ __align__(16) float sm[];
    ap_pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y;
    const int a = A.seq_start[s], n = A.seq_start[s + 1] - a;
    if (n <= 0) return;
    constexpr int DS = PER * NP, MAIN = REC_SIZE + (CHANNEL ? 3 * LT + 1 : 2 * LT) * DS;
    constexpr int COLS = 128 / NP * CPT, M = NP / CPT, ONE = MAIN + LT * COLS;
    const int D = A.D, V = A.V, VS = B.VS;
    const int col0 = blockIdx.z * COLS;
    const int vcols = min(COLS, VS - col0);                   // columns to bring: whole 16-byte runs
    const int part = threadIdx.x % NP, swap = part % CPT, idx = part / CPT;
    const int first = threadIdx.x / NP * CPT;                 // this lane's columns in the block: first + (c ^ swap)
    float* st = A.state + (size_t)A.state_slots[s] * A.state_stride + (size_t)h * D * V + col0 + first;
    const bool fresh = A.positions[a] == 0;
    la_pair S[CPT][PER / 2];
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const bool live = col0 + first + (c ^ swap) < V;
#pragma unroll
        for (int i = 0; i < PER / 2; ++i) {
            float e[2];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int m = 2 * i + k, nn = (m >> 2) * 4 * NP + 4 * part + (m & 3);
                e[k] = (!fresh && live && nn < D) ? st[(size_t)nn * V + (c ^ swap)] : 0.f;
            }
            S[c][i] = la_pack(e[0], e[1]);
        }
    }
    const int groups = (n + LT - 1) / LT;
    const float* src = B.at + ((size_t)(a / LT + s) * A.heads + h) * B.size;
    const size_t step = (size_t)A.heads * B.size;

    auto fetch = [&](int g0, float* buf) {
        const int cnt = min(stage, groups - g0);
        for (int g = 0; g < cnt; ++g) {
            const float* from = src + (size_t)(g0 + g) * step;
            float* to = buf + g * ONE;
#pragma unroll
            for (int i = 0; i < (MAIN + 511) / 512; ++i) {
                const int at = (i * 128 + threadIdx.x) * 4;
                if (at < MAIN) la_copy16(to + at, from + at);
            }
            const float* vfrom = from + MAIN + col0;
            for (int i = threadIdx.x; i < LT * (COLS / 4); i += 128) {
                const int r = i / (COLS / 4), c = i % (COLS / 4) * 4;
                if (c < vcols) la_copy16(to + MAIN + r * COLS + c, vfrom + (size_t)r * VS + c);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    // the token (or the tokens, with fewer lanes to a column) whose read-out of this lane's column it finishes; of the
    // lanes that end with the same one the first stores it
    constexpr int QN = M >= LT ? 1 : LT / M;
    int q_first = 0;
#pragma unroll
    for (int o = M >> 1, n2 = LT >> 1; o > 0 && n2 > 0; o >>= 1, n2 >>= 1) q_first += (idx & o) ? n2 : 0;
    const bool writer = col0 + first + swap < V && (M <= LT || (idx & (M / LT - 1)) == 0);
    float* yp = A.y + (size_t)a * A.ld_y + (size_t)h * V + col0 + first + swap;

    fetch(0, sm);
    int which = 0;
    for (int g0 = 0; g0 < groups; g0 += stage, which ^= 1) {
        const int cnt = min(stage, groups - g0);
        float* buf = sm + which * stage * ONE;
        if (g0 + stage < groups) {
            fetch(g0 + stage, sm + (which ^ 1) * stage * ONE);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        for (int g = 0; g < cnt; ++g) {
            const float* rec = buf + g * ONE;
            const float* kt = rec + REC_SIZE + 4 * part;
            const float* qt = kt + LT * DS;
            const float* kh = CHANNEL ? qt + LT * DS : kt;
            const float* ct = kh + LT * DS;
            const float* vs = rec + MAIN + first + swap;
            float kd[LT][CPT], qd[LT][CPT];
#pragma unroll
            for (int r = 0; r < LT; ++r) {
                la_pair ak[CPT], aq[CPT];
#pragma unroll
                for (int i = 0; i < PER / 4; ++i) {
                    const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(qt + r * DS + i * 4 * NP);
#pragma unroll
                    for (int c = 0; c < CPT; ++c) {
                        aq[c] = i == 0 ? la_mul2(S[c][0], q.x) : la_fma2(S[c][2 * i], q.x, aq[c]);
                        aq[c] = la_fma2(S[c][2 * i + 1], q.y, aq[c]);
                    }
                    if (DELTA) {
                        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(kt + r * DS + i * 4 * NP);
#pragma unroll
                        for (int c = 0; c < CPT; ++c) {
                            ak[c] = i == 0 ? la_mul2(S[c][0], k.x) : la_fma2(S[c][2 * i], k.x, ak[c]);
                            ak[c] = la_fma2(S[c][2 * i + 1], k.y, ak[c]);
                        }
                    }
                }
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    qd[r][c] = la_sum2(aq[c]);
                    kd[r][c] = DELTA ? la_sum2(ak[c]) : 0.f;
                }
            }
            // the sums over the lanes: first the columns part ways ...
#pragma unroll
            for (int o = CPT >> 1; o > 0; o >>= 1)
#pragma unroll
                for (int r = 0; r < LT; ++r)
#pragma unroll
                    for (int c = 0; c < o; ++c) {
                        if (DELTA) kd[r][c] += __shfl_xor_sync(0xffffffffu, kd[r][c + o], o);
                        qd[r][c] += __shfl_xor_sync(0xffffffffu, qd[r][c + o], o);
                    }
            // ... then the keys' sums end on every lane of a column, the queries' on one lane (or a few) to a token
            if (DELTA) {
#pragma unroll
                for (int o = M >> 1; o > 0; o >>= 1)
#pragma unroll
                    for (int r = 0; r < LT; ++r) kd[r][0] += __shfl_xor_sync(0xffffffffu, kd[r][0], o * CPT);
            }
            float qs[LT], u[LT];
#pragma unroll
            for (int r = 0; r < LT; ++r) { qs[r] = qd[r][0]; u[r] = vs[r * COLS]; }
#pragma unroll
            for (int o = M >> 1, n2 = LT >> 1; o > 0; o >>= 1, n2 >>= 1) {
                if (n2 > 0) {
                    const bool up = (idx & o) != 0;
#pragma unroll
                    for (int i = 0; i < LT / 2; ++i) {
                        if (i < n2) {
                            const float send = up ? qs[i] : qs[i + n2], keep = up ? qs[i + n2] : qs[i];
                            qs[i] = keep + __shfl_xor_sync(0xffffffffu, send, o * CPT);
                        }
                    }
                } else {
                    qs[0] += __shfl_xor_sync(0xffffffffu, qs[0], o * CPT);
                }
            }
            if (DELTA) {
                float num[REC_GAMMA];                        // beta C and the rows of earlier tokens' shares, 16 bytes a read
#pragma unroll
                for (int i = 0; i < REC_GAMMA; i += 4)
                    *reinterpret_cast<float4*>(num + i) = *reinterpret_cast<const float4*>(rec + i);
#pragma unroll
                for (int r = 0; r < LT; ++r) u[r] = fmaf(-num[REC_BA + r], kd[r][0], u[r]);
#pragma unroll
                for (int j = 0; j + 1 < LT; ++j)
#pragma unroll
                    for (int r = j + 1; r < LT; ++r) u[r] = fmaf(-num[rec_a_row(r) + j], u[j], u[r]);
            }
            // the write of every column this lane holds (with what the head's decays leave of it, where the vectors
            // hold none)
            float w[LT];
            if (CHANNEL) {
#pragma unroll
                for (int r = 0; r < LT; ++r) w[r] = u[r];
            } else {
#pragma unroll
                for (int r = 0; r < LT; ++r) w[r] = rec[REC_GAMMA + r] * u[r];
            }
            la_pair w2[LT][CPT];
#pragma unroll
            for (int r = 0; r < LT; ++r)
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    const float x = c == 0 ? w[r] : __shfl_xor_sync(0xffffffffu, w[r], c);
                    w2[r][c] = la_pack(x, x);
                }
            const float total = rec[REC_TOTAL];
            const la_pair tot2 = la_pack(total, total);
#pragma unroll
            for (int i = 0; i < PER / 4; ++i) {
                ulonglong2 d = make_ulonglong2(tot2, tot2);
                if (CHANNEL) d = *reinterpret_cast<const ulonglong2*>(ct + i * 4 * NP);
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    S[c][2 * i] = la_mul2(S[c][2 * i], d.x);
                    S[c][2 * i + 1] = la_mul2(S[c][2 * i + 1], d.y);
                }
#pragma unroll
                for (int r = 0; r < LT; ++r) {
                    const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(kh + r * DS + i * 4 * NP);
#pragma unroll
                    for (int c = 0; c < CPT; ++c) {
                        S[c][2 * i] = la_fma2(k.x, w2[r][c], S[c][2 * i]);
                        S[c][2 * i + 1] = la_fma2(k.y, w2[r][c], S[c][2 * i + 1]);
                    }
                }
            }
            const int t0 = (g0 + g) * LT;
#pragma unroll
            for (int i = 0; i < QN; ++i) {
                const int r = q_first + i;
                float y = rec[REC_ALPHA + r] * qs[i];
#pragma unroll
                for (int j = 0; j < LT; j += 4) {
                    const float4 p = *reinterpret_cast<const float4*>(rec + REC_P + LT * r + j);
                    y = fmaf(p.w, u[j + 3], fmaf(p.z, u[j + 2], fmaf(p.y, u[j + 1], fmaf(p.x, u[j], y))));
                }
                if (writer && t0 + r < n) yp[(size_t)(t0 + r) * A.ld_y] = y;
            }
        }
        __syncthreads();                                     // this buffer is filled again two stages on
    }
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        if (col0 + first + (c ^ swap) >= V) continue;
#pragma unroll
        for (int i = 0; i < PER / 2; ++i) {
            const float2 e = la_unpack(S[c][i]);
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int m = 2 * i + k, nn = (m >> 2) * 4 * NP + 4 * part + (m & 3);
                if (nn < D) st[(size_t)nn * V + (c ^ swap)] = k ? e.y : e.x;
            }
        }
    }
}

// State entries to threads: as few lanes to a column as hold it (up to 16 entries a thread: the fewest instructions
// per state entry); more of them (shorter chains per thread, more warps) only while the step's columns leave
// schedulers without a warp.
static void la_plan(int nseq, int heads, int D, int V, int& NP, int& per) {
    NP = 1;
    while (NP * LA_PER_MAX < D) NP *= 2;
    while (NP < 32 && NP * 4 < D && (long long)nseq * heads * V * NP / 32 < 148 * 4) NP *= 2;
    per = ((D + NP - 1) / NP + 3) / 4 * 4;
    per = per <= 4 ? 4 : (per <= 8 ? 8 : LA_PER_MAX);
}
// whether a step of T rows goes eight tokens at a time: where its sequences bring several rows
static bool la_in_blocks(int T, int nseq) { return T > 2 * nseq; }

// The same for la_chunk_kernel: keys over as many lanes as give each four entries of a column (up to 32 lanes), and as
// many columns to a lane as still leave every scheduler a warp.
static void lc_plan(int nseq, int heads, int D, int V, int& NP, int& per, int& cpt) {
    NP = 1;
    while (NP < 32 && NP * 4 < D) NP *= 2;
    per = D <= NP * 4 ? 4 : (D <= NP * 8 ? 8 : LA_PER_MAX);
    cpt = NP < 4 ? 1 : ((long long)nseq * heads * V * NP / 32 >= LC_WARPS_WANTED * 4 ? 4 : 2);
}

// numbers of scratch per (block of eight tokens, head) that ap_linear_scan takes for such a step; 0: it takes none
AP_EXPORT int ap_linear_scan_block(int T, int nseq, int heads, int D, int V, int decay_mode) {
    if (T <= 0 || nseq <= 0 || heads <= 0 || D <= 0 || V <= 0 || !la_in_blocks(T, nseq)) return 0;
    int NP, per, cpt;
    lc_plan(nseq, heads, D, V, NP, per, cpt);
    return REC_SIZE + (la_per_channel(decay_mode) ? 3 * LT + 1 : 2 * LT) * per * NP + LT * ((V + 3) / 4 * 4);
}

typedef void (*la_chunk_fn)(const LaScanArgs, const LaBlocks, int);
template <bool CHANNEL, bool DELTA> static la_chunk_fn lc_pick(int per, int NP, int cpt) {
#define LC_PICK(P, N) if (per == P && NP == N) return cpt == 4 ? la_chunk_kernel<P, N, 4, CHANNEL, DELTA> : la_chunk_kernel<P, N, 2, CHANNEL, DELTA>
    LC_PICK(4, 4); LC_PICK(4, 8); LC_PICK(4, 16); LC_PICK(4, 32); LC_PICK(8, 32); LC_PICK(LA_PER_MAX, 32);
#undef LC_PICK
    return NP == 1 ? la_chunk_kernel<4, 1, 1, CHANNEL, DELTA> : la_chunk_kernel<4, 2, 1, CHANNEL, DELTA>;
}

static int la_run_blocks(LaScanArgs& A, int nseq, float* scratch, cudaStream_t stream) {
    int NP, per, cpt;
    lc_plan(nseq, A.heads, A.D, A.V, NP, per, cpt);
    LaBlocks B;
    B.at = scratch;
    B.DS = per * NP;
    B.VS = (A.V + 3) / 4 * 4;
    const bool channel = la_per_channel(A.decay_mode), delta = A.delta != 0;
    const int main_floats = REC_SIZE + (channel ? 3 * LT + 1 : 2 * LT) * B.DS;
    B.size = main_floats + LT * B.VS;
    const int cols = 128 / NP * cpt;
    const dim3 grid((unsigned)nseq, (unsigned)A.heads, (unsigned)((A.V + cols - 1) / cols));
    int stage = 2;
    size_t smem;
    while ((smem = 2 * (size_t)stage * (main_floats + LT * cols) * sizeof(float)) > 100 * 1024 && stage > 1) stage /= 2;
    AP_REQUIRE(smem <= 200 * 1024 && grid.z <= 65535, "linear_scan: keys of %d do not fit the staging buffers", A.D);
    const long long units = ((long long)A.T / LT + nseq) * A.heads;
    AP_REQUIRE(units <= 0x7fffffffLL, "linear_scan: %d rows of %d heads exceed the grid", A.T, A.heads);
    int threads = (A.D + 31) / 32 * 32;
    if (threads > 128) threads = 128;
    auto blocks = A.decay_mode == DECAY_CHANNEL ? la_blocks_kernel<DECAY_CHANNEL>
                : A.decay_mode == DECAY_CHANNEL_TOKEN ? la_blocks_kernel<DECAY_CHANNEL_TOKEN> : la_blocks_kernel<0>;
    AP_CHECK_PDL_LAUNCH("linear_scan (blocks)", ap_launch_pdl(blocks, dim3((unsigned)units), dim3(threads), 0, stream, A, B, nseq));
    la_chunk_fn kern = channel ? (delta ? lc_pick<true, true>(per, NP, cpt) : lc_pick<true, false>(per, NP, cpt))
                               : (delta ? lc_pick<false, true>(per, NP, cpt) : lc_pick<false, false>(per, NP, cpt));
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        AP_REQUIRE(e == cudaSuccess, "linear_scan: cannot reserve %zu bytes of shared memory", smem);
    }
    // the kernel before does not let this one start early: CTAs placed while others still hold most SMs would crowd
    // on the few that are free, and a chain this long does not recover from that
    AP_CHECK_PDL_LAUNCH("linear_scan (eight tokens at a time)", ap_launch_pdl(kern, grid, dim3(128), smem, stream, A, B, stage));
    return AP_OK;
}

AP_EXPORT int ap_linear_scan(float* q, long long ld_q, float* k, long long ld_k, float* v,
                             long long ld_v, float* decay_channel, long long ld_dc, float* decay_head,
                             long long ld_dh, const float* decay_const, const float* dt_bias, float* beta,
                             long long ld_beta, const float* cos_sin, int rot_dims, float* state,
                             long long state_stride, const int* seq_start, const int* positions,
                             const int* state_slots, float* y, long long ld_y, int T, int nseq, int heads,
                             int qk_heads, int D, int V, int decay_mode, int qk_mode, int delta, int unit_column, float tau,
                             float unit_eps, float out_scale, float* scratch, cudaStream_t stream) {
    AP_REQUIRE(T >= 0 && nseq >= 0 && heads > 0 && qk_heads > 0 && heads % qk_heads == 0 && D > 0 && V > 0,
               "linear_scan: bad sizes heads=%d qk_heads=%d key=%d value=%d", heads, qk_heads, D, V);
    AP_REQUIRE(D <= LA_PER_MAX * 32, "linear_scan: keys of %d exceed %d", D, LA_PER_MAX * 32);
    AP_REQUIRE(q && k && v && y && state && state_stride >= (long long)heads * D * V,
               "linear_scan: an operand is missing or the state is too small");
    AP_REQUIRE(decay_mode == DECAY_HEAD_CONST ? decay_const != nullptr
               : decay_mode == DECAY_HEAD_TOKEN ? (decay_head != nullptr && decay_const != nullptr)
               : decay_mode == DECAY_CHANNEL ? (decay_channel != nullptr && tau > 0.f)
               : decay_mode == DECAY_HEAD_READY ? decay_head != nullptr
               : (decay_mode == DECAY_CHANNEL_TOKEN && decay_channel != nullptr && decay_const != nullptr),
               "linear_scan: decay mode %d lacks its numbers", decay_mode);
    AP_REQUIRE(!delta || beta != nullptr, "linear_scan: the delta rule lacks its gates");
    AP_REQUIRE(!unit_column || (V > 1 && qk_mode != QKV_SILU), "linear_scan: a unit column goes with plain values");
    AP_REQUIRE(qk_mode == QK_PLAIN || qk_mode == QK_UNIT || qk_mode == QKV_SILU ||
               (qk_mode == QK_ROTATE && cos_sin && rot_dims > 0 && rot_dims % 2 == 0 && rot_dims <= D),
               "linear_scan: query/key mode %d with %d rotated coordinates of %d", qk_mode, rot_dims, D);
    AP_REQUIRE((((uintptr_t)scratch) & 15) == 0, "linear_scan: the scratch must start on a 16-byte boundary");
    if (T == 0 || nseq == 0) return AP_OK;
    int NP, per;
    la_plan(nseq, heads, D, V, NP, per);
    int cols = 128 / NP;
    if (cols > V) cols = V;
    int threads = (cols * NP + 31) / 32 * 32;
    cols = threads / NP;
    if (cols >= 4) cols = cols / 4 * 4;                     // whole 16-byte runs of the values per CTA
    if (cols > V) cols = V;
    const dim3 grid((unsigned)nseq, (unsigned)heads, (unsigned)((V + cols - 1) / cols));
    AP_REQUIRE(heads <= 65535 && grid.z <= 65535, "linear_scan: %d heads exceed the grid", heads);
    auto aligned = [](const void* p, long long ld) { return p == nullptr || ((((uintptr_t)p) & 15) == 0 && ld % 4 == 0); };
    const int VI = V - (unit_column ? 1 : 0);
    const int vec = (D % 4 == 0 && VI % 4 == 0 && cols % 4 == 0 && aligned(q, ld_q) && aligned(k, ld_k) &&
                     aligned(v, ld_v) && aligned(decay_channel, ld_dc)) ? 1 : 0;
    const bool channel = la_per_channel(decay_mode);
    LaScanArgs A;
    A.q = q; A.ld_q = ld_q; A.k = k; A.ld_k = ld_k; A.v = v; A.ld_v = ld_v;
    A.decay_channel = decay_channel; A.ld_dc = ld_dc; A.decay_head = decay_head; A.ld_dh = ld_dh;
    A.decay_const = decay_const; A.dt_bias = dt_bias; A.beta = beta; A.ld_beta = ld_beta;
    A.cos_sin = cos_sin; A.rot_dims = rot_dims; A.state = state; A.state_stride = state_stride;
    A.seq_start = seq_start; A.positions = positions; A.state_slots = state_slots; A.y = y; A.ld_y = ld_y;
    A.T = T; A.heads = heads; A.qk_heads = qk_heads; A.D = D; A.V = V; A.NP = NP; A.cols = cols;
    A.decay_mode = decay_mode; A.qk_mode = qk_mode; A.vec = vec; A.delta = delta ? 1 : 0; A.VI = VI;
    A.inv_tau = decay_mode == DECAY_CHANNEL ? 1.0f / tau : 0.f; A.unit_eps = unit_eps; A.out_scale = out_scale;
    if (scratch != nullptr && la_in_blocks(T, nseq)) return la_run_blocks(A, nseq, scratch, stream);
    const int units = (qk_mode == QK_PLAIN ? 0 : 2 * qk_heads) + (qk_mode == QKV_SILU ? heads : 0) + (channel ? heads : 0) +
                      ((decay_mode == DECAY_HEAD_TOKEN || delta) ? 1 : 0);
    if (units > 0) {
        const long long blocks = ((long long)T * units + 3) / 4;
        AP_CHECK_PDL_LAUNCH("linear_scan (rows made ready)",
                            ap_launch_pdl(la_prepare_kernel, dim3((unsigned)blocks), dim3(128), 0, stream, A));
    }
    const size_t smem = 2 * ((size_t)LA_CHUNK * ((cols + 3) / 4 * 4 + (channel ? 3 : 2) * (per * NP)) + 2 * LA_CHUNK) *
                        sizeof(float);
    void (*kern)(const LaScanArgs) = nullptr;
#define LA_PICK(P)                                                                                     \
    if (per == P)                                                                                      \
        kern = NP == 1 ? la_scan_kernel<P, 1> : NP == 2 ? la_scan_kernel<P, 2> : NP == 4 ? la_scan_kernel<P, 4> \
             : NP == 8 ? la_scan_kernel<P, 8> : NP == 16 ? la_scan_kernel<P, 16> : la_scan_kernel<P, 32>;
    LA_PICK(4) LA_PICK(8) LA_PICK(LA_PER_MAX)
#undef LA_PICK
    if (smem > 48 * 1024) {
        AP_REQUIRE(smem <= 200 * 1024, "linear_scan: keys of %d do not fit the staging buffers", D);
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        AP_REQUIRE(e == cudaSuccess, "linear_scan: cannot reserve %zu bytes of shared memory", smem);
    }
    AP_CHECK_PDL_LAUNCH("linear_scan", ap_launch_pdl(kern, grid, dim3(threads), smem, stream, A));
    return AP_OK;
}

// ---- exponential gates under a running maximum ------------------------------------------------
// A head's log input gate i = cap tanh((raw_i + b_i) / cap) and log forget gate f = logsigmoid(cap tanh((raw_f + b_f) / cap))
// may differ by many orders of magnitude from token to token, so the state is kept as exp(-m) times what the gates
// alone would make of it, with m a running maximum that a request carries from step to step (0 at its start):
//
//   m_t = max(f_t + m_{t-1}, i_t)     decay_t = exp(f_t + m_{t-1} - m_t)     write_t = exp(i_t - m_t)     floor_t = exp(-m_t)
//
// Decay and write replace the raw numbers in place (both are at most 1); floor is what 1 has become under the same scale.
// One CTA per (head, sequence).  A token is the map m -> max(f + m, i); maps compose (sums of f, a maximum), so a thread
// composes XG_PER tokens, the threads' maps meet in a scan, and each thread then walks its tokens from the m it starts at.
#define XG_PER 4
#define XG_THREADS 256

__device__ __forceinline__ float la_logsigmoid(float v) { return fminf(v, 0.f) - log1pf(expf(-fabsf(v))); }

__global__ void __launch_bounds__(XG_THREADS)
exp_gates_kernel(float* __restrict__ gi, float* __restrict__ gf, long long ld, const float* __restrict__ bi,
                 const float* __restrict__ bf, float cap, float* __restrict__ state, long long state_stride,
                 const int* __restrict__ seq_start, const int* __restrict__ positions,
                 const int* __restrict__ state_slots, float* __restrict__ floor_out, int heads) {
    __shared__ float sum_s[XG_THREADS / 32], top_s[XG_THREADS / 32];
    ap_pdl_trigger();
    ap_pdl_wait();
    const int h = blockIdx.x, s = blockIdx.y;
    const int a = seq_start[s], n = seq_start[s + 1] - a;
    if (n <= 0) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    float* mine = state + (size_t)state_slots[s] * state_stride + h;
    float m0 = positions[a] == 0 ? 0.f : *mine;
    const float add_i = bi ? bi[h] : 0.f, add_f = bf ? bf[h] : 0.f;
    for (int t0 = 0; t0 < n; t0 += XG_PER * blockDim.x) {
        float in[XG_PER], fo[XG_PER];
        float sum = 0.f, top = -INFINITY;                    // this thread's map: m -> max(sum + m, top)
#pragma unroll
        for (int j = 0; j < XG_PER; ++j) {
            const int t = t0 + threadIdx.x * XG_PER + j;
            in[j] = -INFINITY;                               // beyond the end: m stays
            fo[j] = 0.f;
            if (t < n) {
                in[j] = cap * tanhf((gi[(size_t)(a + t) * ld + h] + add_i) / cap);
                fo[j] = la_logsigmoid(cap * tanhf((gf[(size_t)(a + t) * ld + h] + add_f) / cap));
            }
            sum += fo[j];
            top = fmaxf(fo[j] + top, in[j]);
        }
        // scan over the lanes: the map of everything up to and with this thread
        float psum = sum, ptop = top;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float bs = __shfl_up_sync(0xffffffffu, psum, o), bt = __shfl_up_sync(0xffffffffu, ptop, o);
            if (lane >= o) {
                ptop = fmaxf(psum + bt, ptop);
                psum += bs;
            }
        }
        if (lane == 31) { sum_s[warp] = psum; top_s[warp] = ptop; }
        __syncthreads();
        float m = m0;                                        // the m before this warp's first token, and after the last
        for (int w = 0; w < nwarps; ++w) {
            if (w == warp) m = m0;
            m0 = fmaxf(sum_s[w] + m0, top_s[w]);
        }
        const float es = __shfl_up_sync(0xffffffffu, psum, 1), et = __shfl_up_sync(0xffffffffu, ptop, 1);
        if (lane > 0) m = fmaxf(es + m, et);
        float last = m;
#pragma unroll
        for (int j = 0; j < XG_PER; ++j) {
            const int t = t0 + threadIdx.x * XG_PER + j;
            if (t >= n) break;
            const float next = fmaxf(fo[j] + last, in[j]);
            gf[(size_t)(a + t) * ld + h] = expf(fo[j] + last - next);
            gi[(size_t)(a + t) * ld + h] = expf(in[j] - next);
            floor_out[(size_t)(a + t) * heads + h] = expf(-next);
            last = next;
        }
        __syncthreads();
    }
    if (threadIdx.x == 0) *mine = m0;
}

AP_EXPORT int ap_exp_gates(float* gi, float* gf, long long ld, const float* bi, const float* bf, float cap, float* state,
                           long long state_stride, const int* seq_start, const int* positions, const int* state_slots,
                           float* floor_out, int T, int nseq, int heads, cudaStream_t stream) {
    AP_REQUIRE(T >= 0 && nseq >= 0 && heads > 0 && ld >= heads && cap > 0.f && state_stride >= heads && gi && gf && state &&
               floor_out, "exp_gates: bad arguments heads=%d cap=%f", heads, (double)cap);
    AP_REQUIRE(nseq <= 65535, "exp_gates: %d sequences exceed the grid", nseq);
    if (T == 0 || nseq == 0) return AP_OK;
    int threads = 32;                                        // as many as the longest portion could fill
    while (threads < XG_THREADS && threads * XG_PER < T - nseq + 1) threads *= 2;
    AP_CHECK_PDL_LAUNCH("exp_gates", ap_launch_pdl(exp_gates_kernel, dim3((unsigned)heads, (unsigned)nseq), dim3((unsigned)threads), 0,
                                                   stream, gi, gf, ld, bi, bf, cap, state, state_stride, seq_start, positions,
                                                   state_slots, floor_out, heads));
    return AP_OK;
}

// ---- a head's read-out: RMS norm, gate, constant ------------------------------------------
// y: [T, ld_y] 32-bit, head h at column h * hs; gate: [T, ld_g] 32-bit raw, head h at column h * V; `threads` (a warp, or a
// CTA where the heads are long: a norm over all heads together is one head of their whole width) per (row, head).
// With `floor` [T, heads] (hs is V + 1 then) the head's numbers are first divided by max(|number V|, floor) + floor_eps.
// The weight has V numbers that the heads share, or (`own_weights`) V for each head.
#define GATE_SILU 0
#define GATE_SIGMOID 1
#define HNG_THREADS 128

template <typename TO, bool WHOLE_CTA>
__global__ void __launch_bounds__(HNG_THREADS)
head_norm_gate_kernel(const float* __restrict__ y, long long ld_y, int hs, const float* __restrict__ floor_in,
                      float floor_eps, const float* __restrict__ gate, long long ld_g, const float* __restrict__ w,
                      int own_weights, float eps, float out_scale, int act, TO* __restrict__ out, int T, int heads, int V) {
    __shared__ float scratch[32];
    ap_pdl_trigger();
    ap_pdl_wait();
    const long long unit = WHOLE_CTA ? (long long)blockIdx.x : (long long)blockIdx.x * (HNG_THREADS / 32) + (threadIdx.x >> 5);
    if (unit >= (long long)T * heads) return;                // (a whole CTA always has its unit)
    const int first = WHOLE_CTA ? threadIdx.x : (threadIdx.x & 31), stride = WHOLE_CTA ? HNG_THREADS : 32;
    const int t = (int)(unit / heads), h = (int)(unit % heads);
    const float* yr = y + (size_t)t * ld_y + (size_t)h * hs;
    const float* gr = gate + (size_t)t * ld_g + (size_t)h * V;
    if (w && own_weights) w += (size_t)h * V;
    const float pre = floor_in ? 1.0f / (fmaxf(fabsf(yr[V]), floor_in[(size_t)t * heads + h]) + floor_eps) : 1.0f;
    float ss = 0.f;
    for (int i = first; i < V; i += stride) {
        const float v = yr[i] * pre;
        ss = fmaf(v, v, ss);
    }
    ss = WHOLE_CTA ? ap_block_sum(ss, scratch) : ap_warp_sum(ss);
    const float inv = pre * (out_scale / sqrtf(ss / (float)V + eps));
    TO* o = out + ((size_t)t * heads + h) * V;
    for (int i = first; i < V; i += stride) {
        const float s = 1.0f / (1.0f + expf(-gr[i]));
        o[i] = ap_from_float<TO>(yr[i] * inv * (w ? w[i] : 1.0f) * (act == GATE_SILU ? gr[i] * s : s));
    }
}

AP_EXPORT int ap_head_norm_gate(const float* y, long long ld_y, int hs, const float* floor_in, float floor_eps,
                                const float* gate, long long ld_g, const float* w, int own_weights, float eps,
                                float out_scale, int act, void* out, int out_dtype, int T, int heads, int V,
                                cudaStream_t stream) {
    AP_REQUIRE(T >= 0 && heads > 0 && V > 0 && hs >= V + (floor_in ? 1 : 0) && ld_y >= (long long)heads * hs &&
               ld_g >= (long long)heads * V, "head_norm_gate: bad sizes heads=%d value=%d stride=%d", heads, V, hs);
    AP_REQUIRE(act == GATE_SILU || act == GATE_SIGMOID, "head_norm_gate: gate %d is not known", act);
    if (T == 0) return AP_OK;
    const bool whole = V > 256;
    const long long units = (long long)T * heads, per = whole ? 1 : HNG_THREADS / 32;
    const dim3 grid((unsigned)((units + per - 1) / per));
#define LAUNCH(TO, WHOLE)                                                                                           \
    AP_CHECK_PDL_LAUNCH("head_norm_gate", ap_launch_pdl(head_norm_gate_kernel<TO, WHOLE>, grid, dim3(HNG_THREADS), 0, stream, \
                                                        y, ld_y, hs, floor_in, floor_eps, gate, ld_g, w, own_weights, eps, \
                                                        out_scale, act, (TO*)out, T, heads, V))
    if (out_dtype == AP_F32) { if (whole) LAUNCH(float, true); else LAUNCH(float, false); }
    else if (out_dtype == AP_BF16) { if (whole) LAUNCH(bf16, true); else LAUNCH(bf16, false); }
    else AP_REQUIRE(false, "head_norm_gate: unknown dtype %d", out_dtype);
#undef LAUNCH
    return AP_OK;
}
