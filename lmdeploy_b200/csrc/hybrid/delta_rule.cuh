// Kernels of two linear recurrences over rotated or convolved queries and keys: retention (a fixed decay per head) and the gated delta
// rule (a decay per key channel and token, and a state that is corrected towards the token's value instead of only added to).
// Included by hybrid_ops.cu inside namespace b200h, after its helpers and gated_recurrence.cuh (load_vals / store_vals).
//
// Number formats: projections (T) are read once; rotated queries and keys, the convolutions' outputs, unit vectors, decays, step sizes,
// the recurrence and its state are float.

// One block per row: every head of q and k turns by the row's position (first 2 * rot.pairs dimensions), k is multiplied by k_scale.
// qk: float [n, 2 * heads * dim] = rotated q | rotated k.  Shared memory: 2 * rot.pairs floats of cos / sin.
template <typename T>
__global__ void __launch_bounds__(256) retention_prep_kernel(const T* __restrict__ q, const T* __restrict__ k, int64_t ld, int heads, int dim,
                                                            float k_scale, Rotary rot, const int* __restrict__ tok_pos, float* __restrict__ qk)
{
    extern __shared__ __align__(16) float rp_smem[];
    const int t = blockIdx.x, pos = tok_pos[t], HD = heads * dim, P = rot.pairs;
    float* cs = rp_smem;
    float* sn = rp_smem + P;
    for (int i = threadIdx.x; i < P; i += blockDim.x) {
        double sv, cv;
        sincos((double)pos * rot.freqs[i], &sv, &cv);
        cs[i] = (float)cv * rot.magnitude;
        sn[i] = (float)sv * rot.magnitude;
    }
    __syncthreads();
    float* out = qk + (size_t)t * 2 * HD;
    const int per = dim - P;                                  // one thread per turning pair or passing dimension
    for (int it = threadIdx.x; it < 2 * heads * per; it += blockDim.x) {
        const int h = it / per, i = it - h * per;             // h < heads: query heads, then key heads
        const bool key = h >= heads;
        const T* src = (key ? k : q) + (size_t)t * ld + (size_t)(key ? h - heads : h) * dim;
        float* dst = out + (size_t)h * dim;
        const float f = key ? k_scale : 1.0f;
        if (i < P) {
            const int a = rot.halves ? i : 2 * i, b = rot.halves ? i + P : 2 * i + 1;
            const float u = to_f(src[a]), v = to_f(src[b]);
            dst[a] = (u * cs[i] - v * sn[i]) * f;
            dst[b] = (v * cs[i] + u * sn[i]) * f;
        } else {
            dst[P + i] = to_f(src[P + i]) * f;
        }
    }
}

struct DeltaPrep {
    const float* w;           // [taps, channels]: the convolutions' weights, transposed; channels = q (kv_heads * dim) | k | v (heads * vdim)
    int taps;
    const float* state;       // the last taps - 1 projected rows, oldest first
    int64_t slot_stride;
    const int* tok_seq;
    const int* cu_q;
    const int* seq_slot;
    int n, heads, kv_heads, dim, vdim;
    float q_scale, unit_eps;
    float* qkv;               // [n, channels]
    float* kq;                // [n, kv_heads]: the scaled q . k of every head
    float* beta;              // [n, heads]
};

// A thread's V channels c .. c + V - 1 of ROWS consecutive rows from t0: silu(sum_j w[j, c] u[t - taps + 1 + j, c]).  Rows before the
// step's first row of a sequence come from its state.  TAPS >= taps: the leading weights are zero.
template <typename T, int TAPS, int ROWS, int V>
__device__ __forceinline__ void conv_silu_rows(const T* __restrict__ u, int64_t ld, const DeltaPrep& d, int channels, int c, int t0, int rows,
                                               float (&y)[ROWS][V])
{
    float wt[TAPS][V], win[TAPS][V], x[ROWS][V];
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
        if (r < rows) load_vals<V>(u + (size_t)(t0 + r) * ld + c, x[r]);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
        if (j >= TAPS - d.taps) load_vals<V>(d.w + (size_t)(j - (TAPS - d.taps)) * channels + c, wt[j]);
        else
#pragma unroll
            for (int e = 0; e < V; ++e) wt[j][e] = 0.f;
    }
    int seq = -1;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        if (r < rows) {
            const int s = d.tok_seq[t0 + r];
            if (s != seq) {                                   // this block's first row of the sequence: its predecessors from the step or the state
                seq = s;
                const int first = d.cu_q[s], local = t0 + r - first;
                const float* st = d.state + (int64_t)d.seq_slot[s] * d.slot_stride;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
                    const int src = local - (TAPS - 1) + j;
#pragma unroll
                    for (int e = 0; e < V; ++e) win[j][e] = 0.f;
                    if (j >= TAPS - d.taps) {
                        if (src >= 0) load_vals<V>(u + (size_t)(first + src) * ld + c, win[j]);
                        else
#pragma unroll
                            for (int e = 0; e < V; ++e) win[j][e] = st[(size_t)(src + d.taps - 1) * channels + c + e];
                    }
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) {
                win[TAPS - 1][e] = x[r][e];
                float acc = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc = fmaf(wt[j][e], win[j][e], acc);
                y[r][e] = silu_f(acc);
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) win[j][e] = win[j + 1][e];
            }
        }
    }
}

// What the gated delta rule reads, from the projection's columns u = q | k | v and b (one column per head):  every channel's convolution
// and silu; q and k of every head divided by sqrt(sum of squares + unit_eps), q times q_scale; their dot product; beta = sigmoid(b).
// grid (row groups, kv_heads + blocks of v channels), 128 threads: block y < kv_heads takes query head y and key head y (through shared
// memory [ROWS][2 * dim]), the others V * 128 channels of v each; block y == 0 also the row group's betas.
template <typename T, int TAPS, int ROWS, int V>
__global__ void __launch_bounds__(128) delta_prep_kernel(const T* __restrict__ u, const T* __restrict__ b, int64_t ld, DeltaPrep d)
{
    extern __shared__ __align__(16) float dp_smem[];
    const int t0 = blockIdx.x * ROWS, rows = min(ROWS, d.n - t0), g = blockIdx.y, D = d.dim, KD = d.kv_heads * D;
    const int channels = 2 * KD + d.heads * d.vdim;
    float y[ROWS][V];
    if (g >= d.kv_heads) {
        const int c = 2 * KD + ((g - d.kv_heads) * 128 + threadIdx.x) * V;
        if (c >= channels) return;
        conv_silu_rows<T, TAPS, ROWS, V>(u, ld, d, channels, c, t0, rows, y);
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
            if (r < rows) store_vals<V>(d.qkv + (size_t)(t0 + r) * channels + c, y[r]);
        return;
    }
    for (int i = threadIdx.x * V; i < 2 * D; i += 128 * V) {
        const int c = i < D ? g * D + i : KD + g * D + i - D;
        conv_silu_rows<T, TAPS, ROWS, V>(u, ld, d, channels, c, t0, rows, y);
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
            if (r < rows)
#pragma unroll
                for (int e = 0; e < V; ++e) dp_smem[r * 2 * D + i + e] = y[r][e];
    }
    if (g == 0)
        for (int i = threadIdx.x; i < rows * d.heads; i += 128) {
            const int r = i / d.heads, h = i - r * d.heads;
            d.beta[(size_t)(t0 + r) * d.heads + h] = sigmoid_f(to_f(b[(size_t)(t0 + r) * ld + h]));
        }
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int r = warp; r < rows; r += 4) {
        const float* q = dp_smem + r * 2 * D;
        const float* k = q + D;
        float sq = 0.f, sk = 0.f, qk = 0.f;
        for (int i = lane; i < D; i += 32) {
            sq = fmaf(q[i], q[i], sq);
            sk = fmaf(k[i], k[i], sk);
            qk = fmaf(q[i], k[i], qk);
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        qk = warp_sum(qk);
        const float rq = d.q_scale / sqrtf(sq + d.unit_eps), rk = 1.0f / sqrtf(sk + d.unit_eps);
        float* out = d.qkv + (size_t)(t0 + r) * channels + g * D;
        for (int i = lane; i < D; i += 32) {
            out[i] = q[i] * rq;
            out[KD + i] = k[i] * rk;
        }
        if (lane == 0) d.kq[(size_t)(t0 + r) * d.kv_heads + g] = qk * rq * rk;
    }
}

struct HeadScan {
    const float* q;           // row stride ld_qk; head h reads q / k head h / (heads / kv_heads)
    const float* k;
    int64_t ld_qk, ld_v;
    const float* decay;       // delta: [n, heads * dim]; retention: [heads]
    const float* beta;        // delta: [n, heads]
    const float* kq;          // delta: [n, kv_heads]
    float* state;             // [heads, vdim, dim] per slot
    int64_t slot_stride;
    const int* cu_q;
    const int* seq_slot;
    int heads, kv_heads, dim, vdim, aligned;      // aligned: 16-byte copies of q, k and decay rows
    float* out;               // [n, heads * vdim]
    // the convolution's state, advanced after the scan (delta; taps 1: none)
    const void* u;            // T, row stride ld_u
    int64_t ld_u;
    float* conv_state;
    int channels, taps;
};

__device__ __forceinline__ void copy_async4(float* dst, const float* src)
{
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async16(float* dst, const float* src)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// Per head, S a [dim, vdim] float matrix per sequence, columns independent:
//   retention:  S <- decay_h S + k v^T;  o = S^T q
//   delta:      S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q = (diag(g) S_old)^T q + u (k . q)
// The delta form takes both dot products of the decayed state in ONE pass and one round of shuffles; k . q comes from the preparation.
// Eight lanes own a value column: lane p keeps the state's entries 4 p + 32 e .. 4 p + 32 e + 3 in registers (e < NE) for NC columns, so a
// warp holds 4 NC columns and a row costs three shuffles per sum and no block barrier.  R rows of q, k and decays pass through shared
// memory at a time (asynchronous copies, double-buffered), v through registers (lane p of a column's eight holds row p's value).
// blockDim (32, 4); grid (heads * ceil(vdim / (16 NC)), batch).  Entries past dim hold zeros and stay zero.
template <typename T, bool DELTA, int NE, int NC>
__global__ void __launch_bounds__(128) head_scan_kernel(HeadScan g, const T* __restrict__ v_t, const float* __restrict__ v_f)
{
    constexpr int R = 8, DP = NE * 32, ARR = DELTA ? 3 : 2, STAGE = R * (ARR * DP + (DELTA ? 2 : 0));
    extern __shared__ __align__(16) float hs_smem[];
    const int lane = threadIdx.x, w = threadIdx.y, tid = w * 32 + lane, p = lane & 7;
    const int s = blockIdx.y, first = g.cu_q[s], last = g.cu_q[s + 1];
    if (first == last) return;                                // the whole block leaves
    const int groups = (g.vdim + 16 * NC - 1) / (16 * NC), h = blockIdx.x / groups, kh = h / (g.heads / g.kv_heads), D = g.dim;
    const int col = (blockIdx.x - h * groups) * 16 * NC + w * 4 * NC + (lane >> 3) * NC;
    float* sp = g.state + (int64_t)g.seq_slot[s] * g.slot_stride + (size_t)h * g.vdim * D;
    const bool vec = D % 4 == 0 && (reinterpret_cast<uintptr_t>(sp) & 15) == 0;
    float S[NC][NE * 4];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            const int d = 4 * p + 32 * e;
            const float* src = sp + (size_t)(col + c) * D + d;
            if (vec && col + c < g.vdim && d < D) {
                const float4 q4 = *reinterpret_cast<const float4*>(src);
                S[c][4 * e] = q4.x; S[c][4 * e + 1] = q4.y; S[c][4 * e + 2] = q4.z; S[c][4 * e + 3] = q4.w;
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i) S[c][4 * e + i] = (col + c < g.vdim && d + i < D) ? src[i] : 0.f;
            }
        }
    for (int i = tid; i < 2 * STAGE; i += 128) hs_smem[i] = 0.f;
    __syncthreads();
    const float lam = DELTA ? 0.f : g.decay[h];
    const size_t hd = (size_t)g.heads * D;
    // rows [t0, t0 + R) into stage buffer b
    auto stage_rows = [&](int t0, int b) {
        float* buf = hs_smem + b * STAGE;
        const int rows = min(R, last - t0), per = g.aligned ? D / 4 : D;
        for (int i = tid; i < rows * per; i += 128) {
            const int r = i / per, c = i - r * per;
            const size_t t = (size_t)(t0 + r);
            if (g.aligned) {
                copy_async16(buf + r * DP + 4 * c, g.q + t * g.ld_qk + (size_t)kh * D + 4 * c);
                copy_async16(buf + (R + r) * DP + 4 * c, g.k + t * g.ld_qk + (size_t)kh * D + 4 * c);
                if (DELTA) copy_async16(buf + (2 * R + r) * DP + 4 * c, g.decay + t * hd + (size_t)h * D + 4 * c);
            } else {
                copy_async4(buf + r * DP + c, g.q + t * g.ld_qk + (size_t)kh * D + c);
                copy_async4(buf + (R + r) * DP + c, g.k + t * g.ld_qk + (size_t)kh * D + c);
                if (DELTA) copy_async4(buf + (2 * R + r) * DP + c, g.decay + t * hd + (size_t)h * D + c);
            }
        }
        if (DELTA && tid < 2 * rows) {
            const int r = tid >> 1;
            if (tid & 1) copy_async4(buf + 3 * R * DP + R + r, g.kq + (size_t)(t0 + r) * g.kv_heads + kh);
            else copy_async4(buf + 3 * R * DP + r, g.beta + (size_t)(t0 + r) * g.heads + h);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float vn[NC];
    auto load_v = [&](int t0) {
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const size_t at = (size_t)(t0 + p) * g.ld_v + (size_t)h * g.vdim + col + c;
            vn[c] = (t0 + p < last && col + c < g.vdim) ? (DELTA ? v_f[at] : to_f(v_t[at])) : 0.f;
        }
    };
    stage_rows(first, 0);
    load_v(first);
    int b = 0;
    for (int t0 = first; t0 < last; t0 += R, b ^= 1) {
        float vc[NC], oc[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) { vc[c] = vn[c]; oc[c] = 0.f; }
        if (t0 + R < last) {
            stage_rows(t0 + R, b ^ 1);                       // in flight while the staged rows are computed
            load_v(t0 + R);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* buf = hs_smem + b * STAGE + 4 * p;
        const int rows = min(R, last - t0);
#pragma unroll 2
        for (int r = 0; r < rows; ++r) {
            float4 k4[NE];
            float a[NC][2], o[NC][2], vr[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                a[c][0] = a[c][1] = o[c][0] = o[c][1] = 0.f;
                vr[c] = __shfl_sync(0xffffffffu, vc[c], (lane & 24) | r);
            }
#pragma unroll
            for (int e = 0; e < NE; ++e) {
                const float4 q4 = *reinterpret_cast<const float4*>(buf + r * DP + 32 * e);
                k4[e] = *reinterpret_cast<const float4*>(buf + (R + r) * DP + 32 * e);
                if (DELTA) {
                    const float4 g4 = *reinterpret_cast<const float4*>(buf + (2 * R + r) * DP + 32 * e);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        float* st = S[c] + 4 * e;
                        st[0] *= g4.x; st[1] *= g4.y; st[2] *= g4.z; st[3] *= g4.w;
                        a[c][0] = fmaf(st[0], k4[e].x, a[c][0]); o[c][0] = fmaf(st[0], q4.x, o[c][0]);
                        a[c][1] = fmaf(st[1], k4[e].y, a[c][1]); o[c][1] = fmaf(st[1], q4.y, o[c][1]);
                        a[c][0] = fmaf(st[2], k4[e].z, a[c][0]); o[c][0] = fmaf(st[2], q4.z, o[c][0]);
                        a[c][1] = fmaf(st[3], k4[e].w, a[c][1]); o[c][1] = fmaf(st[3], q4.w, o[c][1]);
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        float* st = S[c] + 4 * e;
                        st[0] = fmaf(lam, st[0], k4[e].x * vr[c]); o[c][0] = fmaf(st[0], q4.x, o[c][0]);
                        st[1] = fmaf(lam, st[1], k4[e].y * vr[c]); o[c][1] = fmaf(st[1], q4.y, o[c][1]);
                        st[2] = fmaf(lam, st[2], k4[e].z * vr[c]); o[c][0] = fmaf(st[2], q4.z, o[c][0]);
                        st[3] = fmaf(lam, st[3], k4[e].w * vr[c]); o[c][1] = fmaf(st[3], q4.w, o[c][1]);
                    }
                }
            }
            const float beta = DELTA ? hs_smem[b * STAGE + 3 * R * DP + r] : 0.f, kq = DELTA ? hs_smem[b * STAGE + 3 * R * DP + R + r] : 0.f;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                float oo = o[c][0] + o[c][1], aa = a[c][0] + a[c][1];
#pragma unroll
                for (int m = 4; m > 0; m >>= 1) {
                    oo += __shfl_xor_sync(0xffffffffu, oo, m);
                    if (DELTA) aa += __shfl_xor_sync(0xffffffffu, aa, m);
                }
                if (DELTA) {
                    const float uu = beta * (vr[c] - aa);
                    oo = fmaf(uu, kq, oo);
#pragma unroll
                    for (int e = 0; e < NE; ++e) {
                        float* st = S[c] + 4 * e;
                        st[0] = fmaf(k4[e].x, uu, st[0]); st[1] = fmaf(k4[e].y, uu, st[1]);
                        st[2] = fmaf(k4[e].z, uu, st[2]); st[3] = fmaf(k4[e].w, uu, st[3]);
                    }
                }
                if (p == r) oc[c] = oo;
            }
        }
        if (t0 + p < last) {
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (col + c < g.vdim) g.out[((size_t)(t0 + p) * g.heads + h) * g.vdim + col + c] = oc[c];
        }
        __syncthreads();                                      // the buffer's readers are done before it is filled again
    }
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            const int d = 4 * p + 32 * e;
            float* dst = sp + (size_t)(col + c) * D + d;
            if (vec && col + c < g.vdim && d < D) {
                *reinterpret_cast<float4*>(dst) = make_float4(S[c][4 * e], S[c][4 * e + 1], S[c][4 * e + 2], S[c][4 * e + 3]);
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    if (col + c < g.vdim && d + i < D) dst[i] = S[c][4 * e + i];
            }
        }
    if (!DELTA || g.taps <= 1) return;
    // the last taps - 1 inputs of (old state ++ this step's rows); a thread reads all it needs of its channel and then writes
    float* cst = g.conv_state + (int64_t)g.seq_slot[s] * g.slot_stride;
    const T* u = reinterpret_cast<const T*>(g.u);
    const int cnt = last - first;
    for (int c = blockIdx.x * 128 + tid; c < g.channels; c += gridDim.x * 128) {
        float keep[B200H_MAX_TAPS];
#pragma unroll
        for (int i = 0; i < B200H_MAX_TAPS - 1; ++i) {
            if (i < g.taps - 1) {
                const int src = cnt + i - (g.taps - 1);
                keep[i] = src >= 0 ? to_f(u[(size_t)(first + src) * g.ld_u + c]) : cst[(size_t)(src + g.taps - 1) * g.channels + c];
            }
        }
#pragma unroll
        for (int i = 0; i < B200H_MAX_TAPS - 1; ++i)
            if (i < g.taps - 1) cst[(size_t)i * g.channels + c] = keep[i];
    }
}
