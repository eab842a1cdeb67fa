// Kernels of two linear recurrences over rotated or convolved queries and keys: retention (a fixed decay per head) and the gated delta
// rule (a decay per key channel and token, and a state that is corrected towards the token's value instead of only added to).
// Included by hybrid_ops.cu inside namespace b200h, after its helpers and gated_recurrence.cuh (load_vals / store_vals).
//
// Number formats: projections (T) are read once; rotated queries and keys, the convolutions' outputs, unit vectors, decays, step sizes,
// the recurrence and its state are float.

// z / (1 + exp(-z)) by the hardware's approximate exponential and division (relative error about 1e-6)
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// Two floats of one 64-bit register pair: a * b and a * b + c by sm_100's packed instructions
__device__ __forceinline__ unsigned long long pack2(float lo, float hi)
{
    unsigned long long r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float sum2(unsigned long long v)
{
    float lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
    return lo + hi;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b)
{
    unsigned long long r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c)
{
    unsigned long long r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

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
// step's first row of a sequence come from its state.  TAPS >= taps: the leading weights are zero.  The rows' loads and those of the
// rows before t0 are issued before the sequence is known; what belongs to another sequence is replaced by the state afterwards.
template <typename T, int TAPS, int ROWS, int V>
__device__ __forceinline__ void conv_silu_rows(const T* __restrict__ u, int64_t ld, const DeltaPrep& d, int channels, int c, int t0, int rows,
                                               float (&y)[ROWS][V])
{
    float wt[TAPS][V], win[TAPS][V], x[ROWS][V];
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
        if (r < rows) load_vals<V>(u + (size_t)(t0 + r) * ld + c, x[r]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
        const int src = t0 - (TAPS - 1) + j;
        if (j >= TAPS - d.taps && src >= 0) load_vals<V>(u + (size_t)src * ld + c, win[j]);
        else
#pragma unroll
            for (int e = 0; e < V; ++e) win[j][e] = 0.f;
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
        if (j >= TAPS - d.taps) load_vals<V>(d.w + (size_t)(j - (TAPS - d.taps)) * channels + c, wt[j]);
        else
#pragma unroll
            for (int e = 0; e < V; ++e) wt[j][e] = 0.f;
    }
    int s = d.tok_seq[t0], first = d.cu_q[s], end = d.cu_q[s + 1];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        if (r < rows) {
            if (t0 + r >= end) {                              // the next sequence that has rows in this step starts here
                s = d.tok_seq[t0 + r];
                first = t0 + r;
                end = d.cu_q[s + 1];
            }
            const int local = t0 + r - first;
            if (local < d.taps - 1 && (r == 0 || local == 0)) {
                const float* st = d.state + (int64_t)d.seq_slot[s] * d.slot_stride;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
                    const int src = local - (TAPS - 1) + j;
                    if (j >= TAPS - d.taps && src < 0)
#pragma unroll
                        for (int e = 0; e < V; ++e) win[j][e] = st[(size_t)(src + d.taps - 1) * channels + c + e];
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) {
                win[TAPS - 1][e] = x[r][e];
                float acc = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc = fmaf(wt[j][e], win[j][e], acc);
                y[r][e] = silu_fast(acc);
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) win[j][e] = win[j + 1][e];
            }
        }
    }
}

// What the gated delta rule reads, from the projection's columns u = q | k | v and b (one column per head):  every channel's convolution
// and silu; q and k of every head divided by sqrt(sum of squares + unit_eps), q times q_scale; their dot product; beta = sigmoid(b).
// grid (row groups, blocks of key heads + blocks of v channels), 128 threads: the first `head_blocks` blocks take `per` query heads and the
// same key heads each (through shared memory [ROWS][per][2 * dim]), the others V * 128 channels of v; block y == 0 also the row group's
// betas.
template <typename T, int TAPS, int ROWS, int V>
__global__ void __launch_bounds__(128, ROWS == 8 ? 6 : 1) delta_prep_kernel(const T* __restrict__ u, const T* __restrict__ b, int64_t ld, DeltaPrep d, int per,
                                                        int head_blocks)
{
    extern __shared__ __align__(16) float dp_smem[];
    const int t0 = blockIdx.x * ROWS, rows = min(ROWS, d.n - t0), D = d.dim, KD = d.kv_heads * D;
    const int channels = 2 * KD + d.heads * d.vdim;
    float y[ROWS][V];
    if ((int)blockIdx.y >= head_blocks) {
        const int c = 2 * KD + ((blockIdx.y - head_blocks) * 128 + threadIdx.x) * V;
        if (c >= channels) return;
        conv_silu_rows<T, TAPS, ROWS, V>(u, ld, d, channels, c, t0, rows, y);
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
            if (r < rows) store_vals<V>(d.qkv + (size_t)(t0 + r) * channels + c, y[r]);
        return;
    }
    const int g0 = blockIdx.y * per, heads = min(per, d.kv_heads - g0), span = heads * D;      // q channels g0 D .. + span, k the same
    for (int i = threadIdx.x * V; i < 2 * span; i += 128 * V) {
        const int key = i >= span, at = key ? i - span : i, g = at / D;
        conv_silu_rows<T, TAPS, ROWS, V>(u, ld, d, channels, key * KD + g0 * D + at, t0, rows, y);
        float* dst = dp_smem + g * 2 * D + key * D + at - g * D;
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
            if (r < rows) store_vals<V>(dst + (size_t)r * per * 2 * D, y[r]);
    }
    if (blockIdx.y == 0)
        for (int i = threadIdx.x; i < rows * d.heads; i += 128) {
            const int r = i / d.heads, h = i - r * d.heads;
            d.beta[(size_t)(t0 + r) * d.heads + h] = sigmoid_f(to_f(b[(size_t)(t0 + r) * ld + h]));
        }
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int it = warp; it < rows * heads; it += 4) {
        const int r = it / heads, g = it - r * heads;
        const float* q = dp_smem + (size_t)(r * per + g) * 2 * D;
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
        float* out = d.qkv + (size_t)(t0 + r) * channels + (size_t)(g0 + g) * D;
        for (int i = lane * V; i < D; i += 32 * V) {
            float a[V], c[V];
            load_vals<V>(q + i, a);
            load_vals<V>(k + i, c);
#pragma unroll
            for (int e = 0; e < V; ++e) { a[e] *= rq; c[e] *= rk; }
            store_vals<V>(out + i, a);
            store_vals<V>(out + KD + i, c);
        }
        if (lane == 0) d.kq[(size_t)(t0 + r) * d.kv_heads + g0 + g] = qk * rq * rk;
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

// Where the values come from: the projection (T, retention) or the convolution (float, delta)
template <typename T, bool DELTA> struct HeadScanValue {
    typedef T type;
    static __device__ __forceinline__ const T* pick(const T* t, const float*) { return t; }
};
template <typename T> struct HeadScanValue<T, true> {
    typedef float type;
    static __device__ __forceinline__ const float* pick(const T*, const float* f) { return f; }
};

// part[r] of eight neighbouring lanes -> the sum over the lanes of part[p] at lane p
__device__ __forceinline__ float scatter_sum8(float (&part)[8], int p)
{
#pragma unroll
    for (int m = 4; m > 0; m >>= 1) {
        const bool upper = p & m;
#pragma unroll
        for (int i = 0; i < m; ++i) {
            const float give = upper ? part[i] : part[i + m], keep = upper ? part[i + m] : part[i];
            part[i] = keep + __shfl_xor_sync(0xffffffffu, give, m);
        }
    }
    return part[0];
}

// Per head, S a [dim, vdim] float matrix per sequence, columns independent:
//   retention:  S <- decay_h S + k v^T;  o = S^T q
//   delta:      S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q = (diag(g) S_old)^T q + u (k . q)
// The delta form takes both dot products of the decayed state in ONE pass; k . q comes from the preparation.
// Eight lanes own a value column: lane p keeps the state's entries 4 p + 32 e .. 4 p + 32 e + 3 in registers (e < NE) for NC columns, so a
// warp holds 4 NC columns and rows meet no block barrier.  R = 8 rows of q, k and decays pass through shared memory at a time
// (asynchronous copies, double-buffered), v through registers (lane p of a column's eight holds row p's value).  S^T k is summed over
// the eight lanes row by row (the next row needs it); the R rows' partial S^T q are kept and summed together, seven shuffles that leave
// row p's sum with lane p, which stores it.
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
    unsigned long long S[NC][NE * 2];                         // pairs of neighbouring entries
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int e = 0; e < NE; ++e) {
            S[c][2 * e] = S[c][2 * e + 1] = 0ull;
            const int d = 4 * p + 32 * e;
            if (vec && col + c < g.vdim && d < D) {           // all of a thread's reads are in flight together
                const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(sp + (size_t)(col + c) * D + d);
                S[c][2 * e] = q4.x;
                S[c][2 * e + 1] = q4.y;
            }
        }
    if (!vec) {
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int e = 0; e < 2 * NE; ++e) {
                const int d = 4 * p + 32 * (e / 2) + 2 * (e & 1);
                const float* src = sp + (size_t)(col + c) * D + d;
                const bool live = col + c < g.vdim;
                S[c][e] = pack2(live && d < D ? src[0] : 0.f, live && d + 1 < D ? src[1] : 0.f);
            }
    }
    for (int i = tid; i < 2 * STAGE; i += 128) hs_smem[i] = 0.f;
    __syncthreads();
    const unsigned long long lam = DELTA ? 0ull : pack2(g.decay[h], g.decay[h]);
    const size_t hd = (size_t)g.heads * D;
    // this thread's 16-byte pieces of a stage: row and first column
    constexpr int PIECES = (R * NE * 8 + 127) / 128;
    int pr[PIECES], pc[PIECES];
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
        pr[i] = (tid + i * 128) / (D / 4 > 0 ? D / 4 : 1);
        pc[i] = 4 * (tid + i * 128 - pr[i] * (D / 4));
    }
    const float* q_at = g.q + (size_t)kh * D;
    const float* k_at = g.k + (size_t)kh * D;
    const float* d_at = DELTA ? g.decay + (size_t)h * D : nullptr;
    // rows [t0, t0 + R) into stage buffer b
    auto stage_rows = [&](int t0, int b) {
        float* buf = hs_smem + b * STAGE;
        const int rows = min(R, last - t0);
        if (g.aligned) {
#pragma unroll
            for (int i = 0; i < PIECES; ++i) {
                if (pr[i] < rows) {
                    const size_t t = (size_t)(t0 + pr[i]);
                    float* dst = buf + pr[i] * DP + pc[i];
                    copy_async16(dst, q_at + t * g.ld_qk + pc[i]);
                    copy_async16(dst + R * DP, k_at + t * g.ld_qk + pc[i]);
                    if (DELTA) copy_async16(dst + 2 * R * DP, d_at + t * hd + pc[i]);
                }
            }
        } else {
            for (int i = tid; i < rows * D; i += 128) {
                const int r = i / D, c = i - r * D;
                const size_t t = (size_t)(t0 + r);
                copy_async4(buf + r * DP + c, q_at + t * g.ld_qk + c);
                copy_async4(buf + (R + r) * DP + c, k_at + t * g.ld_qk + c);
                if (DELTA) copy_async4(buf + (2 * R + r) * DP + c, d_at + t * hd + c);
            }
        }
        if (DELTA && tid < 2 * rows) {
            const int r = tid >> 1;
            if (tid & 1) copy_async4(buf + 3 * R * DP + tid, g.kq + (size_t)(t0 + r) * g.kv_heads + kh);
            else copy_async4(buf + 3 * R * DP + tid, g.beta + (size_t)(t0 + r) * g.heads + h);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    typedef typename HeadScanValue<T, DELTA>::type TV;
    const TV* v = HeadScanValue<T, DELTA>::pick(v_t, v_f);
    TV vn[NC];                                                // as stored: a conversion here would wait for the load
    auto load_v = [&](int t0) {
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const size_t at = (size_t)(t0 + p) * g.ld_v + (size_t)h * g.vdim + col + c;
            vn[c] = (t0 + p < last && col + c < g.vdim) ? v[at] : from_f<TV>(0.f);
        }
    };
    stage_rows(first, 0);
    load_v(first);
    int b = 0;
    for (int t0 = first; t0 < last; t0 += R, b ^= 1) {
        float vc[NC], oc[NC], part[NC][R];
#pragma unroll
        for (int c = 0; c < NC; ++c) { vc[c] = to_f(vn[c]); oc[c] = 0.f; }
        if (t0 + R < last) {
            stage_rows(t0 + R, b ^ 1);                       // in flight while the staged rows are computed
            load_v(t0 + R);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* buf = hs_smem + b * STAGE + 4 * p;
        const float* row_nums = hs_smem + b * STAGE + 3 * R * DP;         // delta: (beta, k . q) of every row
        const int rows = min(R, last - t0);
        auto row = [&](int r) {
            unsigned long long k2[NE * 2], a[NC][2], o[NC][2];
            float vr[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                a[c][0] = a[c][1] = o[c][0] = o[c][1] = 0ull;
                vr[c] = __shfl_sync(0xffffffffu, vc[c], (lane & 24) | r);
            }
#pragma unroll
            for (int e = 0; e < NE; ++e) {
                const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(buf + r * DP + 32 * e);
                const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(buf + (R + r) * DP + 32 * e);
                k2[2 * e] = k4.x;
                k2[2 * e + 1] = k4.y;
                if (DELTA) {
                    const ulonglong2 g4 = *reinterpret_cast<const ulonglong2*>(buf + (2 * R + r) * DP + 32 * e);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        S[c][2 * e] = mul2(S[c][2 * e], g4.x);
                        S[c][2 * e + 1] = mul2(S[c][2 * e + 1], g4.y);
                        a[c][0] = fma2(S[c][2 * e], k4.x, a[c][0]);
                        a[c][1] = fma2(S[c][2 * e + 1], k4.y, a[c][1]);
                        o[c][0] = fma2(S[c][2 * e], q4.x, o[c][0]);
                        o[c][1] = fma2(S[c][2 * e + 1], q4.y, o[c][1]);
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        const unsigned long long v2 = pack2(vr[c], vr[c]);
                        S[c][2 * e] = fma2(lam, S[c][2 * e], mul2(k4.x, v2));
                        S[c][2 * e + 1] = fma2(lam, S[c][2 * e + 1], mul2(k4.y, v2));
                        o[c][0] = fma2(S[c][2 * e], q4.x, o[c][0]);
                        o[c][1] = fma2(S[c][2 * e + 1], q4.y, o[c][1]);
                    }
                }
            }
            const float2 nums = DELTA ? *reinterpret_cast<const float2*>(row_nums + 2 * r) : make_float2(0.f, 0.f);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                part[c][r] = sum2(o[c][0]) + sum2(o[c][1]);
                if (DELTA) {
                    float aa = sum2(a[c][0]) + sum2(a[c][1]);
#pragma unroll
                    for (int m = 4; m > 0; m >>= 1) aa += __shfl_xor_sync(0xffffffffu, aa, m);
                    const float uu = nums.x * (vr[c] - aa);
                    if (p == r) oc[c] = uu * nums.y;
                    const unsigned long long u2 = pack2(uu, uu);
#pragma unroll
                    for (int e = 0; e < 2 * NE; ++e) S[c][e] = fma2(k2[e], u2, S[c][e]);
                }
            }
        };
        if (rows == R) {                                      // a whole stage: no branch between its rows
#pragma unroll
            for (int r = 0; r < R; ++r) row(r);
        } else {
#pragma unroll
            for (int r = 0; r < R; ++r) {
                if (r < rows) row(r);
                else
#pragma unroll
                    for (int c = 0; c < NC; ++c) part[c][r] = 0.f;
            }
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) oc[c] += scatter_sum8(part[c], p);
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
                *reinterpret_cast<ulonglong2*>(dst) = make_ulonglong2(S[c][2 * e], S[c][2 * e + 1]);
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    if (col + c < g.vdim && d + i < D) dst[i] = __uint_as_float((unsigned)(S[c][2 * e + i / 2] >> (32 * (i & 1))));
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
