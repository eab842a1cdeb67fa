// Kernels of blocks that norm what a sublayer gives as well as what it reads: the join of a sublayer's output into the stream
// (with the two sides of a paired mixer normed and averaged first) fused with the next norm, and the gated activation between a dense
// feed-forward's stacked gate | up product and its down product.
// Included by hybrid_ops.cu inside namespace b200h, after its helpers.

// Sum of two values over the block with one pass of barriers; every thread gets both.  red: 64 floats.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red)
{
    a = warp_sum(a);
    b = warp_sum(b);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    __syncthreads();
    if (lane == 0) { red[2 * warp] = a; red[2 * warp + 1] = b; }
    __syncthreads();
    float2 r = make_float2(0.f, 0.f);
    for (int i = 0; i < nw; ++i) { r.x += red[2 * i]; r.y += red[2 * i + 1]; }
    return r;
}

// V (1 or 4) consecutive values as float / back
template <int V> __device__ __forceinline__ void load_row(const float* p, float (&o)[V])
{
    if (V == 4) { const float4 v = *reinterpret_cast<const float4*>(p); o[0] = v.x; o[1 % V] = v.y; o[2 % V] = v.z; o[3 % V] = v.w; } else o[0] = p[0];
}
template <int V> __device__ __forceinline__ void load_row(const bf16* p, float (&o)[V])
{
    if (V == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        o[0] = __uint_as_float(raw.x << 16); o[1 % V] = __uint_as_float(raw.x & 0xffff0000u);
        o[2 % V] = __uint_as_float(raw.y << 16); o[3 % V] = __uint_as_float(raw.y & 0xffff0000u);
    } else o[0] = to_f(p[0]);
}
template <int V> __device__ __forceinline__ void store_row(float* p, const float (&v)[V])
{
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]); else p[0] = v[0];
}
template <int V> __device__ __forceinline__ void store_row(bf16* p, const float (&v)[V])
{
    if (V == 4) {
        __nv_bfloat162 q[2] = {__floats2bfloat162_rn(v[0], v[1 % V]), __floats2bfloat162_rn(v[2 % V], v[3 % V])};
        *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(q);
    } else p[0] = from_f<bf16>(v[0]);
}

// One block per row t.  y = branch_scale * (rms(left) wl + rms(right) wr) + m + sum_p ff[p];  x += rms(y) * w_post;  then
// hf = rms(x) * w_next (float) and h the same as T.  Every input row is read once: the row passes from one norm to the next through
// shared memory (width floats, twice that with two sides), where a thread only meets its own values.
template <typename T, int V>
__global__ void __launch_bounds__(256) normed_residual_norm_kernel(float* __restrict__ x, const T* __restrict__ left, const T* __restrict__ right,
                                                                  const float* __restrict__ wl, const float* __restrict__ wr, float branch_scale,
                                                                  const T* __restrict__ m, const float* __restrict__ ff, int parts,
                                                                  const float* __restrict__ w_post, const float* __restrict__ w_next, int width,
                                                                  float eps, T* __restrict__ h, float* __restrict__ hf)
{
    extern __shared__ __align__(16) float nrn_smem[];
    __shared__ float red[64];
    float* ya = nrn_smem;
    float* yb = nrn_smem + width;
    const size_t base = (size_t)blockIdx.x * width;
    const bool joins = left || m || ff;
    float rl = 0.f, rr = 0.f;
    if (left) {
        float sl = 0.f, sr = 0.f;
        for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
            float a[V], b[V];
            load_row<V>(left + base + i, a);
            load_row<V>(right + base + i, b);
#pragma unroll
            for (int e = 0; e < V; ++e) { sl = fmaf(a[e], a[e], sl); sr = fmaf(b[e], b[e], sr); }
            store_row<V>(ya + i, a);
            store_row<V>(yb + i, b);
        }
        const float2 s2 = block_sum2(sl, sr, red);
        rl = branch_scale / sqrtf(s2.x / (float)width + eps);
        rr = branch_scale / sqrtf(s2.y / (float)width + eps);
    }
    float post = 0.f;
    if (joins) {
        float ss = 0.f;
        for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
            float y[V];
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = 0.f;
            if (left) {
                float a[V], b[V], u[V], v[V];
                load_row<V>(ya + i, a);
                load_row<V>(yb + i, b);
                load_row<V>(wl + i, u);
                load_row<V>(wr + i, v);
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] = a[e] * rl * u[e] + b[e] * rr * v[e];
            }
            if (m) {
                float a[V];
                load_row<V>(m + base + i, a);
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] += a[e];
            }
            for (int p = 0; p < parts; ++p) {
                float a[V];
                load_row<V>(ff + ((size_t)blockIdx.x * parts + p) * width + i, a);
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] += a[e];
            }
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(y[e], y[e], ss);
            store_row<V>(ya + i, y);
        }
        post = 1.0f / sqrtf(block_sum2(ss, 0.f, red).x / (float)width + eps);
    }
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V];
        load_row<V>(x + base + i, v);
        if (joins) {
            float y[V], wp[V];
            load_row<V>(ya + i, y);
            load_row<V>(w_post + i, wp);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] += y[e] * post * wp[e];
            store_row<V>(x + base + i, v);
        }
        store_row<V>(ya + i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
    }
    if (!w_next) return;
    const float r = 1.0f / sqrtf(block_sum2(ss, 0.f, red).x / (float)width + eps);
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V], wn[V];
        load_row<V>(ya + i, v);
        load_row<V>(w_next + i, wn);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = v[e] * r * wn[e];
        if (h) store_row<V>(h + base + i, v);
        if (hf) store_row<V>(hf + base + i, v);
    }
}

// out[t, i] = act(gu[t, i]) * gu[t, cols + i]: gu T [n, 2 * cols]; act silu, or GELU: the tanh form of gelu.  V values per thread.
template <typename T, int V, bool GELU>
__global__ void __launch_bounds__(256) gate_mul_rows_kernel(const T* __restrict__ gu, int cols, int64_t count, T* __restrict__ out)
{
    const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= count) return;
    const int64_t t = i / cols;
    const int c = (int)(i - t * cols);
    const T* row = gu + t * 2 * cols;
    float a[V], b[V];
    load_row<V>(row + c, a);
    load_row<V>(row + cols + c, b);
#pragma unroll
    for (int e = 0; e < V; ++e) a[e] = (GELU ? gelu_tanh_f(a[e]) : silu_f(a[e])) * b[e];
    store_row<V>(out + i, a);
}
