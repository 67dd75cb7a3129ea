// fq3_seq.cuh — sequence-model ops of the op-list interpreter (include/fq3_codec.h, kinds 12-33): the pieces a decoder-only
// language model with a 32-bit residual stream is lowered to.  Included by fq3_codec.cu inside its anonymous namespace.
//
// What is 32-bit here whatever the weights' type: norms, softmax scores and weights, router, recurrent state and everything that
// enters the recurrence, the residual sum.  Products take bf16 (or f32) operands and accumulate in f32.

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// sum over a block of up to 1024 threads; every thread gets the result.  red = 32 floats of shared memory.
__device__ __forceinline__ float seq_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = l < nw ? red[l] : 0.f;
  return warp_sum(t);
}

// ---------------------------------------------------------------------------------------------------------------------------
// Generic tiled product on the CUDA cores, f32 accumulate: any M, N, K and leading dimensions.  It is the true-32-bit path, the
// path of shapes the tensor-core kernels do not take, the block-diagonal product (grid.z = block) and the grouped product of a
// mixture of experts (row tiles resolved against the segment starts on the device).
// ---------------------------------------------------------------------------------------------------------------------------
struct SeqGemm {
  const void* A; const void* B; const float* bias; void* C;
  int M, N, K, lda, ldb, ldc, flags;
  int a_mod, a_zstride, c_zstride; long long b_zstride;   // grid.z: A columns (z % a_mod) * a_zstride, B + z * b_zstride, C columns z * c_zstride
  const int* seg; const int* rows; int E; long long b_estride;
  // FQ3C_SWIGLU: the weight rows alternate (gate_n, up_n), so columns (2n, 2n + 1) of the product are one gated unit and the output
  // is C[r, n] = silu(w gate) * (w up) (FQ3C_GELU_TANH: gelu_tanh(w gate) * (w up)), N / 2 columns wide.  w = 1, or rs_w[r], or (rs_pos given: a router's choices) the weight
  // rs_w[m, j] of the choice j of token m = rows[r] whose sorted position rs_pos[m, j] is r.
  const float* rs_w; const int* rs_pos; int rs_top;
};
__device__ __forceinline__ float sg_row_scale(const SeqGemm& g, const int r) {
  if (!g.rs_w) return 1.f;
  if (!g.rs_pos) return g.rs_w[r];
  const int m = g.rows ? g.rows[r] : r;
  for (int j = 0; j < g.rs_top; ++j)
    if (g.rs_pos[(size_t)m * g.rs_top + j] == r) return g.rs_w[(size_t)m * g.rs_top + j];
  return 1.f;
}
__device__ __forceinline__ void sg_store_glu(const SeqGemm& g, const int r, const int ccol, const int n_even, const float gate, const float up,
                                             const float w) {
  const float v = glu_f(g.flags, w * gate, w * up);
  const size_t ci = (size_t)r * g.ldc + ccol + (n_even >> 1);
  if (g.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(g.C)[ci] = v;
  else reinterpret_cast<bf16*>(g.C)[ci] = __float2bfloat16_rn(v);
}
constexpr int SG_BM = 64, SG_BN = 64, SG_BK = 16;

template <typename TA, typename TB>
__global__ void __launch_bounds__(256) fq3s_gemm_kernel(const SeqGemm g) {
  __shared__ float As[SG_BK][SG_BM + 4];
  __shared__ float Bs[SG_BK][SG_BN + 4];
  const int tid = threadIdx.x, z = blockIdx.z;
  int row0, row_end;
  const TB* Bp = reinterpret_cast<const TB*>(g.B) + (size_t)z * g.b_zstride;
  if (g.seg) {
    int t = blockIdx.y, e = 0;
    row0 = -1; row_end = 0;
    for (; e < g.E; ++e) {
      const int s0 = g.seg[e], s1 = g.seg[e + 1];
      const int nt = (s1 - s0 + SG_BM - 1) / SG_BM;
      if (t < nt) { row0 = s0 + t * SG_BM; row_end = s1; break; }
      t -= nt;
    }
    if (row0 < 0) return;
    Bp += (size_t)e * g.b_estride;
  } else {
    row0 = blockIdx.y * SG_BM; row_end = g.M;
  }
  const int col0 = blockIdx.x * SG_BN;
  const TA* Ap = reinterpret_cast<const TA*>(g.A) + (size_t)(z % g.a_mod) * g.a_zstride;
  // loader roles: 4 consecutive k of one row per thread
  const int lr = tid >> 2, lk = (tid & 3) * 4;
  const int ar = row0 + lr;
  long long a_row = -1;
  if (ar < row_end) a_row = g.rows ? g.rows[ar] : ar;
  const int bn = col0 + lr;
  const int ty = tid >> 4, tx = tid & 15;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < g.K; k0 += SG_BK) {
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int k = k0 + lk + q;
      As[lk + q][lr] = (a_row >= 0 && k < g.K) ? ldf<TA>(Ap + (size_t)a_row * g.lda + k) : 0.f;
      Bs[lk + q][lr] = (bn < g.N && k < g.K) ? ldf<TB>(Bp + (size_t)bn * g.ldb + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_BK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&As[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Bs[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
  const int ccol = z * g.c_zstride;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = row0 + ty * 4 + i;
    if (r >= row_end) continue;
    if (g.flags & FQ3C_SWIGLU) {
      const float w = sg_row_scale(g, r);
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        const int n = col0 + tx * 4 + j;
        if (n + 1 < g.N) sg_store_glu(g, r, ccol, n, acc[i][j], acc[i][j + 1], w);
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = col0 + tx * 4 + j;
      if (n >= g.N) continue;
      float v = acc[i][j];
      if (g.flags & FQ3C_BIAS) v += g.bias[ccol + n];
      if (g.flags & FQ3C_GELU) v = gelu_f(v);
      if (g.flags & FQ3C_GELU_TANH) v = gelu_tanh_f(v);
      if (g.flags & FQ3C_SIGMOID) v = sigmoid_f(v);
      if (g.flags & FQ3C_RELU2) { v = fmaxf(v, 0.f); v *= v; }
      const size_t ci = (size_t)r * g.ldc + ccol + n;
      if (g.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(g.C)[ci] = v;
      else reinterpret_cast<bf16*>(g.C)[ci] = __float2bfloat16_rn(v);
    }
  }
}

// Same interface on the bf16 tensor cores (mma.sync m16n8k16, f32 accumulate) for bf16 weights: the block-diagonal and grouped
// products of real-size layers.  64 x 64 x 32 tiles, four warps, each a 32 x 32 quadrant.  A may be f32 (rounded to bf16 as it is
// staged, which is what a bf16 product does to its operand) and rows may be gathered.  Every thread stages 16 consecutive k of
// one A row and one B row: with 16-byte loads where the operand's rows allow it (`vec`), element by element otherwise and at
// the ragged end of K; the next tile's values are fetched into registers before the current tile's MMAs run.
template <typename T>
__device__ __forceinline__ void sg_fetch16(const T* p, const bool vec, const int kleft, uint4 (&r)[2]) {
  // p: the row's element at this thread's first k, or nullptr for a row outside the tile; kleft: valid elements from there on
  if (p == nullptr || kleft <= 0) { r[0] = make_uint4(0u, 0u, 0u, 0u); r[1] = r[0]; return; }
  if (vec && kleft >= 16) {
    if (sizeof(T) == 2) {
      r[0] = *reinterpret_cast<const uint4*>(p);
      r[1] = *reinterpret_cast<const uint4*>(p + 8);
    } else {
      uint32_t u[8];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float4 f = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + 4 * q);
        const __nv_bfloat162 lo = __floats2bfloat162_rn(f.x, f.y), hi = __floats2bfloat162_rn(f.z, f.w);
        u[2 * q] = *reinterpret_cast<const uint32_t*>(&lo);
        u[2 * q + 1] = *reinterpret_cast<const uint32_t*>(&hi);
      }
      r[0] = make_uint4(u[0], u[1], u[2], u[3]);
      r[1] = make_uint4(u[4], u[5], u[6], u[7]);
    }
    return;
  }
  uint32_t u[8];
#pragma unroll
  for (int q = 0; q < 8; ++q) {
    const float a = 2 * q < kleft ? ldf<T>(p + 2 * q) : 0.f, b = 2 * q + 1 < kleft ? ldf<T>(p + 2 * q + 1) : 0.f;
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    u[q] = *reinterpret_cast<const uint32_t*>(&h);
  }
  r[0] = make_uint4(u[0], u[1], u[2], u[3]);
  r[1] = make_uint4(u[4], u[5], u[6], u[7]);
}
template <typename TA, bool GLU = false>      // GLU: the gated-unit epilogue (a variant of its own, so that the plain one compiles as it always did)
__global__ void __launch_bounds__(128) fq3s_gemm_mma_kernel(const SeqGemm g) {
  constexpr int LD = 32 + 8;
  __shared__ __align__(16) bf16 As[64 * LD];
  __shared__ __align__(16) bf16 Bs[64 * LD];
  const int tid = threadIdx.x, z = blockIdx.z, warp = tid >> 5, lane = tid & 31;
  int row0, row_end;
  const bf16* Bp = reinterpret_cast<const bf16*>(g.B) + (size_t)z * g.b_zstride;
  if (g.seg) {
    int t = blockIdx.y, e = 0;
    row0 = -1; row_end = 0;
    for (; e < g.E; ++e) {
      const int s0 = g.seg[e], s1 = g.seg[e + 1];
      const int nt = (s1 - s0 + 63) / 64;
      if (t < nt) { row0 = s0 + t * 64; row_end = s1; break; }
      t -= nt;
    }
    if (row0 < 0) return;
    Bp += (size_t)e * g.b_estride;
  } else {
    row0 = blockIdx.y * 64; row_end = g.M;
  }
  const int col0 = blockIdx.x * 64;
  const TA* Ap = reinterpret_cast<const TA*>(g.A) + (size_t)(z % g.a_mod) * g.a_zstride;
  // loaders: thread -> (row = tid / 2, 16 consecutive k)
  const int lr = tid >> 1, lk = (tid & 1) * 16;
  const int ar = row0 + lr;
  const TA* a_ptr = nullptr;
  if (ar < row_end) a_ptr = Ap + (size_t)(g.rows ? g.rows[ar] : ar) * g.lda + lk;
  const int bn = col0 + lr;
  const bf16* b_ptr = bn < g.N ? Bp + (size_t)bn * g.ldb + lk : nullptr;
  constexpr int AV = 16 / sizeof(TA);   // elements per 16 bytes
  const bool vec_a = (g.lda % AV == 0) && ((reinterpret_cast<uintptr_t>(Ap) & 15) == 0);
  const bool vec_b = (g.ldb % 8 == 0) && ((reinterpret_cast<uintptr_t>(Bp) & 15) == 0);
  const int wm = (warp >> 1) * 32, wn = (warp & 1) * 32;
  float acc[2][4][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) acc[i][j][q] = 0.f;
  uint4 ra[2], rb[2];
  sg_fetch16<TA>(a_ptr, vec_a, g.K - lk, ra);
  sg_fetch16<bf16>(b_ptr, vec_b, g.K - lk, rb);
  for (int k0 = 0; k0 < g.K; k0 += 32) {
    *reinterpret_cast<uint4*>(&As[lr * LD + lk]) = ra[0];
    *reinterpret_cast<uint4*>(&As[lr * LD + lk + 8]) = ra[1];
    *reinterpret_cast<uint4*>(&Bs[lr * LD + lk]) = rb[0];
    *reinterpret_cast<uint4*>(&Bs[lr * LD + lk + 8]) = rb[1];
    __syncthreads();
    if (k0 + 32 < g.K) {
      sg_fetch16<TA>(a_ptr ? a_ptr + k0 + 32 : nullptr, vec_a, g.K - (k0 + 32 + lk), ra);
      sg_fetch16<bf16>(b_ptr ? b_ptr + k0 + 32 : nullptr, vec_b, g.K - (k0 + 32 + lk), rb);
    }
#pragma unroll
    for (int kk = 0; kk < 32; kk += 16) {
      uint32_t a[2][4], b[4][2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = wm + i * 16 + (lane >> 2), c = kk + (lane & 3) * 2;
        a[i][0] = *reinterpret_cast<const uint32_t*>(&As[r * LD + c]);
        a[i][1] = *reinterpret_cast<const uint32_t*>(&As[(r + 8) * LD + c]);
        a[i][2] = *reinterpret_cast<const uint32_t*>(&As[r * LD + c + 8]);
        a[i][3] = *reinterpret_cast<const uint32_t*>(&As[(r + 8) * LD + c + 8]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = wn + j * 8 + (lane >> 2), c = kk + (lane & 3) * 2;
        b[j][0] = *reinterpret_cast<const uint32_t*>(&Bs[n * LD + c]);
        b[j][1] = *reinterpret_cast<const uint32_t*>(&Bs[n * LD + c + 8]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) mma16816(acc[i][j], a[i], b[j][0], b[j][1]);
    }
    __syncthreads();
  }
  const int ccol = z * g.c_zstride;
  if constexpr (GLU) {      // an accumulator pair (q, q + 1) is one gated unit
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int q = 0; q < 4; q += 2) {
        const int r = row0 + wm + i * 16 + (lane >> 2) + (q >> 1) * 8;
        if (r >= row_end) continue;
        const float w = sg_row_scale(g, r);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int n = col0 + wn + j * 8 + (lane & 3) * 2;
          if (n + 1 < g.N) sg_store_glu(g, r, ccol, n, acc[i][j][q], acc[i][j][q + 1], w);
        }
      }
    return;
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int r = row0 + wm + i * 16 + (lane >> 2) + (q >> 1) * 8;
        const int n = col0 + wn + j * 8 + (lane & 3) * 2 + (q & 1);
        if (r >= row_end || n >= g.N) continue;
        float v = acc[i][j][q];
        if (g.flags & FQ3C_BIAS) v += g.bias[ccol + n];
        if (g.flags & FQ3C_GELU) v = gelu_f(v);
        if (g.flags & FQ3C_GELU_TANH) v = gelu_tanh_f(v);
        if (g.flags & FQ3C_SIGMOID) v = sigmoid_f(v);
        if (g.flags & FQ3C_RELU2) { v = fmaxf(v, 0.f); v *= v; }
        const size_t ci = (size_t)r * g.ldc + ccol + n;
        if (g.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(g.C)[ci] = v;
        else reinterpret_cast<bf16*>(g.C)[ci] = __float2bfloat16_rn(v);
      }
}

// The same product for tall operands (hundreds of rows per block / expert): 128 x 128 x 32 tiles, eight warps of 64 x 32 each, fragments
// by ldmatrix.  Halves the operand traffic per output of the 64 x 64 kernel and runs 16 MMAs per warp between two barriers.
template <typename TA, bool GLU = false>
__global__ void __launch_bounds__(256) fq3s_gemm_mma128_kernel(const SeqGemm g) {
  constexpr int LD = 32 + 8, BM = 128, BN = 128;
  __shared__ __align__(16) bf16 As[BM * LD];
  __shared__ __align__(16) bf16 Bs[BN * LD];
  const int tid = threadIdx.x, z = blockIdx.z, warp = tid >> 5, lane = tid & 31;
  int row0, row_end;
  const bf16* Bp = reinterpret_cast<const bf16*>(g.B) + (size_t)z * g.b_zstride;
  if (g.seg) {
    int t = blockIdx.y, e = 0;
    row0 = -1; row_end = 0;
    for (; e < g.E; ++e) {
      const int s0 = g.seg[e], s1 = g.seg[e + 1];
      const int nt = (s1 - s0 + BM - 1) / BM;
      if (t < nt) { row0 = s0 + t * BM; row_end = s1; break; }
      t -= nt;
    }
    if (row0 < 0) return;
    Bp += (size_t)e * g.b_estride;
  } else {
    row0 = blockIdx.y * BM; row_end = g.M;
  }
  const int col0 = blockIdx.x * BN;
  const TA* Ap = reinterpret_cast<const TA*>(g.A) + (size_t)(z % g.a_mod) * g.a_zstride;
  const int lr = tid >> 1, lk = (tid & 1) * 16;       // loaders: thread -> (row = tid / 2, 16 consecutive k)
  const int ar = row0 + lr;
  const TA* a_ptr = nullptr;
  if (ar < row_end) a_ptr = Ap + (size_t)(g.rows ? g.rows[ar] : ar) * g.lda + lk;
  const int bn = col0 + lr;
  const bf16* b_ptr = bn < g.N ? Bp + (size_t)bn * g.ldb + lk : nullptr;
  constexpr int AV = 16 / sizeof(TA);
  const bool vec_a = (g.lda % AV == 0) && ((reinterpret_cast<uintptr_t>(Ap) & 15) == 0);
  const bool vec_b = (g.ldb % 8 == 0) && ((reinterpret_cast<uintptr_t>(Bp) & 15) == 0);
  const int wm = (warp >> 2) * 64, wn = (warp & 3) * 32;
  float acc[4][4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) acc[i][j][q] = 0.f;
  // ldmatrix lanes.  A (row-major [m][k]): matrices rows 0-7 / 8-15 at k, then at k + 8.  B ([n][k]): columns n 0-7 at k, k + 8, then n 8-15.
  const bf16* a_lane = As + (size_t)(wm + (lane & 15)) * LD + (lane >> 4) * 8;
  const bf16* b_lane = Bs + (size_t)(wn + (lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8;
  uint4 ra[2], rb[2];
  sg_fetch16<TA>(a_ptr, vec_a, g.K - lk, ra);
  sg_fetch16<bf16>(b_ptr, vec_b, g.K - lk, rb);
  for (int k0 = 0; k0 < g.K; k0 += 32) {
    *reinterpret_cast<uint4*>(&As[lr * LD + lk]) = ra[0];
    *reinterpret_cast<uint4*>(&As[lr * LD + lk + 8]) = ra[1];
    *reinterpret_cast<uint4*>(&Bs[lr * LD + lk]) = rb[0];
    *reinterpret_cast<uint4*>(&Bs[lr * LD + lk + 8]) = rb[1];
    __syncthreads();
    if (k0 + 32 < g.K) {
      sg_fetch16<TA>(a_ptr ? a_ptr + k0 + 32 : nullptr, vec_a, g.K - (k0 + 32 + lk), ra);
      sg_fetch16<bf16>(b_ptr ? b_ptr + k0 + 32 : nullptr, vec_b, g.K - (k0 + 32 + lk), rb);
    }
#pragma unroll
    for (int kk = 0; kk < 32; kk += 16) {
      uint32_t a[4][4], b[2][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) ldmatrix_x4(a[i], a_lane + (size_t)i * 16 * LD + kk);
#pragma unroll
      for (int j = 0; j < 2; ++j) ldmatrix_x4(b[j], b_lane + (size_t)j * 16 * LD + kk);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) mma16816(acc[i][j], a[i], b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
    }
    __syncthreads();
  }
  const int ccol = z * g.c_zstride;
  if constexpr (GLU) {      // an accumulator pair (q, q + 1) is one gated unit
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int q = 0; q < 4; q += 2) {
        const int r = row0 + wm + i * 16 + (lane >> 2) + (q >> 1) * 8;
        if (r >= row_end) continue;
        const float w = sg_row_scale(g, r);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int n = col0 + wn + j * 8 + (lane & 3) * 2;
          if (n + 1 < g.N) sg_store_glu(g, r, ccol, n, acc[i][j][q], acc[i][j][q + 1], w);
        }
      }
    return;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int r = row0 + wm + i * 16 + (lane >> 2) + (q >> 1) * 8;
        const int n = col0 + wn + j * 8 + (lane & 3) * 2 + (q & 1);
        if (r >= row_end || n >= g.N) continue;
        float v = acc[i][j][q];
        if (g.flags & FQ3C_BIAS) v += g.bias[ccol + n];
        if (g.flags & FQ3C_GELU) v = gelu_f(v);
        if (g.flags & FQ3C_GELU_TANH) v = gelu_tanh_f(v);
        if (g.flags & FQ3C_SIGMOID) v = sigmoid_f(v);
        if (g.flags & FQ3C_RELU2) { v = fmaxf(v, 0.f); v *= v; }
        const size_t ci = (size_t)r * g.ldc + ccol + n;
        if (g.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(g.C)[ci] = v;
        else reinterpret_cast<bf16*>(g.C)[ci] = __float2bfloat16_rn(v);
      }
}

// K values of a row into shared memory as f32: 16-byte loads when the row allows them (one round trip for a few thousand values
// instead of one per 256), else one value per thread and round.
template <typename TA>
__device__ __forceinline__ void stage_row_f32(float* dst, const TA* src, const int K, const int tid, const int nth) {
  constexpr int V = 16 / sizeof(TA);
  if (((reinterpret_cast<uintptr_t>(src) & 15) == 0) && (K % V == 0)) {
    for (int i = tid; i < K / V; i += nth) {
      const uint4 r = __ldg(reinterpret_cast<const uint4*>(src) + i);
      float* d = dst + i * V;
      if (sizeof(TA) == 2) {
        const uint32_t u[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int q = 0; q < 4; ++q) { d[(2 * q) % V] = __uint_as_float(u[q] << 16); d[(2 * q + 1) % V] = __uint_as_float(u[q] & 0xffff0000u); }
      } else {
        d[0] = __uint_as_float(r.x); d[1] = __uint_as_float(r.y); d[2 % V] = __uint_as_float(r.z); d[3 % V] = __uint_as_float(r.w);
      }
    }
  } else {
    for (int i = tid; i < K; i += nth) dst[i] = ldf<TA>(src + i);
  }
}

// One output row with few rows in flight (decode: M <= 8): a warp per output column streams its weight row once, 16 bytes per
// lane and load, and dots it with every A row (f32 or bf16 in shared memory as f32).  Weight-streaming bound.
template <typename TA, typename TB>
__global__ void __launch_bounds__(256) fq3s_gemv_kernel(const SeqGemm g) {
  extern __shared__ float xs[];  // [M][K]
  const int z = blockIdx.z;
  const TA* Ap = reinterpret_cast<const TA*>(g.A) + (size_t)(z % g.a_mod) * g.a_zstride;
  const TB* Bp = reinterpret_cast<const TB*>(g.B) + (size_t)z * g.b_zstride;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * 8 + warp;
  const TB* w = Bp + (size_t)min(n, g.N - 1) * g.ldb;
  constexpr int VEC = 16 / sizeof(TB);
  constexpr int U = 4;                 // 16-byte weight loads a lane keeps in flight
  const bool vec = ((reinterpret_cast<uintptr_t>(w) & 15) == 0) && (g.K % VEC == 0);
  // the first weight loads leave before the rows are staged: the two latencies overlap
  uint4 raw[U];
  if (vec && n < g.N) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = (lane + 32 * u) * VEC;
      raw[u] = k < g.K ? __ldg(reinterpret_cast<const uint4*>(w + k)) : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  for (int m = 0; m < g.M; ++m) stage_row_f32<TA>(xs + (size_t)m * g.K, Ap + (size_t)m * g.lda, g.K, threadIdx.x, blockDim.x);
  __syncthreads();
  if (n >= g.N) return;
  float acc[8];
#pragma unroll
  for (int m = 0; m < 8; ++m) acc[m] = 0.f;
  if (vec) {
    for (int k0 = lane * VEC; k0 < g.K; k0 += 32 * U * VEC) {
      uint4 nxt[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {      // the next batch is on its way while this one is used
        const int k = k0 + 32 * (U + u) * VEC;
        nxt[u] = k < g.K ? __ldg(reinterpret_cast<const uint4*>(w + k)) : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int k = k0 + 32 * u * VEC;
        if (k < g.K) {
          float wv[VEC];
          if (sizeof(TB) == 2) {
            const uint32_t q4[4] = {raw[u].x, raw[u].y, raw[u].z, raw[u].w};
#pragma unroll
            for (int q = 0; q < 4; ++q) { wv[(2 * q) % VEC] = __uint_as_float(q4[q] << 16); wv[(2 * q + 1) % VEC] = __uint_as_float(q4[q] & 0xffff0000u); }
          } else {
            wv[0] = __uint_as_float(raw[u].x); wv[1] = __uint_as_float(raw[u].y); wv[2 % VEC] = __uint_as_float(raw[u].z); wv[3 % VEC] = __uint_as_float(raw[u].w);
          }
#pragma unroll
          for (int m = 0; m < 8; ++m)
            if (m < g.M) {
#pragma unroll
              for (int q = 0; q < VEC; ++q) acc[m] = fmaf(wv[q], xs[m * g.K + k + q], acc[m]);
            }
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) raw[u] = nxt[u];
    }
  } else {
    for (int k = lane; k < g.K; k += 32) {
      const float wv = ldf<TB>(w + k);
#pragma unroll
      for (int m = 0; m < 8; ++m)
        if (m < g.M) acc[m] = fmaf(wv, xs[m * g.K + k], acc[m]);
    }
  }
  const int ccol = z * g.c_zstride;
  if (g.flags & FQ3C_SWIGLU) {      // warps (2k, 2k + 1) hold a unit's gate and up columns: the odd one hands its sums over
    __shared__ float ex[8][8];
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      if (m >= g.M) break;
      acc[m] = warp_sum(acc[m]);
      if ((warp & 1) && lane == 0) ex[warp][m] = acc[m];
    }
    asm volatile("bar.sync %0, 64;" ::"r"(1 + (warp >> 1)) : "memory");
    if (!(warp & 1) && lane == 0 && n + 1 < g.N)
      for (int m = 0; m < g.M; ++m) sg_store_glu(g, m, ccol, n, acc[m], ex[warp + 1][m], sg_row_scale(g, m));
    return;
  }
#pragma unroll
  for (int m = 0; m < 8; ++m) {
    if (m >= g.M) break;
    float v = warp_sum(acc[m]);
    if (lane == 0) {
      if (g.flags & FQ3C_BIAS) v += g.bias[ccol + n];
      if (g.flags & FQ3C_GELU) v = gelu_f(v);
      if (g.flags & FQ3C_GELU_TANH) v = gelu_tanh_f(v);
      if (g.flags & FQ3C_SIGMOID) v = sigmoid_f(v);
      if (g.flags & FQ3C_RELU2) { v = fmaxf(v, 0.f); v *= v; }
      const size_t ci = (size_t)m * g.ldc + ccol + n;
      if (g.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(g.C)[ci] = v;
      else reinterpret_cast<bf16*>(g.C)[ci] = __float2bfloat16_rn(v);
    }
  }
}

// Grouped product with few rows in flight (decode: tokens x chosen experts <= 16 rows): block (column octet, sorted row); the row's
// expert comes from the segment starts, a warp per output column streams that expert's weight row once with 16-byte loads.
template <typename TA, typename TB>
__global__ void __launch_bounds__(256) fq3s_ggemv_kernel(const SeqGemm g) {
  extern __shared__ float xs[];  // [K]
  const int p = blockIdx.y;
  int e = 0;
  while (e < g.E && p >= g.seg[e + 1]) ++e;
  if (e >= g.E) return;          // beyond the last segment: choices without tensors (identity experts) leave fewer rows
  const int arow = g.rows ? g.rows[p] : p;
  const TA* a = reinterpret_cast<const TA*>(g.A) + (size_t)arow * g.lda;
  stage_row_f32<TA>(xs, a, g.K, threadIdx.x, blockDim.x);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * 8 + warp;
  if (n >= g.N) return;
  const TB* w = reinterpret_cast<const TB*>(g.B) + (size_t)e * g.b_estride + (size_t)n * g.ldb;
  float acc = 0.f;
  constexpr int VEC = 16 / sizeof(TB);
  if (((reinterpret_cast<uintptr_t>(w) & 15) == 0) && (g.K % VEC == 0)) {
    for (int k0 = lane * VEC; k0 < g.K; k0 += 4 * 32 * VEC) {      // four 16-byte loads in flight per lane
      uint4 raw[4];
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        const int k = k0 + b * 32 * VEC;
        raw[b] = k < g.K ? __ldg(reinterpret_cast<const uint4*>(w + k)) : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        const int k = k0 + b * 32 * VEC;
        if (k < g.K) {
          const uint32_t u[4] = {raw[b].x, raw[b].y, raw[b].z, raw[b].w};
          if (sizeof(TB) == 2) {
#pragma unroll
            for (int q = 0; q < 4; ++q) {
              acc = fmaf(__uint_as_float(u[q] << 16), xs[k + 2 * q], acc);
              acc = fmaf(__uint_as_float(u[q] & 0xffff0000u), xs[k + 2 * q + 1], acc);
            }
          } else {
#pragma unroll
            for (int q = 0; q < 4; ++q) acc = fmaf(__uint_as_float(u[q]), xs[k + q], acc);
          }
        }
      }
    }
  } else {
    for (int k = lane; k < g.K; k += 32) acc = fmaf(ldf<TB>(w + k), xs[k], acc);
  }
  float v = warp_sum(acc);
  if (g.flags & FQ3C_SWIGLU) {
    __shared__ float ex[8];
    if ((warp & 1) && lane == 0) ex[warp] = v;
    asm volatile("bar.sync %0, 64;" ::"r"(1 + (warp >> 1)) : "memory");
    if (!(warp & 1) && lane == 0 && n + 1 < g.N) sg_store_glu(g, p, 0, n, v, ex[warp + 1], sg_row_scale(g, p));
    return;
  }
  if (lane == 0) {
    if (g.flags & FQ3C_GELU) v = gelu_f(v);
    if (g.flags & FQ3C_GELU_TANH) v = gelu_tanh_f(v);
    if (g.flags & FQ3C_SIGMOID) v = sigmoid_f(v);
    if (g.flags & FQ3C_RELU2) { v = fmaxf(v, 0.f); v *= v; }
    const size_t ci = (size_t)p * g.ldc + n;
    if (g.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(g.C)[ci] = v;
    else reinterpret_cast<bf16*>(g.C)[ci] = __float2bfloat16_rn(v);
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
template <typename TB>
__global__ void fq3s_embed_kernel(const fq3c_op o) {
  const int m = blockIdx.x;
  const int id = reinterpret_cast<const int*>(o.A)[m];
  const TB* row = reinterpret_cast<const TB*>(o.B) + (size_t)id * o.N;
  float* c = reinterpret_cast<float*>(o.C) + (size_t)m * o.ldc;
  const float sc = o.f0 != 0.f ? o.f0 : 1.f;
  const int copies = max(o.i0, 1);
  for (int i = threadIdx.x; i < o.N; i += blockDim.x) {
    const float v = ldf<TB>(row + i) * sc;
    for (int s = 0; s < copies; ++s) c[(size_t)s * (size_t)o.K + i] = v;
    if (o.C2)
      for (int t = 0; t < max(o.i1, 1); ++t) stf(reinterpret_cast<TB*>(o.C2) + (size_t)m * o.ldr + (size_t)t * o.N + i, v);
  }
}

// grid (ceil(N / 256), M + taps - 1): rows >= M write the next history
__global__ void __launch_bounds__(256) fq3s_tconv_kernel(const fq3c_op o) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= o.N) return;
  const int m = blockIdx.y, h = o.taps - 1;
  const float* x = reinterpret_cast<const float*>(o.A);
  const float* hist = reinterpret_cast<const float*>(o.p0);
  if (m >= o.M) {
    const int s = m - o.M, pos = o.M - h + s;
    reinterpret_cast<float*>(const_cast<void*>(o.p1))[(size_t)s * o.N + c] = pos >= 0 ? x[(size_t)pos * o.lda + c] : hist[(size_t)(h + pos) * o.N + c];
    return;
  }
  const float* w = reinterpret_cast<const float*>(o.B) + (size_t)c * o.taps;
  float a = (o.flags & FQ3C_BIAS) ? reinterpret_cast<const float*>(o.bias)[c] : 0.f;
  for (int j = 0; j < o.taps; ++j) {
    const int pos = m - h + j;
    const float v = pos >= 0 ? x[(size_t)pos * o.lda + c] : hist[(size_t)(h + pos) * o.N + c];
    a = fmaf(w[j], v, a);
  }
  if (o.flags & FQ3C_RESID) a += x[(size_t)m * o.lda + c];
  if ((o.flags & FQ3C_SILU) && c >= o.i0) a = a / (1.f + expf(-a));
  if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[(size_t)m * o.ldc + c] = a;
  else reinterpret_cast<bf16*>(o.C)[(size_t)m * o.ldc + c] = __float2bfloat16_rn(a);
}

// The same for many rows of whole 16-byte pieces: a thread takes four columns of TC_ROWS consecutive rows and keeps the last TAPS inputs in
// registers, so that an input is loaded once.  TAPS >= o.taps: the taps in front are zero.  Rows M .. M + taps - 2 are the next history.
// grid (ceil(N / 512), ceil((M + taps - 1) / TC_ROWS)), 128 threads.
constexpr int TC_ROWS = 8;
template <int TAPS>
__global__ void __launch_bounds__(128) fq3s_tconv_vec_kernel(const fq3c_op o) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (c >= o.N) return;
  const int h = o.taps - 1, m0 = blockIdx.y * TC_ROWS;
  const float* x = reinterpret_cast<const float*>(o.A) + c;
  const float* hist = reinterpret_cast<const float*>(o.p0) + c;
  auto input = [&](const int pos) {       // pos in [-h, M); beyond: not used
    if (pos < -h || pos >= o.M) return make_float4(0.f, 0.f, 0.f, 0.f);
    return *reinterpret_cast<const float4*>(pos >= 0 ? x + (size_t)pos * o.lda : hist + (size_t)(h + pos) * o.N);
  };
  float w[4][TAPS];
#pragma unroll
  for (int e = 0; e < 4; ++e)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int t = j - (TAPS - o.taps);
      w[e][j] = t >= 0 ? reinterpret_cast<const float*>(o.B)[(size_t)(c + e) * o.taps + t] : 0.f;
    }
  float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
  if (o.flags & FQ3C_BIAS) { const float* bp = reinterpret_cast<const float*>(o.bias) + c; b = make_float4(bp[0], bp[1], bp[2], bp[3]); }
  const bool act = (o.flags & FQ3C_SILU) && c >= o.i0;
  float4 v[TAPS + TC_ROWS - 1];      // v[i] = input at position m0 + i - (TAPS - 1)
#pragma unroll
  for (int i = 0; i < TAPS + TC_ROWS - 1; ++i) v[i] = input(m0 + i - (TAPS - 1));
#pragma unroll
  for (int r = 0; r < TC_ROWS; ++r) {
    const int m = m0 + r;
    if (m >= o.M + h) return;
    if (m >= o.M) {       // next history row s holds the input at M - h + s = m - h
      const int s = m - o.M, pos = m - h;
      *reinterpret_cast<float4*>(reinterpret_cast<float*>(const_cast<void*>(o.p1)) + (size_t)s * o.N + c) = input(pos);
      continue;
    }
    float a[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const float4 u = v[r + j];
      a[0] = fmaf(w[0][j], u.x, a[0]); a[1] = fmaf(w[1][j], u.y, a[1]); a[2] = fmaf(w[2][j], u.z, a[2]); a[3] = fmaf(w[3][j], u.w, a[3]);
    }
    if (act) {
#pragma unroll
      for (int e = 0; e < 4; ++e) a[e] = a[e] / (1.f + expf(-a[e]));
    }
    if (o.flags & FQ3C_OUT_F32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(o.C) + (size_t)m * o.ldc + c) = make_float4(a[0], a[1], a[2], a[3]);
    else {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(a[0], a[1]), hi = __floats2bfloat162_rn(a[2], a[3]);
      *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(o.C) + (size_t)m * o.ldc + c) =
          make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
  }
}

// grid (M, groups); one block per (row, group): 128 threads, or up to 1024 for a few rows (decoding).  FQ3C_CENTER: mean and variance instead of the mean square.  An optional silu gate (p1, pitch i1;
// FQ3C_SIGMOID: a sigmoid gate) multiplies the row before the statistics (FQ3C_GATE_PRE) or the finished row (FQ3C_GATE_POST); weights repeat
// with period i2 when i2 > 0; divisors (bias, pitch cin) divide a group before anything else.
__device__ __forceinline__ float gate_f(const float z, const bool plain) { return plain ? sigmoid_f(z) : z / (1.f + expf(-z)); }
__global__ void __launch_bounds__(1024) fq3s_gnorm_kernel(const fq3c_op o) {
  __shared__ float red[32];
  const int m = blockIdx.x, gsz = o.N / o.i0, c0 = blockIdx.y * gsz;
  const float* x = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda + c0;
  const bool pre = (o.flags & FQ3C_GATE_PRE) != 0, post = (o.flags & FQ3C_GATE_POST) != 0;
  const float* gate = (pre || post) ? reinterpret_cast<const float*>(o.p1) + (size_t)m * o.i1 + c0 : nullptr;
  const bool plain = (o.flags & FQ3C_SIGMOID) != 0;
  const float inv = o.bias ? 1.f / reinterpret_cast<const float*>(o.bias)[(size_t)m * o.cin + blockIdx.y] : 1.f;
  float mean = 0.f;
  if (o.flags & FQ3C_CENTER) {      // layer norm: the mean first, then the squared deviations from it (two passes, no cancellation)
    float sm = 0.f;
    for (int i = threadIdx.x; i < gsz; i += blockDim.x) {
      float v = x[i] * inv;
      if (pre) v *= gate_f(gate[i], plain);
      sm += v;
    }
    mean = seq_block_sum(sm, red) / (float)gsz;
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < gsz; i += blockDim.x) {
    float v = x[i] * inv;
    if (pre) v *= gate_f(gate[i], plain);
    v -= mean;
    ss = fmaf(v, v, ss);
  }
  ss = seq_block_sum(ss, red);
  const float rs = 1.f / sqrtf(ss / (float)gsz + o.f0);
  const float* w = reinterpret_cast<const float*>(o.scale);
  const int wmod = o.i2 > 0 ? o.i2 : o.N;
  const size_t orow = (size_t)m + (o.p0 ? (size_t)*reinterpret_cast<const int*>(o.p0) : 0);
  for (int i = threadIdx.x; i < gsz; i += blockDim.x) {
    float v = x[i] * inv;
    if (pre) v *= gate_f(gate[i], plain);
    v = (v - mean) * rs;
    if (w) v *= w[(c0 + i) % wmod];
    if (post) v *= gate_f(gate[i], plain);
    if (o.flags & FQ3C_RESID) v += reinterpret_cast<const float*>(o.res)[(size_t)m * o.ldr + c0 + i];
    if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[orow * o.ldc + c0 + i] = v;
    else reinterpret_cast<bf16*>(o.C)[orow * o.ldc + c0 + i] = __float2bfloat16_rn(v);
    if (o.C2) reinterpret_cast<bf16*>(o.C2)[orow * o.ldc + c0 + i] = __float2bfloat16_rn(v);
  }
}

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void st4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void st4(bf16* p, const float (&v)[4]) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}
// The same norm for many (row, group) pairs: a warp each, the group in registers, 16-byte loads.  grid (ceil(M * groups / 4)), 128 threads.
constexpr int GN_VECS = 4;
__global__ void __launch_bounds__(128) fq3s_gnorm_warp_kernel(const fq3c_op o) {
  const long long pair = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (pair >= (long long)o.M * o.i0) return;
  const int lane = threadIdx.x & 31, m = (int)(pair / o.i0), gi = (int)(pair - (long long)m * o.i0), gsz = o.N / o.i0, c0 = gi * gsz;
  const float* x = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda + c0;
  const bool pre = (o.flags & FQ3C_GATE_PRE) != 0, post = (o.flags & FQ3C_GATE_POST) != 0, plain = (o.flags & FQ3C_SIGMOID) != 0;
  const float* gate = (pre || post) ? reinterpret_cast<const float*>(o.p1) + (size_t)m * o.i1 + c0 : nullptr;
  const float inv = o.bias ? 1.f / reinterpret_cast<const float*>(o.bias)[(size_t)m * o.cin + gi] : 1.f;
  float v[GN_VECS][4], g[GN_VECS][4];
#pragma unroll
  for (int q = 0; q < GN_VECS; ++q) {
    const int i = (q * 32 + lane) * 4;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    if (i < gsz) { a = ld4(x + i); if (gate) b = ld4(gate + i); }
    v[q][0] = a.x * inv; v[q][1] = a.y * inv; v[q][2] = a.z * inv; v[q][3] = a.w * inv;
    g[q][0] = b.x; g[q][1] = b.y; g[q][2] = b.z; g[q][3] = b.w;
  }
  float sm = 0.f, ss = 0.f;
#pragma unroll
  for (int q = 0; q < GN_VECS; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (gate) g[q][e] = gate_f(g[q][e], plain);
      if (pre) v[q][e] *= g[q][e];
      sm += v[q][e];
    }
  const float mean = (o.flags & FQ3C_CENTER) ? warp_sum(sm) / (float)gsz : 0.f;
#pragma unroll
  for (int q = 0; q < GN_VECS; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      v[q][e] -= mean;
      if ((q * 32 + lane) * 4 < gsz) ss = fmaf(v[q][e], v[q][e], ss);
    }
  const float rs = 1.f / sqrtf(warp_sum(ss) / (float)gsz + o.f0);
  const float* w = reinterpret_cast<const float*>(o.scale);
  const int wmod = o.i2 > 0 ? o.i2 : o.N;
  const size_t orow = (size_t)m + (o.p0 ? (size_t)*reinterpret_cast<const int*>(o.p0) : 0);
#pragma unroll
  for (int q = 0; q < GN_VECS; ++q) {
    const int i = (q * 32 + lane) * 4;
    if (i >= gsz) continue;
    float4 wv = make_float4(1.f, 1.f, 1.f, 1.f), r = make_float4(0.f, 0.f, 0.f, 0.f);
    if (w) wv = ld4(w + (c0 + i) % wmod);
    if (o.flags & FQ3C_RESID) r = ld4(reinterpret_cast<const float*>(o.res) + (size_t)m * o.ldr + c0 + i);
    const float ww[4] = {wv.x, wv.y, wv.z, wv.w}, rr[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      v[q][e] *= rs;
      if (w) v[q][e] *= ww[e];
      if (post) v[q][e] *= g[q][e];
      if (o.flags & FQ3C_RESID) v[q][e] += rr[e];
    }
    if (o.flags & FQ3C_OUT_F32) st4(reinterpret_cast<float*>(o.C) + orow * o.ldc + c0 + i, v[q]);
    else st4(reinterpret_cast<bf16*>(o.C) + orow * o.ldc + c0 + i, v[q]);
    if (o.C2) st4(reinterpret_cast<bf16*>(o.C2) + orow * o.ldc + c0 + i, v[q]);
  }
}

__global__ void __launch_bounds__(256) fq3s_polynorm_kernel(const fq3c_op o) {
  __shared__ float red[32];
  const int m = blockIdx.x;
  const float* x = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda;
  const float* p = reinterpret_cast<const float*>(o.p0);
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  for (int i = threadIdx.x; i < o.N; i += blockDim.x) {
    const float z = x[i], z2 = z * z, z3 = z2 * z;
    s1 = fmaf(z, z, s1); s2 = fmaf(z2, z2, s2); s3 = fmaf(z3, z3, s3);
  }
  s1 = seq_block_sum(s1, red); s2 = seq_block_sum(s2, red); s3 = seq_block_sum(s3, red);
  const float inv = 1.f / (float)o.N;
  const float r1 = p[0] / sqrtf(s1 * inv + o.f0), r2 = p[1] / sqrtf(s2 * inv + o.f0), r3 = p[2] / sqrtf(s3 * inv + o.f0), e = p[3];
  for (int i = threadIdx.x; i < o.N; i += blockDim.x) {
    const float z = x[i], z2 = z * z, z3 = z2 * z;
    const float v = r1 * z + r2 * z2 + r3 * z3 + e;
    if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[(size_t)m * o.ldc + i] = v;
    else reinterpret_cast<bf16*>(o.C)[(size_t)m * o.ldc + i] = __float2bfloat16_rn(v);
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Gated diagonal linear recurrence.  The recurrence S_t = a_t S_(t-1) + b_t is associative in (a, b), so a long run of rows is
// cut into `chunks` pieces: pass 0 folds every piece from a zero state into (prod a, local S), pass 1 walks the pieces' carries in
// order and writes the outputs.  grid (ceil(N / 128), chunks).  A single piece (decode, short runs) does everything in pass 1.
// ---------------------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void lru_coeffs(const fq3c_op& o, int t, int c, float sp, float& a, float& b) {
  const float* g = reinterpret_cast<const float*>(o.A) + (size_t)t * o.lda;
  const float r = g[c], ig = g[o.N + c];
  const float u = reinterpret_cast<const float*>(o.B)[(size_t)t * o.cin + c];
  const float la = -o.f0 * r * sp;
  a = expf(la);
  b = sqrtf(fmaxf(-expm1f(2.f * la), 0.f)) * ig * u;
}
__global__ void __launch_bounds__(128) fq3s_lru_fold_kernel(const fq3c_op o, const int chunks, const int per, float* carry) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, q = blockIdx.y;
  if (c >= o.N) return;
  const float sp = softplus_f(reinterpret_cast<const float*>(o.scale)[c]);
  const int t0 = q * per, t1 = min(o.M, t0 + per);
  float pa = 1.f, s = 0.f;
  for (int t = t0; t < t1; ++t) {
    float a, b;
    lru_coeffs(o, t, c, sp, a, b);
    s = fmaf(a, s, b);
    pa *= a;
  }
  carry[((size_t)q * 2) * o.N + c] = pa;
  carry[((size_t)q * 2 + 1) * o.N + c] = s;
}
__global__ void __launch_bounds__(128) fq3s_lru_scan_kernel(const fq3c_op o, const int chunks, const int per, const float* carry) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, q = blockIdx.y;
  if (c >= o.N) return;
  const float sp = softplus_f(reinterpret_cast<const float*>(o.scale)[c]);
  float* state = reinterpret_cast<float*>(const_cast<void*>(o.p0));
  float s = state[c];
  for (int j = 0; j < q; ++j) s = fmaf(carry[((size_t)j * 2) * o.N + c], s, carry[((size_t)j * 2 + 1) * o.N + c]);
  const int t0 = q * per, t1 = min(o.M, t0 + per);
  const float* y = reinterpret_cast<const float*>(o.res);
  for (int t = t0; t < t1; ++t) {
    float a, b;
    lru_coeffs(o, t, c, sp, a, b);
    s = fmaf(a, s, b);
    const float v = s * gelu_tanh_f(y[(size_t)t * o.ldr + c]);
    if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[(size_t)t * o.ldc + c] = v;
    else reinterpret_cast<bf16*>(o.C)[(size_t)t * o.ldc + c] = __float2bfloat16_rn(v);
  }
  // the last piece owns the state; every piece read it before (stream order: the fold pass never touches it, and within this
  // launch only the last piece writes) — so the write goes to the staging copy C2 and FQ3C_COMMIT installs it
  if (q == chunks - 1) reinterpret_cast<float*>(o.C2)[c] = s;
}

// ---------------------------------------------------------------------------------------------------------------------------
// Router: one thread per token, its scores in shared memory [n][threads].
// ---------------------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void router_token(const fq3c_op& o, const int m, float* rsm, const int tpb, const int tx) {
  const int n = o.N;
  float* s = rsm + tx;                       // s[i * tpb]
  float* ch = rsm + (size_t)n * tpb + tx;    // choice scores
  const float* z = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda;
  const float* corr = reinterpret_cast<const float*>(o.bias);
  if (o.flags & FQ3C_SIGMOID) {
    for (int i = 0; i < n; ++i) { const float v = sigmoid_f(z[i]); s[i * tpb] = v; ch[i * tpb] = v + (corr ? corr[i] : 0.f); }
  } else {
    float mx = -INFINITY;
    for (int i = 0; i < n; ++i) mx = fmaxf(mx, z[i]);
    float sum = 0.f;
    for (int i = 0; i < n; ++i) { const float e = expf(z[i] - mx); s[i * tpb] = e; sum += e; }
    const float inv = 1.f / sum;
    for (int i = 0; i < n; ++i) { const float v = s[i * tpb] * inv; s[i * tpb] = v; ch[i * tpb] = v + (corr ? corr[i] : 0.f); }
  }
  const int G = o.i1, keep = o.i2, gsz = n / max(G, 1);
  if (G > 1 && keep < G) {
    unsigned long long kept = 0ull;
    for (int k = 0; k < keep; ++k) {
      int best = -1; float bv = 0.f;
      for (int gq = 0; gq < G; ++gq) {
        if ((kept >> gq) & 1ull) continue;
        float gm = -INFINITY;
        for (int i = 0; i < gsz; ++i) gm = fmaxf(gm, ch[(gq * gsz + i) * tpb]);
        if (best < 0 || gm > bv) { best = gq; bv = gm; }
      }
      kept |= 1ull << best;
    }
    for (int gq = 0; gq < G; ++gq)
      if (!((kept >> gq) & 1ull))
        for (int i = 0; i < gsz; ++i) ch[(gq * gsz + i) * tpb] = -INFINITY;
  }
  int* ids = reinterpret_cast<int*>(o.C) + (size_t)m * o.i0;
  float* wt = reinterpret_cast<float*>(o.C2) + (size_t)m * o.i0;
  float wsum = 0.f;
  for (int k = 0; k < o.i0; ++k) {
    int best = -1; float bv = 0.f;
    for (int i = 0; i < n; ++i) {
      const float v = ch[i * tpb];
      if (v == -INFINITY) continue;
      if (best < 0 || v > bv) { best = i; bv = v; }
    }
    if (best < 0) best = 0;   // fewer eligible experts than asked for: cannot happen with a consistent configuration
    ch[best * tpb] = -INFINITY;
    ids[k] = best;
    const float sv = s[best * tpb];
    wt[k] = sv;
    wsum += sv;
  }
  const float sc = (o.flags & FQ3C_RAW_WEIGHTS) ? o.f0 : o.f0 / (wsum + 1e-20f);
  for (int k = 0; k < o.i0; ++k) wt[k] *= sc;
}
// With ws / p0 / p1 set (a single token, at most 16 choices, K = experts that have tensors) the launch also does the grouping
// by expert that fq3s_moe_sort_kernel does for many tokens: segment starts -> p0, rows -> p1, each choice's place -> ws.
__global__ void fq3s_router_kernel(const fq3c_op o) {
  extern __shared__ float rsm[];
  const int m = blockIdx.x * blockDim.x + threadIdx.x;
  if (m < o.M) router_token(o, m, rsm, blockDim.x, threadIdx.x);
  if (!o.ws) return;
  __syncthreads();
  if (threadIdx.x != 0 || blockIdx.x != 0) return;
  const int E = o.K, top = o.i0, n = min(16, o.M * top);
  int* seg = const_cast<int*>(reinterpret_cast<const int*>(o.p0));
  int* rows = const_cast<int*>(reinterpret_cast<const int*>(o.p1));
  int* pos = reinterpret_cast<int*>(o.ws);
  int lid[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) lid[i] = i < n ? reinterpret_cast<const int*>(o.C)[i] : 0x7fffffff;
  int run = 0;
  for (int e = 0; e < E; ++e) {
    seg[e] = run;
#pragma unroll
    for (int i = 0; i < 16; ++i)
      if (lid[i] == e) { rows[run] = i / top; pos[i] = run; ++run; }
  }
  seg[E] = run;
#pragma unroll
  for (int i = 0; i < 16; ++i)
    if (i < n && lid[i] >= E) pos[i] = -1;
}

// One block.  Counting sort of the (token, choice) pairs by expert, token order kept inside an expert.
__global__ void __launch_bounds__(1024) fq3s_moe_sort_kernel(const fq3c_op o) {
  extern __shared__ int ssm[];   // [E + 1] starts, then [nchunk][E] counts
  const int E = o.i1, n = o.M * o.i0, nth = blockDim.x;
  const int* ids = reinterpret_cast<const int*>(o.A);
  int* seg = reinterpret_cast<int*>(o.C);
  int* rows = reinterpret_cast<int*>(o.C2);
  int* pos = reinterpret_cast<int*>(o.ws);
  int* start = ssm;
  int* cnt = ssm + E + 1;        // cnt[t * E + e]: entries of expert e in thread t's contiguous share
  const int per = (n + nth - 1) / nth;
  const int i0 = threadIdx.x * per, i1 = min(n, i0 + per);
  for (int e = 0; e < E; ++e) cnt[threadIdx.x * E + e] = 0;
  for (int i = i0; i < i1; ++i) { const int e = ids[i]; if (e < E) cnt[threadIdx.x * E + e] += 1; }
  __syncthreads();
  // per expert: exclusive scan over the threads' shares (thread e walks column e)
  for (int e = threadIdx.x; e < E; e += nth) {
    int run = 0;
    for (int t = 0; t < nth; ++t) { const int v = cnt[t * E + e]; cnt[t * E + e] = run; run += v; }
    start[e + 1] = run;   // total, turned into starts below
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int run = 0;
    start[0] = 0;
    for (int e = 0; e < E; ++e) { const int v = start[e + 1]; start[e] = run; run += v; }
    start[E] = run;
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= E; e += nth) seg[e] = start[e];
  for (int i = i0; i < i1; ++i) {
    const int e = ids[i];
    if (e < E) {
      const int p = start[e] + cnt[threadIdx.x * E + e]++;
      rows[p] = i / o.i0;
      pos[i] = p;
    } else {
      pos[i] = -1;
    }
  }
}

__global__ void __launch_bounds__(256) fq3s_moe_combine_kernel(const fq3c_op o) {
  const int m = blockIdx.x, top = o.i0;
  const int* ids = reinterpret_cast<const int*>(o.p0) + (size_t)m * top;
  const float* w = o.p1 ? reinterpret_cast<const float*>(o.p1) + (size_t)m * top : nullptr;
  const int* pos = reinterpret_cast<const int*>(o.ws) + (size_t)m * top;
  const float* Y = reinterpret_cast<const float*>(o.A);
  const float* x = reinterpret_cast<const float*>(o.B) + (size_t)m * o.ldr;
  const float* sh = o.res ? reinterpret_cast<const float*>(o.res) + (size_t)m * o.ldr : nullptr;
  const float sg = (sh && o.scale) ? sigmoid_f(reinterpret_cast<const float*>(o.scale)[(size_t)m * o.i2]) : 1.f;   // one gate per token
  float* c = reinterpret_cast<float*>(o.C) + (size_t)m * o.ldc;
  for (int i = threadIdx.x; i < o.N; i += blockDim.x) {
    float acc = 0.f;
    for (int j = 0; j < top; ++j) {
      const float v = ids[j] >= o.i1 ? x[i] : Y[(size_t)pos[j] * o.lda + i];
      acc = w ? fmaf(w[j], v, acc) : acc + v;
    }
    if (sh) acc = fmaf(sg, sh[i], acc);
    c[i] = acc;
  }
}

// grid (copies, 8)
__global__ void __launch_bounds__(256) fq3s_commit_kernel(const long long* desc, int* counter, int by) {
  const long long* d = desc + (size_t)blockIdx.x * 3;
  uint32_t* dst = reinterpret_cast<uint32_t*>(d[0]);
  const uint32_t* src = reinterpret_cast<const uint32_t*>(d[1]);
  const long long n = d[2] >> 2;
  for (long long i = (long long)blockIdx.y * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.y * blockDim.x) dst[i] = src[i];
  if (blockIdx.x == 0 && blockIdx.y == 0 && threadIdx.x == 0 && counter) *counter += by;
}

// ---------------------------------------------------------------------------------------------------------------------------
// Latent attention, absorbed form: all heads of a group share the latent rows, so a block stages a tile of TJ rows once and every
// head scores it.  grid (M, head groups, splits), 256 threads.  Shared memory (f32): q [HG][R], tile [TJ][R + 1], p [HG][TJ],
// out [HG][R], running max / sum / rescale [3][HG].  Online softmax over the tiles; a single split finishes in place (sink
// included), several leave (max, sum, out) per split in ws and fq3s_latent_merge_kernel finishes.
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int LA_TJ = 32;
__host__ __device__ inline size_t latent_attn_smem(int HG, int R, int E) {
  return sizeof(float) * ((size_t)HG * (2 * R + E) + (size_t)LA_TJ * (R + E + 1) + (size_t)HG * LA_TJ + 3 * (size_t)HG);
}
template <typename TC>
__global__ void __launch_bounds__(256) fq3s_latent_attn_kernel(const fq3c_op o, const int HG, const int splits) {
  extern __shared__ float lsm[];
  // E more columns behind the R latent ones (a rotated key part) enter the scores only; D = R + E is a cache row's width
  const int R = o.i1, E = o.cin, D = R + E, H = o.i0, m = blockIdx.x, h0 = blockIdx.y * HG, z = blockIdx.z;
  const int hg = min(HG, H - h0);
  float* qs = lsm;
  float* os = qs + (size_t)HG * D;
  float* tile = os + (size_t)HG * R;
  float* sc = tile + (size_t)LA_TJ * (D + 1);
  float* mx = sc + (size_t)HG * LA_TJ;
  float* ls = mx + HG;
  float* al = ls + HG;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int P = o.p0 ? *reinterpret_cast<const int*>(o.p0) : 0;
  const int nkeys = P + m + 1, jbeg = o.a_rows > 0 ? max(0, nkeys - o.a_rows) : 0;      // a window's first key
  int per = (nkeys - jbeg + splits - 1) / splits;
  per = (per + LA_TJ - 1) / LA_TJ * LA_TJ;
  const int j0 = jbeg + z * per, j1 = min(nkeys, j0 + per);
  const float* q = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda + (size_t)h0 * R;
  const float* qe = E > 0 ? reinterpret_cast<const float*>(o.p1) + (size_t)m * o.taps + (size_t)h0 * E : nullptr;
  for (int i = tid; i < hg * D; i += blockDim.x) {
    const int h = i / D, r = i - h * D;
    qs[i] = (r < R ? q[(size_t)h * R + r] : qe[(size_t)h * E + r - R]) * o.f0;
  }
  for (int i = tid; i < hg * R; i += blockDim.x) os[i] = 0.f;
  for (int i = tid; i < hg; i += blockDim.x) { mx[i] = -INFINITY; ls[i] = 0.f; }
  const TC* cache = reinterpret_cast<const TC*>(o.B);
  __syncthreads();
  for (int jt = j0; jt < j1; jt += LA_TJ) {
    for (int i = tid; i < LA_TJ * D; i += blockDim.x) {
      const int j = i / D, r = i - j * D;
      tile[j * (D + 1) + r] = (jt + j < j1) ? ldf<TC>(cache + (size_t)(jt + j) * o.ldr + r) : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < hg * LA_TJ; i += blockDim.x) {
      const int h = i / LA_TJ, j = i - h * LA_TJ;
      const float* qq = qs + (size_t)h * D;
      const float* tt = tile + (size_t)j * (D + 1);
      float d0 = 0.f, d1 = 0.f;
      int r = 0;
      for (; r + 1 < D; r += 2) { d0 = fmaf(qq[r], tt[r], d0); d1 = fmaf(qq[r + 1], tt[r + 1], d1); }
      if (r < D) d0 = fmaf(qq[r], tt[r], d0);
      sc[i] = (jt + j < j1) ? d0 + d1 : -INFINITY;
    }
    __syncthreads();
    for (int h = warp; h < hg; h += (blockDim.x >> 5)) {   // LA_TJ == 32: one lane per key of the tile
      const float s = sc[h * LA_TJ + lane];
      const float tm = warp_max(s);
      const float mo = mx[h], mn = fmaxf(mo, tm);
      const float p = s == -INFINITY ? 0.f : expf(s - mn);
      const float ps = warp_sum(p);
      sc[h * LA_TJ + lane] = p;
      if (lane == 0) {
        const float a = mo == -INFINITY ? 0.f : expf(mo - mn);
        al[h] = a; ls[h] = ls[h] * a + ps; mx[h] = mn;
      }
    }
    __syncthreads();
    for (int i = tid; i < hg * R; i += blockDim.x) {
      const int h = i / R, r = i - h * R;
      float acc = os[i] * al[h];
      const float* pp = sc + h * LA_TJ;
#pragma unroll 8
      for (int j = 0; j < LA_TJ; ++j) acc = fmaf(pp[j], tile[j * (D + 1) + r], acc);
      os[i] = acc;
    }
    __syncthreads();
  }
  if (splits == 1) {
    const float* sink = reinterpret_cast<const float*>(o.scale);
    const float* gate = o.res ? reinterpret_cast<const float*>(o.res) + (size_t)m * o.m_begin + h0 : nullptr;
    float* c = reinterpret_cast<float*>(o.C) + (size_t)m * o.ldc + (size_t)h0 * R;
    for (int i = tid; i < hg * R; i += blockDim.x) {
      const int h = i / R;
      float den = ls[h], f = 1.f;
      if (sink) {
        const float sk = sink[h0 + h], mm = fmaxf(mx[h], sk);
        f = expf(mx[h] - mm);
        den = ls[h] * f + expf(sk - mm);
      }
      if (gate) f *= sigmoid_f(gate[h]);
      c[i] = os[i] * f / den;
    }
  } else {
    float* ws = reinterpret_cast<float*>(o.ws);
    // partial state of (m, head, split): [max, sum] then R outputs
    for (int i = tid; i < hg * R; i += blockDim.x) {
      const int h = i / R, r = i - h * R;
      float* dst = ws + (((size_t)m * H + h0 + h) * splits + z) * (R + 2);
      dst[2 + r] = os[i];
      if (r == 0) { dst[0] = mx[h]; dst[1] = ls[h]; }
    }
  }
}
// grid (M, H).  The splits' maxima and sums are read once (a thread per split), their weights exp(max_s - max) live in shared
// memory, and every thread then adds its columns with the loads of eight splits in flight.
__global__ void __launch_bounds__(128) fq3s_latent_merge_kernel(const fq3c_op o, const int splits) {
  __shared__ float wsm[64];
  __shared__ float red[8];
  const int R = o.i1, H = o.i0, m = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float* base = reinterpret_cast<const float*>(o.ws) + ((size_t)m * H + h) * splits * (R + 2);
  const float* sink = reinterpret_cast<const float*>(o.scale);
  const float sk = sink ? sink[h] : -INFINITY;
  const float ms = tid < splits ? base[(size_t)tid * (R + 2)] : -INFINITY;
  const float ls = tid < splits ? base[(size_t)tid * (R + 2) + 1] : 0.f;
  float mm = fmaxf(ms, sk);
#pragma unroll
  for (int d = 16; d > 0; d >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffffu, mm, d));
  if (lane == 0) red[warp] = mm;
  __syncthreads();
  mm = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
  const float wt = ms == -INFINITY ? 0.f : expf(ms - mm);
  if (tid < splits) wsm[tid] = wt;
  float den = ls * wt;
#pragma unroll
  for (int d = 16; d > 0; d >>= 1) den += __shfl_xor_sync(0xffffffffu, den, d);
  if (lane == 0) red[4 + warp] = den;
  __syncthreads();
  den = red[4] + red[5] + red[6] + red[7] + (sink ? expf(sk - mm) : 0.f);
  if (o.res) den /= sigmoid_f(reinterpret_cast<const float*>(o.res)[(size_t)m * o.m_begin + h]);      // the head's output gate
  float* c = reinterpret_cast<float*>(o.C) + (size_t)m * o.ldc + (size_t)h * R;
  for (int r = tid; r < R; r += blockDim.x) {
    float acc = 0.f;
    int s = 0;
    for (; s + 8 <= splits; s += 8) {
      float v[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) v[u] = base[(size_t)(s + u) * (R + 2) + 2 + r];
#pragma unroll
      for (int u = 0; u < 8; ++u) acc = fmaf(v[u], wsm[s + u], acc);
    }
    for (; s < splits; ++s) acc = fmaf(base[(size_t)s * (R + 2) + 2 + r], wsm[s], acc);
    c[r] = acc / den;
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Latent attention on the tensor cores (bf16 cache).  The heads are the M dimension of the MMA: one query's 16 heads share every
// latent row, so scores S [16 heads x TJ keys] = Q' [16 x R] . C^T and outputs O' [16 x R] += P [16 x TJ] . C [TJ x R] are
// m16n8k16 tiles whose B operand is the staged tile of latent rows itself (row-major for the scores, ldmatrix.trans for the
// outputs).  A block takes QB = 4 consecutive queries (they see almost the same keys) x RS slices of R (<= 256 columns of O' per
// warp: 128 accumulator registers); the RS warps of a query compute its scores redundantly.  A single query (decoding) gets a
// block of its own (QB = 1) whose up to eight warps split R.  Scores, maxima, sums and the
// rescaling are f32; a weight enters the output product as a bf16 pair p_hi + p_lo (two MMAs), i.e. with 16 mantissa bits, the
// query as one bf16 (the rounding a bf16 product applies to its operand).  grid (ceil(M / 4), ceil(H / 16), splits).
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int LM_QB = 4;
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&h);
}
template <int NTM>
__global__ void __launch_bounds__(256) fq3s_latent_attn_mma_kernel(const fq3c_op o, const int RS, const int splits, const int TJ, const int QB) {
  extern __shared__ __align__(16) unsigned char lm_raw[];
  const int R = o.i1, E = o.cin, D = R + E, H = o.i0, LDQ = D + 8;      // E score-only columns behind the R latent ones
  bf16* Qs = reinterpret_cast<bf16*>(lm_raw);          // [QB][16][LDQ]
  bf16* Ct0 = Qs + (size_t)QB * 16 * LDQ;           // two tiles [TJ][LDQ]: one is read while the next one arrives (cp.async)
  const int tid = threadIdx.x, nth = blockDim.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int wq = warp / RS, wr = warp - wq * RS;
  // the last queries see the most keys: their blocks start first
  const int m0 = (gridDim.x - 1 - blockIdx.x) * QB, h0 = blockIdx.y * 16, z = blockIdx.z;
  const int P = o.p0 ? *reinterpret_cast<const int*>(o.p0) : 0;
  const int nk_max = P + min(o.M, m0 + QB), W = o.a_rows;
  const int jbeg = W > 0 ? max(0, P + m0 + 1 - W) : 0;      // the first key of the block's first (widest-reaching) window
  int per = (nk_max - jbeg + splits - 1) / splits;
  per = (per + TJ - 1) / TJ * TJ;
  const int j0 = jbeg + z * per, j1 = min(nk_max, j0 + per);
  const int m = m0 + wq;
  const bool active = m < o.M;
  const int nk = min(P + m + 1, j1);                   // this query's keys end here (inside this split)
  const int klo = W > 0 ? P + m + 1 - W : 0;           // ... and begin here
  const float* A = reinterpret_cast<const float*>(o.A);
  const float* A2 = reinterpret_cast<const float*>(o.p1);
  const int nq = min(QB, o.M - m0);                 // live queries of this block: the others' warps never read their rows
  for (int i = tid; i < nq * 16 * D; i += nth) {
    const int q = i / (16 * D), rem = i - q * 16 * D, h = rem / D, r = rem - h * D;
    float v = 0.f;
    if (h0 + h < H)
      v = (r < R ? A[(size_t)(m0 + q) * o.lda + (size_t)(h0 + h) * R + r] : A2[(size_t)(m0 + q) * o.taps + (size_t)(h0 + h) * E + r - R]) * o.f0;
    Qs[(q * 16 + h) * LDQ + r] = __float2bfloat16_rn(v);
  }
  float oacc[NTM][4];
#pragma unroll
  for (int i = 0; i < NTM; ++i) { oacc[i][0] = 0.f; oacc[i][1] = 0.f; oacc[i][2] = 0.f; oacc[i][3] = 0.f; }
  float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
  const int cw = R / RS, nt_o = cw >> 3, c0 = wr * cw;
  const bf16* cache = reinterpret_cast<const bf16*>(o.B);
  const int chunks = D >> 3;
  const bf16* Qw = Qs + (size_t)wq * 16 * LDQ;
  auto fetch_tile = [&](const int jt, bf16* dst) {       // rows beyond the range arrive as zeros
    for (int i = tid; i < TJ * chunks; i += nth) {
      const int row = i / chunks, c = i - row * chunks;
      const bool ok = jt + row < j1;
      cp_async16(dst + (size_t)row * LDQ + c * 8, cache + (size_t)(ok ? jt + row : j0) * o.ldr + c * 8, ok);
    }
    cp_async_commit();
  };
  if (j0 < j1) fetch_tile(j0, Ct0);
  int it = 0;
  for (int jt = j0; jt < j1; jt += TJ, ++it) {
    bf16* Ct = Ct0 + (size_t)(it & 1) * TJ * LDQ;
    if (jt + TJ < j1) {
      fetch_tile(jt + TJ, Ct0 + (size_t)((it + 1) & 1) * TJ * LDQ);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (active && jt < nk && jt + TJ > klo) {
      float s[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) { s[i][0] = 0.f; s[i][1] = 0.f; s[i][2] = 0.f; s[i][3] = 0.f; }
      {
        const int mi = lane >> 3, l7 = lane & 7;
        // ldmatrix lanes: A = 16 heads x 16 columns of the query (matrices: rows 0-7 / 8-15 at kk, then at kk + 8);
        // B = two key octets x 16 columns of the tile (matrices: octet nt at kk, kk + 8, octet nt + 1 at kk, kk + 8)
        const bf16* qa = Qw + (size_t)((mi & 1) * 8 + l7) * LDQ + (mi >> 1) * 8;
        const bf16* cb = Ct + (size_t)((mi >> 1) * 8 + l7) * LDQ + (mi & 1) * 8;
        for (int kk = 0; kk < D; kk += 16) {
          uint32_t a[4];
          ldmatrix_x4(a, qa + kk);
#pragma unroll
          for (int nt = 0; nt < 8; nt += 2) {
            if (nt * 8 < TJ) {
              uint32_t b[4];
              ldmatrix_x4(b, cb + (size_t)nt * 8 * LDQ + kk);
              mma16816(s[nt], a, b[0], b[1]);
              mma16816(s[nt + 1], a, b[2], b[3]);
            }
          }
        }
      }
      float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const int key = jt + nt * 8 + t * 2;
        const bool v0 = (nt * 8 < TJ) && key < nk && key >= klo, v1 = (nt * 8 < TJ) && key + 1 < nk && key + 1 >= klo;
        if (!v0) { s[nt][0] = -INFINITY; s[nt][2] = -INFINITY; }
        if (!v1) { s[nt][1] = -INFINITY; s[nt][3] = -INFINITY; }
        mx0 = fmaxf(mx0, fmaxf(s[nt][0], s[nt][1]));
        mx1 = fmaxf(mx1, fmaxf(s[nt][2], s[nt][3]));
      }
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1)); mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      const float mn0 = fmaxf(mrow[0], mx0), mn1 = fmaxf(mrow[1], mx1);
      const float u0 = mn0 == -INFINITY ? 0.f : mn0, u1 = mn1 == -INFINITY ? 0.f : mn1;
      const float al0 = mrow[0] == -INFINITY ? 0.f : expf(mrow[0] - u0), al1 = mrow[1] == -INFINITY ? 0.f : expf(mrow[1] - u1);
      float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        s[nt][0] = expf(s[nt][0] - u0); s[nt][1] = expf(s[nt][1] - u0);
        s[nt][2] = expf(s[nt][2] - u1); s[nt][3] = expf(s[nt][3] - u1);
        sum0 += s[nt][0] + s[nt][1];
        sum1 += s[nt][2] + s[nt][3];
      }
      sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1); sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
      sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1); sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
      lrow[0] = lrow[0] * al0 + sum0; lrow[1] = lrow[1] * al1 + sum1;
      mrow[0] = mn0; mrow[1] = mn1;
#pragma unroll
      for (int nt = 0; nt < NTM; ++nt) { oacc[nt][0] *= al0; oacc[nt][1] *= al0; oacc[nt][2] *= al1; oacc[nt][3] *= al1; }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks * 16 < TJ) {
          uint32_t ah[4], al[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const float p0 = s[2 * ks + (q >> 1)][(q & 1) * 2], p1 = s[2 * ks + (q >> 1)][(q & 1) * 2 + 1];
            const float h0f = bf16r(p0), h1f = bf16r(p1);
            ah[q] = pack_bf16(h0f, h1f);
            al[q] = pack_bf16(p0 - h0f, p1 - h1f);
          }
          const int mi = lane >> 3;
          const bf16* base = Ct + (size_t)(ks * 16 + (mi & 1) * 8 + (lane & 7)) * LDQ + c0 + (mi >> 1) * 8;
          // eight column octets at a time: their high-part MMAs, then their low-part ones, so that an accumulator's two MMAs
          // are eight apart and none waits for the one before it
#pragma unroll
          for (int nt0 = 0; nt0 < NTM; nt0 += 8) {
            uint32_t b[4][4];
#pragma unroll
            for (int q = 0; q < 4; ++q)
              if (nt0 + 2 * q < nt_o) ldmatrix_x4_trans(b[q], base + (nt0 + 2 * q) * 8);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
              const int nt = nt0 + 2 * q;
              if (nt < nt_o) mma16816(oacc[nt], ah, b[q][0], b[q][1]);
              if (nt + 1 < nt_o) mma16816(oacc[nt + 1], ah, b[q][2], b[q][3]);
            }
#pragma unroll
            for (int q = 0; q < 4; ++q) {
              const int nt = nt0 + 2 * q;
              if (nt < nt_o) mma16816(oacc[nt], al, b[q][0], b[q][1]);
              if (nt + 1 < nt_o) mma16816(oacc[nt + 1], al, b[q][2], b[q][3]);
            }
          }
        }
      }
    }
    __syncthreads();
  }
  if (!active) return;
  const float* sink = reinterpret_cast<const float*>(o.scale);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int h = h0 + g + half * 8;
    if (h >= H) continue;
    const float mr = mrow[half], lr = lrow[half];
    if (splits == 1) {
      float f = 1.f, den = lr;
      if (sink) {
        const float mm = fmaxf(mr, sink[h]);
        f = mr == -INFINITY ? 0.f : expf(mr - mm);
        den = lr * f + expf(sink[h] - mm);
      }
      float sc = f / den;
      if (o.res) sc *= sigmoid_f(reinterpret_cast<const float*>(o.res)[(size_t)m * o.m_begin + h]);
      float* c = reinterpret_cast<float*>(o.C) + (size_t)m * o.ldc + (size_t)h * R + c0;
#pragma unroll
      for (int nt = 0; nt < NTM; ++nt)
        if (nt < nt_o) { c[nt * 8 + t * 2] = oacc[nt][half * 2] * sc; c[nt * 8 + t * 2 + 1] = oacc[nt][half * 2 + 1] * sc; }
    } else {
      float* dst = reinterpret_cast<float*>(o.ws) + (((size_t)m * H + h) * splits + z) * (R + 2);
      if (wr == 0 && t == 0) { dst[0] = mr; dst[1] = lr; }
#pragma unroll
      for (int nt = 0; nt < NTM; ++nt)
        if (nt < nt_o) { dst[2 + c0 + nt * 8 + t * 2] = oacc[nt][half * 2]; dst[2 + c0 + nt * 8 + t * 2 + 1] = oacc[nt][half * 2 + 1]; }
    }
  }
}

// ===========================================================================================================================
// ABI 7 (kinds 24-29): dynamic-tanh norm, depth mix, xIELU, rotary cache append, cached softmax attention with windows / sinks /
// distance penalties / output gates, and recurrences with a matrix state per head (gated delta rule, state-space scan).
// ===========================================================================================================================

// what follows a finished f32 value of the residual stream: the stream itself, its bf16 copy, and the next norm's output
__device__ __forceinline__ void stream_out(const fq3c_op& o, const int m, const int c, const float v) {
  reinterpret_cast<float*>(o.C)[(size_t)m * o.ldc + c] = v;
  if (o.C2) reinterpret_cast<bf16*>(o.C2)[(size_t)m * o.ldc + c] = __float2bfloat16_rn(v);
  if (o.norm_out) {
    const float* w = reinterpret_cast<const float*>(o.norm_w);
    const float n = fmaf(tanhf(o.norm_eps * v), w[c], w[o.N + c]);
    if (o.flags & FQ3C_F32) reinterpret_cast<float*>(o.norm_out)[(size_t)m * o.norm_ld + c] = n;
    else reinterpret_cast<bf16*>(o.norm_out)[(size_t)m * o.norm_ld + c] = __float2bfloat16_rn(n);
  }
}

// grid (ceil(N / 256), M)
__global__ void __launch_bounds__(256) fq3s_dyt_kernel(const fq3c_op o) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, m = blockIdx.y;
  if (c >= o.N) return;
  float v = tanhf(o.f0 * reinterpret_cast<const float*>(o.A)[(size_t)m * o.lda + c]) * reinterpret_cast<const float*>(o.scale)[c];
  if (o.bias) v += reinterpret_cast<const float*>(o.bias)[c];
  if (o.flags & FQ3C_RESID) v += reinterpret_cast<const float*>(o.res)[(size_t)m * o.ldr + c];
  if (o.flags & FQ3C_OUT_F32) stream_out(o, m, c, v);
  else reinterpret_cast<bf16*>(o.C)[(size_t)m * o.ldc + c] = __float2bfloat16_rn(v);
}

// grid (ceil(N / 256), M)
__global__ void __launch_bounds__(256) fq3s_depth_mix_kernel(const fq3c_op o) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, m = blockIdx.y;
  if (c >= o.N) return;
  const float* a = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda + c;
  const float* w = reinterpret_cast<const float*>(o.p0);
  float v = 0.f;
  for (int j = 0; j < o.i0; ++j) v = fmaf(w[j], a[(size_t)j * (size_t)o.K], v);
  stream_out(o, m, c, v);
}

// grid (ceil(N / 256), M)
__global__ void __launch_bounds__(256) fq3s_xielu_kernel(const fq3c_op o) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, m = blockIdx.y;
  if (c >= o.N) return;
  const float* p = reinterpret_cast<const float*>(o.p0);
  const float ap = softplus_f(p[0]), aq = 0.5f + softplus_f(p[1]);
  const float z = reinterpret_cast<const float*>(o.A)[(size_t)m * o.lda + c];
  const float v = z > 0.f ? fmaf(ap * z, z, 0.5f * z) : fmaf(aq, expm1f(z) - z, 0.5f * z);
  if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[(size_t)m * o.ldc + c] = v;
  else reinterpret_cast<bf16*>(o.C)[(size_t)m * o.ldc + c] = __float2bfloat16_rn(v);
}

// the mean of the P rows of block b of a cache -> row b of its pooled rows, for columns c0, c0 + step, .. below c1
template <typename TC>
__device__ __forceinline__ void pool_run(const TC* cache, const int ld, TC* pooled, const int b, const int P, const int c0, const int c1, const int step) {
  for (int c = c0; c < c1; c += step) {
    const TC* src = cache + (size_t)b * P * ld + c;
    float sum = 0.f;
    for (int r = 0; r < P; ++r) sum += ldf<TC>(src + (size_t)r * ld);
    stf(pooled + (size_t)b * ld + c, sum / (float)P);
  }
}
// grid (M / P + 1, ceil(i1 * max(i2, cin) / 256), 2): z = 0 keys, 1 values
template <typename TC>
__global__ void __launch_bounds__(256) fq3s_pool_append_kernel(const fq3c_op o) {
  const int pos0 = o.p0 ? *reinterpret_cast<const int*>(o.p0) : 0, P = o.m_begin, b = pos0 / P + blockIdx.x;
  if ((b + 1) * P > pos0 + o.M) return;
  const int c = blockIdx.y * blockDim.x + threadIdx.x, n = o.i1 * (blockIdx.z ? o.cin : o.i2);
  if (blockIdx.z == 0) pool_run<TC>(reinterpret_cast<const TC*>(o.C), o.ldc, reinterpret_cast<TC*>(o.norm_out), b, P, c, min(n, c + 1), 1);
  else pool_run<TC>(reinterpret_cast<const TC*>(o.C2), o.ldr, reinterpret_cast<TC*>(o.ws), b, P, c, min(n, c + 1), 1);
}

// grid (M), up to THREADS threads (256, or 1024 for a few rows), a warp per query / key head.  Angles in f32: position (exact as a float below 2^24) times the frequency,
// full-range sincosf; cos and sin times the amplitude f1 when that is set.  With norm weights a head is first divided by its root
// mean square (eps f0) and multiplied by them; with FQ3C_UNIT it is divided only (a rotation keeps the root mean square, so it does
// not matter which comes first).  Queries in place, keys (read from `res` rows when given) into the cache.
// m_begin = P > 0: every run of P positions bP .. bP + P - 1 that the step completes leaves the mean of its P cached keys and values as
// row b of norm_out / ws.  A single row does it here (POOL; its block has just written the run's last row); more rows take
// fq3s_pool_append_kernel behind this launch.
template <typename TC, bool POOL = false, int THREADS = 256>
__global__ void __launch_bounds__(THREADS) fq3s_rot_append_kernel(const fq3c_op o) {
  const int m = blockIdx.x, H = o.i0, G = o.i1, d = o.i2, dv = o.cin, half = o.taps >> 1;
  const int pos = (o.p0 ? *reinterpret_cast<const int*>(o.p0) : 0) + m;
  float* row = const_cast<float*>(reinterpret_cast<const float*>(o.A)) + (size_t)m * o.lda;
  const float* krow = o.res ? reinterpret_cast<const float*>(o.res) + (size_t)m * o.norm_ld : row;
  const float* freq = reinterpret_cast<const float*>(o.B);
  const float* flo = reinterpret_cast<const float*>(o.p1);
  const float fp = (float)pos, amp = o.f1 != 0.f ? o.f1 : 1.f;
  // query temperature: grows with every f3 positions (the quotient of two integers below 2^24 never rounds up to the next integer)
  const float temp = o.f3 > 0.f ? fmaf(o.f2, logf(floorf((fp + 1.f) / o.f3) + 1.f), 1.f) : 1.f;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarp = blockDim.x >> 5;
  TC* kc = G > 0 ? reinterpret_cast<TC*>(o.C) + (size_t)pos * o.ldc : nullptr;
  for (int hh = warp; hh < H + G; hh += nwarp) {
    const bool isq = hh < H;
    const float* src = isq ? row + (size_t)hh * d : krow + o.K + (size_t)(hh - H) * d;
    const float* nw = reinterpret_cast<const float*>(isq ? o.scale : o.bias);
    const bool unit = nw || (o.flags & FQ3C_UNIT), normed = unit || (isq && o.f3 > 0.f);
    float rs = 1.f;
    if (unit) {
      float ss = 0.f;
      for (int c = lane; c < d; c += 32) ss = fmaf(src[c], src[c], ss);
      rs = 1.f / sqrtf(warp_sum(ss) / (float)d + o.f0);
    }
    if (isq) rs *= temp;
    float* qd = isq ? row + (size_t)hh * d : nullptr;
    TC* kd = isq ? nullptr : kc + (size_t)(hh - H) * d;
    const bool halves = (o.flags & FQ3C_ROT_HALF) != 0;      // pairs (i, i + half) instead of (2i, 2i + 1)
    for (int i = lane; i < half; i += 32) {
      float sn, cs;
      const float ang = fp * freq[i];
      sincosf(ang, &sn, &cs);
      // what the product (and, with p1, the frequency) lost to rounding turns the pair a little further: at large angles it would show
      float rest = fmaf(fp, freq[i], -ang);
      if (flo) rest = fmaf(fp, flo[i], rest);
      const float s1 = fmaf(cs, rest, sn), c1 = fmaf(-sn, rest, cs);
      sn = s1 * amp; cs = c1 * amp;
      const int ia = halves ? i : 2 * i, ib = halves ? i + half : 2 * i + 1;
      float a = src[ia], b = src[ib];
      if (normed) { a *= rs; b *= rs; }
      if (nw) { a *= nw[ia]; b *= nw[ib]; }
      const float x = a * cs - b * sn, y = b * cs + a * sn;
      if (isq) { qd[ia] = x; qd[ib] = y; }
      else { stf(kd + ia, x); stf(kd + ib, y); }
    }
    if (isq && !normed) continue;     // the rest of a query head stays as it is
    for (int c = 2 * half + lane; c < d; c += 32) {
      float v = normed ? src[c] * rs : src[c];
      if (nw) v *= nw[c];
      if (isq) qd[c] = v;
      else stf(kd + c, v);
    }
  }
  if (G <= 0 || dv <= 0) return;
  TC* vc = reinterpret_cast<TC*>(o.C2) + (size_t)pos * o.ldr;
  const float* v = krow + o.a_rows;
  for (int idx = threadIdx.x; idx < G * dv; idx += blockDim.x) stf(vc + idx, v[idx]);
  if (POOL && (pos + 1) % o.m_begin == 0) {
    __syncthreads();
    pool_run<TC>(reinterpret_cast<const TC*>(o.C), o.ldc, reinterpret_cast<TC*>(o.norm_out), pos / o.m_begin, o.m_begin, threadIdx.x, G * d, blockDim.x);
    pool_run<TC>(reinterpret_cast<const TC*>(o.C2), o.ldr, reinterpret_cast<TC*>(o.ws), pos / o.m_begin, o.m_begin, threadIdx.x, G * dv, blockDim.x);
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Softmax attention over a key / value cache on the CUDA cores, every sum in f32.  A block takes QB consecutive queries x the HG
// query heads of one key / value head (R = QB * HG rows that score the same staged key tile), 256 threads, online softmax over
// tiles of TJ keys; tiles that no row of the block can see (outside the window and beyond the kept first positions) are skipped.
// Pooled blocks (tap_off[1] = P > 0): the rows of the pooled caches C2 / norm_out (means of P positions each) are keys and values of the
// same softmax; position i sees the blocks that lie wholly before its window, i.e. the first (i - window + 1) / P.  Their tiles come first.
// grid (ceil(M / QB), key heads, splits).  One split finishes in place (sink, output gate); several leave (max, sum, out) per
// (row, split) in ws for fq3s_cache_attn_merge_kernel.
// Shared memory (f32): q [R][d], keys [TJ][d + 1], values [TJ][dv], p [R][TJ], out [R][dv], max / sum / rescale [3][R].
// ---------------------------------------------------------------------------------------------------------------------------
__host__ __device__ inline size_t cache_attn_smem(int R, int TJ, int d, int dv) {
  return sizeof(float) * ((size_t)R * d + (size_t)TJ * (d + 1) + (size_t)TJ * dv + (size_t)R * TJ + (size_t)R * dv + 3 * (size_t)R);
}
struct CacheAttnMask {
  int window, keep, chunk, pool;
  __device__ __forceinline__ int blocks(int i) const { return pool > 0 ? max(0, i - window + 1) / pool : 0; }
  __device__ __forceinline__ bool sees(int i, int j) const {
    return j <= i && (window <= 0 || i - j < window || j < keep) && (chunk <= 0 || j >= i - i % chunk);
  }
  // no query at position >= i sees a key below this
  __device__ __forceinline__ int lowest(int i) const {
    const int wlo = (window > 0 && keep <= 0) ? max(0, i - window + 1) : 0;
    return max(wlo, chunk > 0 ? i - i % chunk : 0);
  }
};
// rows [0, nvalid) of a cache tile into shared memory as f32 (the rest of the nrows as zeros): 16-byte loads, several in flight,
// where the rows allow them
__device__ __forceinline__ void ca_unpack(float* d, const uint4& u, const float*) {
  d[0] = __uint_as_float(u.x); d[1] = __uint_as_float(u.y); d[2] = __uint_as_float(u.z); d[3] = __uint_as_float(u.w);
}
__device__ __forceinline__ void ca_unpack(float* d, const uint4& u, const bf16*) {
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) { d[2 * i] = __uint_as_float(w[i] << 16); d[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
}
template <typename TC>
__device__ __forceinline__ void ca_stage_rows(float* dst, const int dld, const TC* src, const int sld, const int nvalid, const int nrows,
                                              const int cols, const int tid, const int nth) {
  constexpr int V = 16 / (int)sizeof(TC);
  if (cols % V == 0 && sld % V == 0 && !(reinterpret_cast<uintptr_t>(src) & 15)) {
    const int cpr = cols / V;
#pragma unroll 4
    for (int idx = tid; idx < nrows * cpr; idx += nth) {
      const int jj = idx / cpr, c = (idx - jj * cpr) * V;
      float* d = dst + (size_t)jj * dld + c;
      if (jj < nvalid) {
        const uint4 u = *reinterpret_cast<const uint4*>(src + (size_t)jj * sld + c);
        ca_unpack(d, u, src);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) d[i] = 0.f;
      }
    }
    return;
  }
  for (int idx = tid; idx < nrows * cols; idx += nth) {
    const int jj = idx / cols, c = idx - jj * cols;
    dst[(size_t)jj * dld + c] = jj < nvalid ? ldf<TC>(src + (size_t)jj * sld + c) : 0.f;
  }
}
template <typename TC, bool POOL = false>
__global__ void __launch_bounds__(256) fq3s_cache_attn_kernel(const fq3c_op o, const int QB, const int TJ, const int splits) {
  extern __shared__ float csm[];
  const int H = o.i0, G = o.i1, d = o.i2, dv = o.cin, HG = H / G, R = QB * HG;
  const int m0 = blockIdx.x * QB, g = blockIdx.y, z = blockIdx.z;
  const int nq = min(QB, o.M - m0);
  float* qs = csm;
  float* kt = qs + (size_t)R * d;
  float* vt = kt + (size_t)TJ * (d + 1);
  float* ps = vt + (size_t)TJ * dv;
  float* oa = ps + (size_t)R * TJ;
  float* mx = oa + (size_t)R * dv;
  float* ls = mx + R;
  float* al = ls + R;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nwarp = blockDim.x >> 5;
  const int P = o.p0 ? *reinterpret_cast<const int*>(o.p0) : 0;
  const CacheAttnMask mask{o.K, o.a_rows, o.tap_off[0], o.tap_off[1]};
  const int ifirst = P + m0, ilast = P + m0 + nq - 1;
  // the splits share the tiles: those of the pooled blocks, then the tokens' from the first one any query of the block can see
  const int npool = POOL ? mask.blocks(ilast) : 0, npt = (npool + TJ - 1) / TJ;
  const int tbeg = mask.lowest(ifirst) / TJ, total = npt + ilast / TJ + 1 - tbeg;
  const int per = (total + splits - 1) / splits;
  const int u0 = z * per, u1 = min(total, u0 + per);
  for (int idx = tid; idx < R * d; idx += blockDim.x) {
    const int r = idx / d, c = idx - r * d, qi = r / HG, hh = r - qi * HG;
    qs[idx] = qi < nq ? reinterpret_cast<const float*>(o.A)[(size_t)(m0 + qi) * o.lda + (size_t)(g * HG + hh) * d + c] : 0.f;
  }
  for (int idx = tid; idx < R * dv; idx += blockDim.x) oa[idx] = 0.f;
  for (int idx = tid; idx < R; idx += blockDim.x) { mx[idx] = -INFINITY; ls[idx] = 0.f; }
  const TC* kc = reinterpret_cast<const TC*>(o.B) + (size_t)g * d;
  const TC* vc = reinterpret_cast<const TC*>(o.p1) + (size_t)g * dv;
  const TC* kp = reinterpret_cast<const TC*>(o.C2) + (size_t)g * d;
  const TC* vp = reinterpret_cast<const TC*>(o.norm_out) + (size_t)g * dv;
  const float* r12 = reinterpret_cast<const float*>(o.bias);
  const float cap = o.f1, icap = o.f1 > 0.f ? 1.f / o.f1 : 0.f;
  for (int u = u0; u < u1; ++u) {
    const bool pooled = POOL && u < npt;
    const int j0 = (pooled ? u : tbeg + u - npt) * TJ, jn = min(TJ, (pooled ? npool : ilast + 1) - j0);
    // nothing of this tile is inside the widest window of the block (that of its first query) nor among the kept positions
    if (!pooled && mask.window > 0 && j0 + jn <= ifirst - mask.window + 1 && j0 >= mask.keep) continue;
    if (mask.chunk > 0 && j0 + jn <= ifirst - ifirst % mask.chunk) continue;
    __syncthreads();
    ca_stage_rows<TC>(kt, d + 1, (pooled ? kp : kc) + (size_t)j0 * o.ldr, o.ldr, jn, TJ, d, tid, blockDim.x);
    ca_stage_rows<TC>(vt, dv, (pooled ? vp : vc) + (size_t)j0 * o.taps, o.taps, jn, TJ, dv, tid, blockDim.x);
    __syncthreads();
    for (int idx = tid; idx < R * TJ; idx += blockDim.x) {
      const int r = idx / TJ, jj = idx - r * TJ, qi = r / HG, i = ifirst + qi, j = j0 + jj;
      float s = -INFINITY;
      if (qi < nq && jj < jn && (pooled ? j < mask.blocks(i) : mask.sees(i, j))) {
        const float* qv = qs + (size_t)r * d;
        const float* kv = kt + (size_t)jj * (d + 1);
        float acc = 0.f;
        for (int c = 0; c < d; ++c) acc = fmaf(qv[c], kv[c], acc);
        s = acc * o.f0;
        if (cap > 0.f) s = cap * tanhf(s * icap);
        if (r12) {
          const int h = g * HG + (r - qi * HG);
          s -= r12[h] * log1pf(r12[H + h] * (float)(i - j));
        }
      }
      ps[idx] = s;
    }
    __syncthreads();
    for (int r = warp; r < R; r += nwarp) {
      float tm = -INFINITY;
      for (int jj = lane; jj < TJ; jj += 32) tm = fmaxf(tm, ps[(size_t)r * TJ + jj]);
      tm = warp_max(tm);
      const float mo = mx[r], mn = fmaxf(mo, tm);
      float sum = 0.f;
      for (int jj = lane; jj < TJ; jj += 32) {
        const float s = ps[(size_t)r * TJ + jj];
        const float p = s == -INFINITY ? 0.f : expf(s - mn);
        ps[(size_t)r * TJ + jj] = p;
        sum += p;
      }
      sum = warp_sum(sum);
      if (lane == 0) {
        const float a = mo == -INFINITY ? 0.f : expf(mo - mn);     // mn is finite whenever mo is
        al[r] = a;
        ls[r] = ls[r] * a + sum;
        mx[r] = mn;
      }
    }
    __syncthreads();
    for (int idx = tid; idx < R * dv; idx += blockDim.x) {
      const int r = idx / dv, c = idx - r * dv;
      const float* p = ps + (size_t)r * TJ;
      float acc = oa[idx] * al[r];
      for (int jj = 0; jj < jn; ++jj) acc = fmaf(p[jj], vt[(size_t)jj * dv + c], acc);
      oa[idx] = acc;
    }
  }
  __syncthreads();
  const float* sink = reinterpret_cast<const float*>(o.scale);
  const float* gate = reinterpret_cast<const float*>(o.res);
  const bool entry = (o.flags & FQ3C_GATE_ENTRY) != 0;
  for (int idx = tid; idx < R * dv; idx += blockDim.x) {
    const int r = idx / dv, c = idx - r * dv, qi = r / HG, h = g * HG + (r - qi * HG), m = m0 + qi;
    if (qi >= nq) continue;
    if (splits > 1) {
      float* dst = reinterpret_cast<float*>(o.ws) + (((size_t)m * H + h) * splits + z) * (dv + 2);
      if (c == 0) { dst[0] = mx[r]; dst[1] = ls[r]; }
      dst[2 + c] = oa[idx];
      continue;
    }
    float f = 1.f, den = ls[r];
    if (sink) {
      const float mm = fmaxf(mx[r], sink[h]);
      f = mx[r] == -INFINITY ? 0.f : expf(mx[r] - mm);
      den = den * f + expf(sink[h] - mm);
    }
    float v = oa[idx] * f / den;
    if (gate) v *= sigmoid_f(gate[(size_t)m * o.col_mod + (entry ? h * dv + c : h)]);
    if (o.f2 != 0.f) v *= o.f2;
    if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[(size_t)m * o.ldc + (size_t)h * dv + c] = v;
    else reinterpret_cast<bf16*>(o.C)[(size_t)m * o.ldc + (size_t)h * dv + c] = __float2bfloat16_rn(v);
  }
}

// grid (M, H), 128 threads
__global__ void __launch_bounds__(128) fq3s_cache_attn_merge_kernel(const fq3c_op o, const int splits) {
  __shared__ float wsm[64];
  __shared__ float red[32];
  const int m = blockIdx.x, h = blockIdx.y, H = o.i0, dv = o.cin;
  const float* src = reinterpret_cast<const float*>(o.ws) + ((size_t)m * H + h) * splits * (dv + 2);
  const float* sink = reinterpret_cast<const float*>(o.scale);
  float mv = -INFINITY, lv = 0.f;
  if ((int)threadIdx.x < splits) { mv = src[(size_t)threadIdx.x * (dv + 2)]; lv = src[(size_t)threadIdx.x * (dv + 2) + 1]; }
  float mm = warp_max(mv);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = mm;
  __syncthreads();
  mm = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
  if (sink) mm = fmaxf(mm, sink[h]);
  const float w = mv == -INFINITY ? 0.f : expf(mv - mm);
  if ((int)threadIdx.x < splits) wsm[threadIdx.x] = w;
  float den = seq_block_sum(w * lv, red);
  if (sink) den += expf(sink[h] - mm);
  const bool entry = (o.flags & FQ3C_GATE_ENTRY) != 0;
  const float* gr = o.res ? reinterpret_cast<const float*>(o.res) + (size_t)m * o.col_mod : nullptr;
  const float gate = (gr && !entry) ? sigmoid_f(gr[h]) : 1.f;
  const float sc = gate * (o.f2 != 0.f ? o.f2 : 1.f) / den;
  for (int c = threadIdx.x; c < dv; c += blockDim.x) {
    float acc = 0.f;
#pragma unroll 16
    for (int s = 0; s < splits; ++s) acc = fmaf(wsm[s], src[(size_t)s * (dv + 2) + 2 + c], acc);
    float v = acc * sc;
    if (entry) v *= sigmoid_f(gr[(size_t)h * dv + c]);
    if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[(size_t)m * o.ldc + (size_t)h * dv + c] = v;
    else reinterpret_cast<bf16*>(o.C)[(size_t)m * o.ldc + (size_t)h * dv + c] = __float2bfloat16_rn(v);
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// The same attention on the tensor cores for bf16 caches and many queries (prompt portions).  The rows of an MMA tile are
// (query, head of the group) pairs: a block takes 64 / HG consecutive queries x the HG query heads of one key / value head = 64
// rows (128 for long portions; another multiple of 16 when HG does not divide 64), 16 per warp, which score the same staged key tile.  Key and value tiles of 64 positions arrive by cp.async into two
// buffers (one is read while the next arrives); tiles outside every window of the block and beyond the kept first positions are
// never fetched.  S [16 x 64] = Q K^T (m16n8k16, keys row-major as the B operand), then scale / cap / distance penalty / mask and
// the online softmax in f32 (fast exponential, logarithm and reciprocal: errors around 1e-6), then O [16 x dv] += P V with every weight as a bf16 pair p_hi + p_lo (two MMAs: 16 mantissa bits)
// and the value tile through ldmatrix.trans.  Queries are rounded to bf16 once, as a bf16 product rounds its operand.
// grid (ceil(M / (rows / HG)), key heads), 2 threads per row; the last queries (most keys) start first.
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int CM_TJ = 64;
// tanh through one fast exponential and one fast reciprocal (relative error around 1e-6: far below the bf16 operands' rounding,
// which is the precision this kernel serves; the 32-bit mode runs the CUDA-core kernel with the full-precision functions)
__device__ __forceinline__ float fast_tanh(float x) {
  const float e = __expf(2.f * fminf(fmaxf(x, -15.f), 15.f));
  return 1.f - __fdividef(2.f, e + 1.f);
}
__host__ __device__ inline size_t cache_attn_mma_smem(int rows, int d, int dv) { return 2 * ((size_t)rows * (d + 8) + 2 * (size_t)CM_TJ * (d + 8) + 2 * (size_t)CM_TJ * (dv + 8)); }
template <int NTM, bool POOL = false>      // POOL: tiles of pooled blocks in front of the tokens' (a variant of its own: the plain one compiles as it always did)
__global__ void __launch_bounds__(256) fq3s_cache_attn_mma_kernel(const fq3c_op o, const int ROWS) {
  extern __shared__ __align__(16) unsigned char cm_raw[];
  const int H = o.i0, G = o.i1, d = o.i2, dv = o.cin, HG = H / G, QBLK = ROWS / HG, LDK = d + 8, LDV = dv + 8;
  bf16* Qs = reinterpret_cast<bf16*>(cm_raw);            // [ROWS][LDK]
  bf16* Kt0 = Qs + (size_t)ROWS * LDK;                     // 2 x [CM_TJ][LDK]
  bf16* Vt0 = Kt0 + (size_t)2 * CM_TJ * LDK;             // 2 x [CM_TJ][LDV]
  const int tid = threadIdx.x, nth = blockDim.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int m0 = (gridDim.x - 1 - blockIdx.x) * QBLK, kvh = blockIdx.y;
  const int P = o.p0 ? *reinterpret_cast<const int*>(o.p0) : 0;
  const int nq = min(QBLK, o.M - m0), ifirst = P + m0, ilast = ifirst + nq - 1;
  const int W = o.K, keep = o.a_rows, chunk = o.tap_off[0];
  // pooled blocks position i sees, those any query of the block sees, and their tiles (numbered -npt .. -1)
  auto blocks = [&](const int i) { return POOL ? max(0, i - W + 1) / o.tap_off[1] : 0; };
  const int npool = blocks(ilast), npt = POOL ? (npool + CM_TJ - 1) / CM_TJ : 0;
  int nb[2] = {0, 0}, wblocks[2] = {0, 0};      // blocks this thread's two rows see; the first and the last row of its warp
  const float* A = reinterpret_cast<const float*>(o.A);
  if (o.lda % 4 == 0 && !(reinterpret_cast<uintptr_t>(A) & 15)) {      // 16-byte loads, four in flight per thread
    const int c4 = d >> 2;
#pragma unroll 4
    for (int i = tid; i < ROWS * c4; i += nth) {
      const int r = i / c4, c = (i - r * c4) * 4, qi = r / HG, hh = r - qi * HG;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (qi < nq) v = *reinterpret_cast<const float4*>(A + (size_t)(m0 + qi) * o.lda + (size_t)(kvh * HG + hh) * d + c);
      __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(Qs + (size_t)r * LDK + c);
      dst[0] = __floats2bfloat162_rn(v.x, v.y);
      dst[1] = __floats2bfloat162_rn(v.z, v.w);
    }
  } else {
    for (int i = tid; i < ROWS * d; i += nth) {
      const int r = i / d, c = i - r * d, qi = r / HG, hh = r - qi * HG;
      Qs[(size_t)r * LDK + c] = __float2bfloat16_rn(qi < nq ? A[(size_t)(m0 + qi) * o.lda + (size_t)(kvh * HG + hh) * d + c] : 0.f);
    }
  }
  // the two rows this thread holds of its warp's 16
  int qpos[2], head[2], clo[2];
  bool live[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = warp * 16 + g + e * 8, qi = r / HG;
    live[e] = qi < nq;
    qpos[e] = ifirst + qi;
    clo[e] = chunk > 0 ? qpos[e] - qpos[e] % chunk : 0;      // first key of the query's chunk
    head[e] = kvh * HG + (r - qi * HG);
  }
  const bool wactive = (warp * 16) / HG < nq;
  const int wfirst = ifirst + (warp * 16) / HG, wlast = ifirst + min(nq - 1, (warp * 16 + 15) / HG);
  const int ntiles = ilast / CM_TJ + 1;
  const int tkeep = W > 0 ? (keep + CM_TJ - 1) / CM_TJ : 0, tlo = W > 0 ? max(0, ifirst - W + 1) / CM_TJ : 0;
  const int tstart = chunk > 0 ? (ifirst - ifirst % chunk) / CM_TJ : 0;      // tiles below the first query's chunk: nobody sees them
  if (POOL) { nb[0] = live[0] ? blocks(qpos[0]) : 0; nb[1] = live[1] ? blocks(qpos[1]) : 0; wblocks[0] = blocks(wfirst); wblocks[1] = blocks(wlast); }
  auto next_tile = [&](int tt) { ++tt; if (POOL && tt < 0) return tt; if (tt < tstart) tt = tstart; if (W > 0 && tt >= tkeep && tt < tlo) tt = tlo; return tt; };
  const bf16* kc = reinterpret_cast<const bf16*>(o.B) + (size_t)kvh * d;
  const bf16* vc = reinterpret_cast<const bf16*>(o.p1) + (size_t)kvh * dv;
  const int kch = d >> 3, vch = dv >> 3;
  auto fetch_tile = [&](const int tt, const int buf) {       // rows beyond the last needed position arrive as zeros
    bf16* kd = Kt0 + (size_t)buf * CM_TJ * LDK;
    bf16* vd = Vt0 + (size_t)buf * CM_TJ * LDV;
    const bool pooled = POOL && tt < 0;
    const int j0 = (pooled ? tt + npt : tt) * CM_TJ, jend = pooled ? npool - 1 : ilast;
    const bf16* ks = pooled ? reinterpret_cast<const bf16*>(o.C2) + (size_t)kvh * d : kc;
    const bf16* vs = pooled ? reinterpret_cast<const bf16*>(o.norm_out) + (size_t)kvh * dv : vc;
    for (int i = tid; i < CM_TJ * kch; i += nth) {
      const int row = i / kch, c = i - row * kch;
      const bool ok = j0 + row <= jend;
      cp_async16(kd + (size_t)row * LDK + c * 8, ks + (size_t)(ok ? j0 + row : 0) * o.ldr + c * 8, ok);
    }
    for (int i = tid; i < CM_TJ * vch; i += nth) {
      const int row = i / vch, c = i - row * vch;
      const bool ok = j0 + row <= jend;
      cp_async16(vd + (size_t)row * LDV + c * 8, vs + (size_t)(ok ? j0 + row : 0) * o.taps + c * 8, ok);
    }
    cp_async_commit();
  };
  float oacc[NTM][4];
#pragma unroll
  for (int i = 0; i < NTM; ++i) { oacc[i][0] = 0.f; oacc[i][1] = 0.f; oacc[i][2] = 0.f; oacc[i][3] = 0.f; }
  float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
  const int nt_o = dv >> 3;
  const float* r12 = reinterpret_cast<const float*>(o.bias);
  const float cap = o.f1, icap = o.f1 > 0.f ? 1.f / o.f1 : 0.f;
  float r1v[2] = {0.f, 0.f}, r2v[2] = {0.f, 0.f};
  if (r12) { r1v[0] = r12[head[0]]; r1v[1] = r12[head[1]]; r2v[0] = r12[H + head[0]]; r2v[1] = r12[H + head[1]]; }
  const bf16* Qw = Qs + (size_t)warp * 16 * LDK;
  int tcur = next_tile(-1 - npt);
  if (tcur < ntiles) fetch_tile(tcur, 0);
  for (int it = 0; tcur < ntiles; ++it) {
    const int tn = next_tile(tcur);
    if (tn < ntiles) {
      fetch_tile(tn, (it + 1) & 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const bool pooled = POOL && tcur < 0;
    const int jt = (pooled ? tcur + npt : tcur) * CM_TJ;
    const bf16* Kt = Kt0 + (size_t)(it & 1) * CM_TJ * LDK;
    const bf16* Vt = Vt0 + (size_t)(it & 1) * CM_TJ * LDV;
    if (wactive && (pooled ? jt < wblocks[1] : jt <= wlast)) {
      float s[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) { s[i][0] = 0.f; s[i][1] = 0.f; s[i][2] = 0.f; s[i][3] = 0.f; }
      {
        const int mi = lane >> 3, l7 = lane & 7;
        const bf16* qa = Qw + (size_t)((mi & 1) * 8 + l7) * LDK + (mi >> 1) * 8;
        const bf16* cb = Kt + (size_t)((mi >> 1) * 8 + l7) * LDK + (mi & 1) * 8;
        for (int kk = 0; kk < d; kk += 16) {
          uint32_t a[4];
          ldmatrix_x4(a, qa + kk);
#pragma unroll
          for (int nt = 0; nt < 8; nt += 2) {
            uint32_t b[4];
            ldmatrix_x4(b, cb + (size_t)nt * 8 * LDK + kk);
            mma16816(s[nt], a, b[0], b[1]);
            mma16816(s[nt + 1], a, b[2], b[3]);
          }
        }
      }
      // a tile every row of the warp sees whole needs no per-score test (most tiles of a long portion)
      const bool whole = nq == QBLK && (pooled ? jt + CM_TJ <= wblocks[0]
                                               : jt + CM_TJ - 1 <= wfirst && (W <= 0 || wlast - jt < W) && (chunk <= 0 || jt >= wlast - wlast % chunk));
      int lo[2], hi[2];      // POOL: the keys of this tile each of the two rows sees lie in [lo, hi)
      if (POOL) {
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          lo[hf] = (pooled ? 0 : qpos[hf] - W + 1) - jt - t * 2;
          hi[hf] = (pooled ? nb[hf] : live[hf] ? qpos[hf] + 1 : 0) - jt - t * 2;
        }
      }
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = jt + nt * 8 + t * 2 + (e & 1), hf = e >> 1, i = qpos[hf];
          float v = -INFINITY;
          if (POOL) {
            const int at = nt * 8 + (e & 1);
            if (whole || (at >= lo[hf] && at < hi[hf])) {
              v = s[nt][e] * o.f0;
              if (cap > 0.f) v = cap * fast_tanh(v * icap);
            }
          } else if (whole || (live[hf] && key <= i && key >= clo[hf] && (W <= 0 || i - key < W || key < keep))) {
            v = s[nt][e] * o.f0;
            if (cap > 0.f) v = cap * fast_tanh(v * icap);
            if (r12) v -= r1v[hf] * __logf(fmaf(r2v[hf], (float)(i - key), 1.f));
          }
          s[nt][e] = v;
          mx[hf] = fmaxf(mx[hf], v);
        }
      }
      float al[2], u[2], sum[2] = {0.f, 0.f};
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        mx[hf] = fmaxf(mx[hf], __shfl_xor_sync(0xffffffffu, mx[hf], 1));
        mx[hf] = fmaxf(mx[hf], __shfl_xor_sync(0xffffffffu, mx[hf], 2));
        const float mn = fmaxf(mrow[hf], mx[hf]);
        u[hf] = mn == -INFINITY ? 0.f : mn;
        al[hf] = mrow[hf] == -INFINITY ? 0.f : expf(mrow[hf] - u[hf]);
        mrow[hf] = mn;
      }
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        s[nt][0] = __expf(s[nt][0] - u[0]); s[nt][1] = __expf(s[nt][1] - u[0]);
        s[nt][2] = __expf(s[nt][2] - u[1]); s[nt][3] = __expf(s[nt][3] - u[1]);
        sum[0] += s[nt][0] + s[nt][1];
        sum[1] += s[nt][2] + s[nt][3];
      }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        sum[hf] += __shfl_xor_sync(0xffffffffu, sum[hf], 1);
        sum[hf] += __shfl_xor_sync(0xffffffffu, sum[hf], 2);
        lrow[hf] = lrow[hf] * al[hf] + sum[hf];
      }
#pragma unroll
      for (int nt = 0; nt < NTM; ++nt) { oacc[nt][0] *= al[0]; oacc[nt][1] *= al[0]; oacc[nt][2] *= al[1]; oacc[nt][3] *= al[1]; }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        uint32_t ah[4], alo[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float p0 = s[2 * ks + (q >> 1)][(q & 1) * 2], p1 = s[2 * ks + (q >> 1)][(q & 1) * 2 + 1];
          const float h0f = bf16r(p0), h1f = bf16r(p1);
          ah[q] = pack_bf16(h0f, h1f);
          alo[q] = pack_bf16(p0 - h0f, p1 - h1f);
        }
        const int mi = lane >> 3;
        const bf16* base = Vt + (size_t)(ks * 16 + (mi & 1) * 8 + (lane & 7)) * LDV + (mi >> 1) * 8;
#pragma unroll
        for (int nt0 = 0; nt0 < NTM; nt0 += 8) {
          uint32_t b[4][4];
#pragma unroll
          for (int q = 0; q < 4; ++q)
            if (nt0 + 2 * q < nt_o) ldmatrix_x4_trans(b[q], base + (nt0 + 2 * q) * 8);
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int nt = nt0 + 2 * q;
            if (nt < nt_o) mma16816(oacc[nt], ah, b[q][0], b[q][1]);
            if (nt + 1 < nt_o) mma16816(oacc[nt + 1], ah, b[q][2], b[q][3]);
          }
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int nt = nt0 + 2 * q;
            if (nt < nt_o) mma16816(oacc[nt], alo, b[q][0], b[q][1]);
            if (nt + 1 < nt_o) mma16816(oacc[nt + 1], alo, b[q][2], b[q][3]);
          }
        }
      }
    }
    __syncthreads();
    tcur = tn;
  }
  const float* sink = reinterpret_cast<const float*>(o.scale);
  const float* gate = reinterpret_cast<const float*>(o.res);
  const bool entry = gate && (o.flags & FQ3C_GATE_ENTRY);
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    if (!live[hf]) continue;
    const int h = head[hf], m = qpos[hf] - P;
    float f = 1.f, den = lrow[hf];
    if (sink) {
      const float mm = fmaxf(mrow[hf], sink[h]);
      f = mrow[hf] == -INFINITY ? 0.f : expf(mrow[hf] - mm);
      den = den * f + expf(sink[h] - mm);
    }
    float sc = f / den;
    if (gate && !entry) sc *= sigmoid_f(gate[(size_t)m * o.col_mod + h]);
    if (o.f2 != 0.f) sc *= o.f2;
    const float* ge = entry ? gate + (size_t)m * o.col_mod + (size_t)h * dv : nullptr;
    const size_t at = (size_t)m * o.ldc + (size_t)h * dv;
#pragma unroll
    for (int nt = 0; nt < NTM; ++nt) {
      if (nt >= nt_o) continue;
      float v0 = oacc[nt][hf * 2] * sc, v1 = oacc[nt][hf * 2 + 1] * sc;
      if (entry) { v0 *= sigmoid_f(ge[nt * 8 + t * 2]); v1 *= sigmoid_f(ge[nt * 8 + t * 2 + 1]); }
      if (o.flags & FQ3C_OUT_F32) { reinterpret_cast<float*>(o.C)[at + nt * 8 + t * 2] = v0; reinterpret_cast<float*>(o.C)[at + nt * 8 + t * 2 + 1] = v1; }
      else *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf16*>(o.C) + at + nt * 8 + t * 2) = __floats2bfloat162_rn(v0, v1);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Recurrences with a matrix state S [dk, dv] per head.  Two launches: the per-token coefficients (and, for the delta rule, the unit
// query / key vectors) are computed row-parallel into ws; then one block per (head, 16 state columns) walks the tokens in order.
// A state column is held by eight lanes (dk / 8 consecutive entries each), so a token costs each lane dk / 8 multiply-adds per
// product plus three shuffles per reduction; tokens arrive in rounds staged through shared memory.
// ws row m (padded to a multiple of four floats): [unit q [G * dk] | unit k [G * dk] |] c1[H] | c2[H] [| q.k [G]]  (bracketed parts: delta
// rule only; delta rule: c1 = decay, c2 = write strength; scan: c1 = decay, c2 = dt)
// Four more modes share the walk.  Mode 2 (a decay per key channel and token): ws row m = alpha [H * dk], staged beside the token's
// key and query as a third vector.  Mode 3 (one fixed decay per head): no per-token coefficients at all, hence no first launch.
// Mode 4 (a forget gate per channel that also decides what is written): ws row m = silu(q) [H * dk] | 1 - f [H * dk] | f [H * dk], walked
// like mode 2.  Mode 5 (exponential gates under a running maximum): ws row m = e^(lf + m' - m) [H] | e^(li - m) [H] | e^(-m) [H]; the
// normaliser is one more state column (index dv) whose value entry is one.
// Up to MS_CH rows (decoding) the walk forms modes 4 and 5's coefficients itself as it stages the tokens: no first launch.
// ---------------------------------------------------------------------------------------------------------------------------
__host__ __device__ inline int mstate_ws_cols(int H, int G, int dk, bool delta) { return ((delta ? 2 * G * dk + G : 0) + 2 * H + 3) & ~3; }
__host__ __device__ inline int mstate_decay_cols(int H, int dk) { return (H * dk + 3) & ~3; }
__host__ __device__ inline int mstate_gate_cols(int H, int dk) { return (3 * H * dk + 3) & ~3; }      // mode 4
__host__ __device__ inline int mstate_max_cols(int H) { return (3 * H + 3) & ~3; }                    // mode 5
__host__ __device__ inline int mstate_ws_coef(int G, int dk, bool delta) { return delta ? 2 * G * dk : 0; }      // column of c1

constexpr int MS_MAX_RANK = 1024;     // inner size of the decay projection (mode 2)
constexpr int MS_PREP_ROWS = 8;       // rows per block of the first launch in mode 2
// grid (M), or (ceil(M / MS_PREP_ROWS)) in mode 2; 128 threads
__global__ void __launch_bounds__(128) fq3s_mstate_prep_kernel(const fq3c_op o) {
  const int m = blockIdx.x, H = o.i0, G = o.i1, dk = o.i2;
  if (o.taps == 2) {
    // z = U lat + b with the row's decay latent lat (m_begin entries of the raw rows, f32) and U = B [H * dk, m_begin] (bf16, F32: f32):
    // the up-projection is a few multiply-adds per channel, done here instead of in a product launch of its own.  A block takes
    // MS_PREP_ROWS rows, so that an entry of U is loaded once for all of them (grid = ceil(M / MS_PREP_ROWS) in this mode).
    // alpha = sigmoid(z)^f1, through its logarithm -f1 softplus(-z): no underflow of the sigmoid on the way.
    __shared__ float lat[MS_PREP_ROWS][MS_MAX_RANK];
    const int R = o.m_begin, m0 = blockIdx.x * MS_PREP_ROWS, nr = min(MS_PREP_ROWS, o.M - m0), cols = mstate_decay_cols(H, dk);
    for (int i = threadIdx.x; i < MS_PREP_ROWS * R; i += blockDim.x) {
      const int j = i / R, r = i - j * R;
      lat[j][r] = j < nr ? reinterpret_cast<const float*>(o.res)[(size_t)(m0 + j) * o.ldr + o.col_mod + r] : 0.f;
    }
    __syncthreads();
    float* a = reinterpret_cast<float*>(o.ws) + (size_t)m0 * cols;
    const float* zb = reinterpret_cast<const float*>(o.bias);
    for (int c = threadIdx.x; c < H * dk; c += blockDim.x) {
      float z[MS_PREP_ROWS];
#pragma unroll
      for (int j = 0; j < MS_PREP_ROWS; ++j) z[j] = zb ? zb[c] : 0.f;
      if (o.flags & FQ3C_F32) {
        const float* u = reinterpret_cast<const float*>(o.B) + (size_t)c * R;
        for (int r = 0; r < R; ++r) {
          const float uv = u[r];
#pragma unroll
          for (int j = 0; j < MS_PREP_ROWS; ++j) z[j] = fmaf(lat[j][r], uv, z[j]);
        }
      } else {
        const bf16* u = reinterpret_cast<const bf16*>(o.B) + (size_t)c * R;
        for (int r = 0; r < R; ++r) {
          const float uv = __bfloat162float(u[r]);
#pragma unroll
          for (int j = 0; j < MS_PREP_ROWS; ++j) z[j] = fmaf(lat[j][r], uv, z[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < MS_PREP_ROWS; ++j)
        if (j < nr) a[(size_t)j * cols + c] = expf(-o.f1 * softplus_f(-z[j]));
    }
    return;
  }
  const bool delta = o.taps == 0;
  float* w = reinterpret_cast<float*>(o.ws) + (size_t)m * mstate_ws_cols(H, G, dk, delta);
  float* cf = w + mstate_ws_coef(G, dk, delta);
  const float* raw = reinterpret_cast<const float*>(o.res) + (size_t)m * o.ldr;
  const float* alog = reinterpret_cast<const float*>(o.scale);
  const float* dtb = reinterpret_cast<const float*>(o.bias);
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    const float sp = softplus_f(raw[o.col_mod + h] + (dtb ? dtb[h] : 0.f));
    cf[h] = expf(-expf(alog[h]) * sp);
    cf[H + h] = delta ? sigmoid_f(raw[o.m_begin + h]) : sp;
  }
  if (!delta) return;
  const float* row = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarp = blockDim.x >> 5;
  const float qs = 1.f / sqrtf((float)dk);
  for (int v = warp; v < 2 * G; v += nwarp) {
    const bool isk = v >= G;
    const int g = isk ? v - G : v;
    const float* x = row + (isk ? o.K : 0) + (size_t)g * dk;
    float ss = 0.f;
    for (int c = lane; c < dk; c += 32) ss = fmaf(x[c], x[c], ss);
    ss = warp_sum(ss);
    const float f = (1.f / sqrtf(ss + 1e-6f)) * (isk ? 1.f : qs);
    float* dst = w + (size_t)v * dk;
    for (int c = lane; c < dk; c += 32) dst[c] = x[c] * f;
  }
  __syncthreads();
  for (int g = warp; g < G; g += nwarp) {          // q.k of the unit vectors: lets the scan read out through the state before the write
    const float* qn = w + (size_t)g * dk;
    const float* kn = qn + (size_t)G * dk;
    float dot = 0.f;
    for (int c = lane; c < dk; c += 32) dot = fmaf(qn[c], kn[c], dot);
    dot = warp_sum(dot);
    if (lane == 0) cf[2 * H + g] = dot;
  }
}

// mode 6: ws row m = unit q [G * dk] | unit k [G * dk] | decays [H * dk] | write strengths [H] | q.k [G].  A block takes MS_PREP_ROWS rows (ROWS:
// how many of them it computes, 1 in decoding) and one share of the columns (grid.y): two channels per thread of the decays' up-projection, or
// of the gate's, or, the last one, the unit vectors with their products and the write strengths.  The up-projections lie transposed [inner size,
// channels]: neighbouring threads load neighbouring entries, each once for all rows of the block, whose latents lie transposed in shared memory
// (sixteen-byte broadcasts).  Dynamic shared memory: 8 x the larger inner size.
__host__ __device__ inline int mstate_cdelta_cols(int H, int G, int dk) { return ((2 * G + H) * dk + H + G + 3) & ~3; }
template <int ROWS>
__device__ __forceinline__ void cdelta_up(const fq3c_op& o, const float* lat, const void* U, const int c, const int n, const int r0, const int R, float (&z)[2][ROWS]) {
#pragma unroll
  for (int j = 0; j < ROWS; ++j) { z[0][j] = 0.f; z[1][j] = 0.f; }
  const bool two = c + 1 < n;
  auto add = [&](const float u0, const float u1, const int r) {
    float l[ROWS];
    if (ROWS == 8) {
      const float4 a = *reinterpret_cast<const float4*>(lat + r * 8), b = *reinterpret_cast<const float4*>(lat + r * 8 + 4);
      l[0] = a.x; l[1 % ROWS] = a.y; l[2 % ROWS] = a.z; l[3 % ROWS] = a.w; l[4 % ROWS] = b.x; l[5 % ROWS] = b.y; l[6 % ROWS] = b.z; l[7 % ROWS] = b.w;
    } else l[0] = lat[r * 8];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) { z[0][j] = fmaf(l[j], u0, z[0][j]); z[1][j] = fmaf(l[j], u1, z[1][j]); }
  };
  if (o.flags & FQ3C_F32) {
    const float* u = reinterpret_cast<const float*>(U) + c;
#pragma unroll 8
    for (int r = r0; r < R; ++r) add(u[(size_t)r * n], two ? u[(size_t)r * n + 1] : 0.f, r);
    return;
  }
  const bf16* u = reinterpret_cast<const bf16*>(U) + c;
  if (n % 2 == 0 && !(reinterpret_cast<uintptr_t>(U) & 3)) {
#pragma unroll 16
    for (int r = r0; r < R; ++r) {
      const uint32_t w = __ldg(reinterpret_cast<const uint32_t*>(u + (size_t)r * n));
      add(__uint_as_float(w << 16), __uint_as_float(w & 0xffff0000u), r);
    }
  } else {
    for (int r = r0; r < R; ++r) add(__bfloat162float(u[(size_t)r * n]), two ? __bfloat162float(u[(size_t)r * n + 1]) : 0.f, r);
  }
}
// With `logs` the rows hold the base-2 logarithms of the decays alone (pitch round_up(H * dk, 4)), for the walk in blocks of tokens.
// channels per block: two per thread; with one row four threads share a pair
__host__ __device__ constexpr int cdelta_prep_channels(int rows) { return rows == 1 ? 128 : 512; }
template <int ROWS>
__global__ void __launch_bounds__(256) fq3s_mstate_cdelta_prep_kernel(const fq3c_op o, const bool logs) {
  extern __shared__ __align__(16) float cd_lat[];       // [inner size][8]
  const int H = o.i0, G = o.i1, dk = o.i2, m0 = blockIdx.x * MS_PREP_ROWS, nr = min(ROWS, o.M - m0), tid = threadIdx.x;
  constexpr int nth = 256, per = cdelta_prep_channels(ROWS);
  const int nd = (H * dk + per - 1) / per, ng = o.tap_off[2] > 0 ? (H * o.cin + per - 1) / per : 0, y = blockIdx.y;
  const int cols = logs ? (H * dk + 3) & ~3 : mstate_cdelta_cols(H, G, dk);
  const float* raw = reinterpret_cast<const float*>(o.res) + (size_t)m0 * o.ldr;
  float* w = reinterpret_cast<float*>(o.ws) + (size_t)m0 * cols;
  if (y < nd + ng) {
    const bool decay = y < nd;
    const int R = o.tap_off[decay ? 0 : 2], lcol = decay ? o.col_mod : o.tap_off[1], c = (decay ? y : y - nd) * per + (tid % (per / 2)) * 2;
    const int n = H * (decay ? dk : o.cin);
    for (int i = tid; i < ROWS * R; i += nth) {
      const int j = i / R, r = i - j * R;
      cd_lat[r * 8 + j] = j < nr ? raw[(size_t)j * o.ldr + lcol + r] : 0.f;
    }
    __syncthreads();
    float z[2][ROWS];
    if (ROWS == 1) {         // one row: quarters of the inner size side by side, added through shared memory
      const int q = tid / (per / 2), len = (R + 3) / 4;
      if (c < n) cdelta_up<ROWS>(o, cd_lat, decay ? o.B : o.p1, c, n, min(R, q * len), min(R, (q + 1) * len), z);
      else z[0][0] = z[1][0] = 0.f;
      __shared__ float2 part[256];
      part[tid] = make_float2(z[0][0], z[1][0]);
      __syncthreads();
      if (q > 0 || c >= n) return;
#pragma unroll
      for (int e = 1; e < 4; ++e) { const float2 p = part[e * (per / 2) + tid]; z[0][0] += p.x; z[1][0] += p.y; }
    } else {
      if (c >= n) return;
      cdelta_up<ROWS>(o, cd_lat, decay ? o.B : o.p1, c, n, 0, R, z);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int ce = c + e;
      if (ce >= n) break;
      if (decay) {
        const float db = reinterpret_cast<const float*>(o.bias)[ce], rate = expf(reinterpret_cast<const float*>(o.scale)[ce / dk]);
#pragma unroll
        for (int j = 0; j < ROWS; ++j) z[e][j] = -rate * softplus_f(z[e][j] + db);
#pragma unroll
        for (int j = 0; j < ROWS; ++j) z[e][j] = logs ? 1.4426950408889634f * z[e][j] : expf(z[e][j]);
      }
    }
    float* d = decay ? w + (logs ? 0 : 2 * G * dk) + c : reinterpret_cast<float*>(o.norm_out) + (size_t)m0 * o.norm_ld + c;
    const int ld = decay ? cols : o.norm_ld;
    const bool pairs = c + 1 < n && ld % 2 == 0 && !(reinterpret_cast<uintptr_t>(d) & 7);
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
      if (j >= nr) break;
      if (pairs) *reinterpret_cast<float2*>(d + (size_t)j * ld) = make_float2(z[0][j], z[1][j]);
      else { d[(size_t)j * ld] = z[0][j]; if (c + 1 < n) d[(size_t)j * ld + 1] = z[1][j]; }
    }
    return;
  }
  float* cf = w + (2 * G + H) * dk;
  for (int i = tid; i < nr * H; i += nth) {
    const int j = i / H, h = i - j * H;
    cf[(size_t)j * cols + h] = sigmoid_f(raw[(size_t)j * o.ldr + o.m_begin + h]);
  }
  const int warp = tid >> 5, lane = tid & 31;
  const float qs = 1.f / sqrtf((float)dk);
  for (int i = warp; i < nr * G; i += nth >> 5) {          // a warp per (row, group): both unit vectors and their product
    const int j = i / G, g = i - j * G;
    const float* q = reinterpret_cast<const float*>(o.A) + (size_t)(m0 + j) * o.lda + (size_t)g * dk;
    const float* k = q + o.K;
    float sq = 0.f, sk = 0.f, qk = 0.f;
    for (int c = lane; c < dk; c += 32) { const float a = q[c], b = k[c]; sq = fmaf(a, a, sq); sk = fmaf(b, b, sk); }
    const float fq = qs / sqrtf(warp_sum(sq) + 1e-6f), fk = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
    float* d = w + (size_t)j * cols + (size_t)g * dk;
    for (int c = lane; c < dk; c += 32) {
      const float a = q[c] * fq, b = k[c] * fk;
      d[c] = a; d[(size_t)G * dk + c] = b;
      qk = fmaf(a, b, qk);
    }
    qk = warp_sum(qk);
    if (lane == 0) cf[(size_t)j * cols + H + g] = qk;
  }
}

constexpr int MS_CH = 16;     // tokens staged per round

// mode 4, one channel: q raw, z the gate's logit, l the lower bound; 1 - f is formed from the mirrored sigmoid, not by a subtraction
__device__ __forceinline__ void forget_coeffs(const float q, const float z, const float l, float& sq, float& in, float& f) {
  const float u = 1.f - l;
  sq = q / (1.f + expf(-q));
  in = u * sigmoid_f(-z);
  f = fmaf(u, sigmoid_f(z), l);
}
// grid (M, ceil(H * dk / 256)): ws row m of mode 4
__global__ void __launch_bounds__(256) fq3s_mstate_gate_kernel(const fq3c_op o) {
  const int m = blockIdx.x, n = o.i0 * o.i2, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= n) return;
  const float* raw = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda;
  float* w = reinterpret_cast<float*>(o.ws) + (size_t)m * mstate_gate_cols(o.i0, o.i2);
  forget_coeffs(raw[c], raw[o.col_mod + c], reinterpret_cast<const float*>(o.scale)[c], w[c], w[n + c], w[2 * n + c]);
}
// mode 5, one token of a head: log input gate and log forget gate from their logits, capped by c tanh(. / c)
__device__ __forceinline__ void log_gates(const float zi, const float zf, const float cap, float& li, float& lf) {
  li = cap * tanhf(zi / cap);
  lf = -softplus_f(-cap * tanhf(zf / cap));
}
// grid (H), MM_THREADS threads: ws rows of mode 5.  m_t = max(lf_t + m_(t-1), li_t) over a run of tokens is the map m -> max(a + m, b) with
// a = sum lf and b = the run's own maximum, so every thread folds a share of the rows, the block scans the maps, and every thread walks its
// share from the maximum it starts with.  The coefficients are differences of the very maxima the walk keeps: whatever the maxima's
// rounding, numerator, normaliser and e^(-m) refer to the same one.  Rows are fetched MM_BATCH at a time, ahead of the stores.
constexpr int MM_THREADS = 512, MM_BATCH = 4;
__global__ void __launch_bounds__(MM_THREADS) fq3s_mstate_max_kernel(const fq3c_op o) {
  __shared__ float sa[MM_THREADS], sb[MM_THREADS];
  const int h = blockIdx.x, H = o.i0, tid = threadIdx.x, per = (o.M + MM_THREADS - 1) / MM_THREADS, t0 = min(o.M, tid * per), t1 = min(o.M, t0 + per);
  const int cols = mstate_max_cols(H);
  const float* raw = reinterpret_cast<const float*>(o.res) + h;
  float* w = reinterpret_cast<float*>(o.ws) + h;
  float a = 0.f, b = -INFINITY;
  for (int t = t0; t < t1; t += MM_BATCH) {
    float li[MM_BATCH], lf[MM_BATCH];
#pragma unroll
    for (int q = 0; q < MM_BATCH; ++q) {
      const float* r = raw + (size_t)min(t + q, t1 - 1) * o.ldr;
      li[q] = __ldg(r + o.col_mod);
      lf[q] = __ldg(r + o.m_begin);
    }
#pragma unroll
    for (int q = 0; q < MM_BATCH; ++q) {
      if (t + q >= t1) break;
      log_gates(li[q], lf[q], o.f1, li[q], lf[q]);
      float* c = w + (size_t)(t + q) * cols;
      c[0] = lf[q]; c[H] = li[q];
      a += lf[q];
      b = fmaxf(b + lf[q], li[q]);
    }
  }
  sa[tid] = a; sb[tid] = b;
  for (int d = 1; d < MM_THREADS; d <<= 1) {      // inclusive scan of the maps, earlier shares applied first
    __syncthreads();
    float pa = 0.f, pb = -INFINITY;
    if (tid >= d) { pa = sa[tid - d]; pb = sb[tid - d]; }
    __syncthreads();
    if (tid >= d) { sb[tid] = fmaxf(sa[tid] + pb, sb[tid]); sa[tid] += pa; }
  }
  __syncthreads();
  float m = reinterpret_cast<const float*>(o.scale)[h];
  if (tid > 0) m = fmaxf(sa[tid - 1] + m, sb[tid - 1]);
  for (int t = t0; t < t1; t += MM_BATCH) {
    float li[MM_BATCH], lf[MM_BATCH];
#pragma unroll
    for (int q = 0; q < MM_BATCH; ++q) {
      const float* c = w + (size_t)min(t + q, t1 - 1) * cols;
      lf[q] = c[0]; li[q] = c[H];
    }
#pragma unroll
    for (int q = 0; q < MM_BATCH; ++q) {
      if (t + q >= t1) break;
      float* c = w + (size_t)(t + q) * cols;
      const float mn = fmaxf(lf[q] + m, li[q]);
      c[0] = expf(lf[q] + m - mn);
      c[H] = expf(li[q] - mn);
      c[2 * H] = expf(-mn);
      m = mn;
    }
  }
  if (t1 == o.M && t0 < t1) reinterpret_cast<float*>(const_cast<void*>(o.p1))[h] = m;
}
constexpr int MS_COLS = 16;   // state columns per block (eight lanes each), times the columns a lane holds
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
// two f32 values side by side: one instruction multiplies (adds) both, each rounded as the scalar operation rounds
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float a, float b) { f32x2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b)); return r; }
__device__ __forceinline__ float lo2(f32x2 v) { float a, b; asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); return a; }
__device__ __forceinline__ float hi2(f32x2 v) { float a, b; asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); return b; }
// PACKED false: the same two operations as scalar instructions (for code that is bound by registers or shared memory, not by issue)
template <bool PACKED>
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  if (!PACKED) return pack2(fmaf(lo2(a), lo2(b), lo2(c)), fmaf(hi2(a), hi2(b), hi2(c)));
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
template <bool PACKED>
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  if (!PACKED) return pack2(lo2(a) * lo2(b), hi2(a) * hi2(b));
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
// floats per staging buffer: (k, q) or (B, C) (and the decays) [CH][NV][8 slices of RPT + 4] | v [CH][columns] | coefficients [CH][4]
__host__ __device__ constexpr int mstate_ch(int cpt) { return MS_CH / cpt; }
__host__ __device__ constexpr int mstate_buf_floats(int rpt, int nv = 2, int cpt = 1) {
  return mstate_ch(cpt) * (nv * 8 * (rpt + 4) + MS_COLS * cpt + 4);
}
// grid (ceil(dv / 16), H), 128 threads: thread = (column tid / 8 of the tile, lane-of-eight tid % 8).  A lane holds RPT consecutive
// rows of its state column (RPT * 8 >= dk; rows beyond dk stay zero: their key / query entries are zero padding), reads its slice
// of the token's key and query with 16-byte shared-memory loads (slices are padded apart by four floats: no bank conflicts),
// and a product is finished by three shuffles.  The next round's tokens arrive by cp.async while the current round is walked.
// NV = 3 (modes 2 and 4): a third staged vector per token, the decays of the head's key channels.  GATED: modes 4 (NV = 3) and 5 (NV = 2).
//
// A long run of rows of a recurrence whose decay does not depend on the state (modes 1-5) is cut into pieces of `piece` rows
// (grid.z) and walked twice.  phase 1: every piece but the last starts from zero and leaves its own contribution S_loc in
// X[z + 1] and the product of its decays per state row in P[z]; fq3s_mstate_carry_kernel then turns X into the states the pieces
// start from (X[0] = the carried state, X[z + 1] = P[z] X[z] + S_loc[z]); phase 3: every piece walks again from X[z] and writes
// the outputs, the last one also the next state.  phase 0: one pass over all rows (short runs, decoding, the delta rule).
//
// CPT = 2 (pieces of long runs, where blocks are plenty): a lane holds two state columns, so a token's vectors are read from shared memory
// once for both; rounds of eight tokens keep the blocks small.  Warps without a live column only stage.
//
// CDELTA (NV = 3): the delta rule with a decay per key channel (mode 6), one pass.  With S' = diag(g) S: u = beta (v - S'^T k) and
// o = S'^T q + u (q . k), so both products run in the pass that decays the state, with one round of shuffles.
template <int RPT, int NV = 2, bool GATED = false, int CPT = 1, bool CDELTA = false>
__global__ void __launch_bounds__(128) fq3s_mstate_scan_kernel(const fq3c_op o, const int phase, const int piece, float* X, float* P) {
  extern __shared__ __align__(16) float msm[];
  constexpr int SL = RPT + 4, ROW = 8 * SL, CH = mstate_ch(CPT), COLS = MS_COLS * CPT;
  constexpr bool PK = NV == 2;      // with three staged vectors the walk is bound by shared memory, and pairs only cost registers
  const int H = o.i0, G = o.i1, dk = o.i2, dv = o.cin, h = blockIdx.y, g = h / (H / G);
  const bool delta = !GATED && NV == 2 && CPT == 1 && o.taps == 0, fixed = !GATED && NV == 2 && o.taps == 3;
  const bool gates = GATED && NV == 3, memory = GATED && NV == 2;
  const bool direct = GATED && o.M <= MS_CH;      // the coefficients are formed here
  const int sv = memory ? dv + 1 : dv;                  // state columns
  const int wc = CDELTA ? mstate_cdelta_cols(H, G, dk) : NV == 3 ? (gates ? mstate_gate_cols(H, dk) : mstate_decay_cols(H, dk)) : memory ? mstate_max_cols(H) : mstate_ws_cols(H, G, dk, delta);
  const int tid = threadIdx.x, sub = tid & 7, cl = tid >> 3;      // this lane's columns: blockIdx.x * COLS + cl (+ MS_COLS)
  const bool wlive = blockIdx.x * COLS + (cl & ~3) < sv;           // the warp (four neighbouring columns) has one
  int col[CPT];
  bool live[CPT];
#pragma unroll
  for (int j = 0; j < CPT; ++j) { col[j] = blockIdx.x * COLS + cl + j * MS_COLS; live[j] = col[j] < sv; }
  const int zc = blockIdx.z, tb = phase == 0 ? 0 : zc * piece, te = phase == 0 ? o.M : min(o.M, tb + piece);
  const bool last_piece = phase == 0 || te == o.M;
  constexpr int per = mstate_buf_floats(RPT, NV, CPT);
  {   // the padding between and behind the slices stays zero for the whole launch (only the token rows that will be used)
    const int used = min(te - tb, CH) * NV * ROW;
    for (int i = tid; i < 2 * used; i += 128) msm[(i < used ? 0 : per - used) + i] = 0.f;
  }
  f32x2 S[CPT][RPT / 2];
  f32x2 Pd[NV == 3 ? RPT / 2 : 1];   // phase 1: the product of the piece's decays (per state row, or one number per head)
#pragma unroll
  for (int r = 0; r < (NV == 3 ? RPT / 2 : 1); ++r) Pd[r] = pack2(1.f, 1.f);
  const size_t hstate = (size_t)dk * sv;
  const float* st = phase == 3 ? X + ((size_t)zc * H + h) * hstate : reinterpret_cast<const float*>(o.p0) + (size_t)h * hstate;
#pragma unroll
  for (int j = 0; j < CPT; ++j)
#pragma unroll
    for (int r = 0; r < RPT / 2; ++r) {
      const int i = sub * RPT + 2 * r;
      const bool ok = phase != 1 && live[j];
      S[j][r] = pack2(ok && i < dk ? st[(size_t)i * sv + col[j]] : 0.f, ok && i + 1 < dk ? st[(size_t)(i + 1) * sv + col[j]] : 0.f);
    }
  const float D = (o.taps == 1 && o.B) ? reinterpret_cast<const float*>(o.B)[h] : 0.f;
  const float* wsb = reinterpret_cast<const float*>(o.ws);
  const float* rows = reinterpret_cast<const float*>(o.A);
  const bool qkv_rows = delta || NV == 3 || fixed || memory;       // layout (q | k | v) of the delta rule: queries at column 0, values at a_rows
  const int vcol = (qkv_rows ? o.a_rows : 0) + h * dv;
  __syncthreads();
  // keys then queries (B then C) of this head's group, as columns of the rows they are staged from
  const bool staged_ws = delta || gates || CDELTA;      // keys and queries come from the first launch's rows
  const float* vsrc = staged_ws ? wsb : rows;
  const int vstride = staged_ws ? wc : o.lda, off0 = (staged_ws ? G * dk : o.K) + g * dk, off1 = ((delta || qkv_rows) ? 0 : o.a_rows) + g * dk;
  const int offa = (CDELTA ? 2 * G * dk : gates ? 2 * H * dk : 0) + h * dk;      // the decays' columns (NV == 3)
  const int cfo = CDELTA ? (2 * G + H) * dk : mstate_ws_coef(G, dk, delta);
  const bool vec = dk % 4 == 0 && vstride % 4 == 0 && off0 % 4 == 0 && off1 % 4 == 0 && !(reinterpret_cast<uintptr_t>(vsrc) & 15) &&
                   (NV < 3 || (wc % 4 == 0 && offa % 4 == 0 && !(reinterpret_cast<uintptr_t>(wsb) & 15)));
  const float fixed_c1 = fixed ? reinterpret_cast<const float*>(o.scale)[h] : 0.f;
  auto fetch = [&](const int t0, float* buf) {
    const int nt = min(CH, te - t0);
    float* kq = buf;
    float* vs = kq + CH * NV * ROW;
    float* cf = vs + CH * COLS;
    if (NV == 3 && direct) {      // few rows: formed from the raw projections as they are staged
      const float* low = reinterpret_cast<const float*>(o.scale) + h * dk;
      for (int idx = tid; idx < nt * dk; idx += 128) {
        const int tt = idx / dk, c = idx - tt * dk, at = (c / RPT) * SL + (c % RPT);
        const float* r = rows + (size_t)(t0 + tt) * o.lda + h * dk + c;
        float* d = kq + tt * NV * ROW + at;
        forget_coeffs(r[0], r[o.col_mod], low[c], d[ROW], d[0], d[(NV - 1) * ROW]);
      }
    } else if (vec) {        // 16-byte copies: four consecutive entries never straddle a lane's slice (RPT is a multiple of four)
      const int n4 = dk >> 2;
      for (int idx = tid; idx < nt * n4; idx += 128) {
        const int tt = idx / n4, c = (idx - tt * n4) * 4, at = (c / RPT) * SL + (c % RPT);
        const float* sr = vsrc + (size_t)(t0 + tt) * vstride;
        cp_async16(kq + tt * NV * ROW + at, sr + off0 + c, true);
        cp_async16(kq + tt * NV * ROW + ROW + at, sr + off1 + c, true);
        if (NV == 3) cp_async16(kq + tt * NV * ROW + 2 * ROW + at, wsb + (size_t)(t0 + tt) * wc + offa + c, true);
      }
    } else {
      for (int tt = 0; tt < nt; ++tt) {
        const float* sr = vsrc + (size_t)(t0 + tt) * vstride;
        for (int c = tid; c < dk; c += 128) {
          const int at = (c / RPT) * SL + (c % RPT);
          cp_async4(kq + tt * NV * ROW + at, sr + off0 + c);
          cp_async4(kq + tt * NV * ROW + ROW + at, sr + off1 + c);
          if (NV == 3) cp_async4(kq + tt * NV * ROW + 2 * ROW + at, wsb + (size_t)(t0 + tt) * wc + offa + c);
        }
      }
    }
    for (int idx = tid; idx < nt * COLS; idx += 128) {
      const int tt = idx / COLS, c = blockIdx.x * COLS + (idx % COLS);
      if (c < dv) cp_async4(vs + idx, rows + (size_t)(t0 + tt) * o.lda + vcol + c);
      else if (memory && c == dv) vs[idx] = 1.f;
    }
    if (memory && direct) {       // few rows: a lane per token, the running maximum handed from lane to lane
      if (tid < 32) {
        float li = 0.f, lf = 0.f, m = reinterpret_cast<const float*>(o.scale)[h], mine = m, next = m;
        if (tid < nt) {
          const float* r = reinterpret_cast<const float*>(o.res) + (size_t)(t0 + tid) * o.ldr + h;
          log_gates(r[o.col_mod], r[o.m_begin], o.f1, li, lf);
        }
        for (int tt = 0; tt < nt; ++tt) {
          const float mn = fmaxf(__shfl_sync(0xffffffffu, lf, tt) + m, __shfl_sync(0xffffffffu, li, tt));
          if (tt == tid) { mine = m; next = mn; }
          m = mn;
        }
        if (tid < nt) { cf[tid * 4] = expf(lf + mine - next); cf[tid * 4 + 1] = expf(li - next); cf[tid * 4 + 2] = expf(-next); }
        if (tid == 0 && blockIdx.x == 0) reinterpret_cast<float*>(const_cast<void*>(o.p1))[h] = m;
      }
    } else if (CDELTA) {       // write strength and q . k
      for (int idx = tid; idx < nt * 2; idx += 128) {
        const int tt = idx >> 1, which = idx & 1;
        cp_async4(cf + tt * 4 + which, wsb + (size_t)(t0 + tt) * wc + cfo + (which ? H + g : h));
      }
    } else if (NV < 3 && !fixed)
      for (int idx = tid; idx < nt * 3; idx += 128) {
        const int tt = idx / 3, which = idx - tt * 3;
        const float* sr = wsb + (size_t)(t0 + tt) * wc + cfo;
        if (which < 2) cp_async4(cf + tt * 4 + which, sr + which * H + h);
        else if (delta || memory) cp_async4(cf + tt * 4 + 2, sr + 2 * H + g);
      }
    cp_async_commit();
  };
  fetch(tb, msm);
  int it = 0;
  for (int t0 = tb; t0 < te; t0 += CH, ++it) {
    const int nt = min(CH, te - t0);
    if (t0 + CH < te) {
      fetch(t0 + CH, msm + ((it + 1) & 1) * per);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* kq = msm + (it & 1) * per;
    const float* vs = kq + CH * NV * ROW;
    const float* cf = vs + CH * COLS;
#pragma unroll CPT
    for (int tt = 0; tt < (wlive ? nt : 0); ++tt) {
      const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(kq + tt * NV * ROW + sub * SL);      // four entries: two pairs
      const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(kq + tt * NV * ROW + ROW + sub * SL);
      float v[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) v[j] = vs[tt * COLS + cl + j * MS_COLS];
      f32x2 os[CPT][2];            // four chains, so that a product's sum is not one long dependent row of multiply-adds
#pragma unroll
      for (int j = 0; j < CPT; ++j) { os[j][0] = 0ull; os[j][1] = 0ull; }
      // a finished product: its four chains, then the eight lanes of the column
      auto total = [&](const f32x2 (&c)[2]) {
        float x = (lo2(c[0]) + hi2(c[0])) + (lo2(c[1]) + hi2(c[1]));
        x += __shfl_xor_sync(0xffffffffu, x, 1);
        x += __shfl_xor_sync(0xffffffffu, x, 2);
        x += __shfl_xor_sync(0xffffffffu, x, 4);
        return x;
      };
      float* orow = reinterpret_cast<float*>(o.C) + (size_t)(t0 + tt) * o.ldc + (size_t)h * dv;
      if (CDELTA) {
        const ulonglong2* a4 = reinterpret_cast<const ulonglong2*>(kq + tt * NV * ROW + 2 * ROW + sub * SL);
        f32x2 ks[2] = {0ull, 0ull};
        ulonglong2 kv[RPT / 4];
#pragma unroll
        for (int r = 0; r < RPT / 4; ++r) {
          kv[r] = k4[r];
          const ulonglong2 qv = q4[r], av = a4[r];
          S[0][2 * r] = mul2<true>(av.x, S[0][2 * r]);
          S[0][2 * r + 1] = mul2<true>(av.y, S[0][2 * r + 1]);
          ks[0] = fma2<true>(kv[r].x, S[0][2 * r], ks[0]);
          ks[1] = fma2<true>(kv[r].y, S[0][2 * r + 1], ks[1]);
          os[0][0] = fma2<true>(qv.x, S[0][2 * r], os[0][0]);
          os[0][1] = fma2<true>(qv.y, S[0][2 * r + 1], os[0][1]);
        }
        float kt = (lo2(ks[0]) + hi2(ks[0])) + (lo2(ks[1]) + hi2(ks[1])), qt = (lo2(os[0][0]) + hi2(os[0][0])) + (lo2(os[0][1]) + hi2(os[0][1]));
        kt += __shfl_xor_sync(0xffffffffu, kt, 1); qt += __shfl_xor_sync(0xffffffffu, qt, 1);
        kt += __shfl_xor_sync(0xffffffffu, kt, 2); qt += __shfl_xor_sync(0xffffffffu, qt, 2);
        kt += __shfl_xor_sync(0xffffffffu, kt, 4); qt += __shfl_xor_sync(0xffffffffu, qt, 4);
        const float u = cf[tt * 4] * (v[0] - kt);
        const f32x2 uu = pack2(u, u);
#pragma unroll
        for (int r = 0; r < RPT / 4; ++r) {
          S[0][2 * r] = fma2<true>(kv[r].x, uu, S[0][2 * r]);
          S[0][2 * r + 1] = fma2<true>(kv[r].y, uu, S[0][2 * r + 1]);
        }
        if (live[0] && sub == 0) orow[col[0]] = fmaf(u, cf[tt * 4 + 1], qt);
        continue;
      }
      if (NV == 3) {      // S <- diag(alpha) S + k v^T, o = f0 S^T q
        const ulonglong2* a4 = reinterpret_cast<const ulonglong2*>(kq + tt * NV * ROW + 2 * ROW + sub * SL);
        f32x2 vv[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) vv[j] = pack2(v[j], v[j]);
        if (phase == 1) {
#pragma unroll
          for (int r = 0; r < RPT / 4; ++r) {
            const ulonglong2 kv = k4[r], av = a4[r];
#pragma unroll
            for (int j = 0; j < CPT; ++j) {
              S[j][2 * r] = fma2<PK>(av.x, S[j][2 * r], mul2<PK>(kv.x, vv[j]));
              S[j][2 * r + 1] = fma2<PK>(av.y, S[j][2 * r + 1], mul2<PK>(kv.y, vv[j]));
            }
            constexpr int PR = NV == 3 ? 1 : 0;     // (this branch only runs with NV == 3; the index stays legal in the other instantiation)
            Pd[PR * (2 * r)] = mul2<PK>(Pd[PR * (2 * r)], av.x);
            Pd[PR * (2 * r + 1)] = mul2<PK>(Pd[PR * (2 * r + 1)], av.y);
          }
          continue;
        }
#pragma unroll
        for (int r = 0; r < RPT / 4; ++r) {
          const ulonglong2 kv = k4[r], qv = q4[r], av = a4[r];
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            S[j][2 * r] = fma2<PK>(av.x, S[j][2 * r], mul2<PK>(kv.x, vv[j]));
            S[j][2 * r + 1] = fma2<PK>(av.y, S[j][2 * r + 1], mul2<PK>(kv.y, vv[j]));
            os[j][0] = fma2<PK>(qv.x, S[j][2 * r], os[j][0]);
            os[j][1] = fma2<PK>(qv.y, S[j][2 * r + 1], os[j][1]);
          }
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          const float ot = total(os[j]);
          if (live[j] && sub == 0) orow[col[j]] = ot * o.f0;
        }
        continue;
      }
      const float c1 = fixed ? fixed_c1 : cf[tt * 4], c2 = fixed ? o.f0 : cf[tt * 4 + 1];
      const f32x2 cc = pack2(c1, c1);
      if (delta) {
        // both products with the stored state in one pass and one round of shuffles: with S' = c1 S + k u^T,
        // S'^T q = c1 S^T q + u (k . q), and u = c2 (v - c1 S^T k); k . q comes with the token
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          f32x2 ks[2] = {0ull, 0ull};
          ulonglong2 kv[RPT / 4];
#pragma unroll
          for (int r = 0; r < RPT / 4; ++r) {
            kv[r] = k4[r];
            const ulonglong2 qv = q4[r];
            ks[0] = fma2<PK>(kv[r].x, S[j][2 * r], ks[0]);
            ks[1] = fma2<PK>(kv[r].y, S[j][2 * r + 1], ks[1]);
            os[j][0] = fma2<PK>(qv.x, S[j][2 * r], os[j][0]);
            os[j][1] = fma2<PK>(qv.y, S[j][2 * r + 1], os[j][1]);
          }
          float kt = (lo2(ks[0]) + hi2(ks[0])) + (lo2(ks[1]) + hi2(ks[1])), qt = (lo2(os[j][0]) + hi2(os[j][0])) + (lo2(os[j][1]) + hi2(os[j][1]));
          kt += __shfl_xor_sync(0xffffffffu, kt, 1); qt += __shfl_xor_sync(0xffffffffu, qt, 1);
          kt += __shfl_xor_sync(0xffffffffu, kt, 2); qt += __shfl_xor_sync(0xffffffffu, qt, 2);
          kt += __shfl_xor_sync(0xffffffffu, kt, 4); qt += __shfl_xor_sync(0xffffffffu, qt, 4);
          const float u = c2 * (v[j] - c1 * kt);
          const f32x2 uu = pack2(u, u);
#pragma unroll
          for (int r = 0; r < RPT / 4; ++r) {
            S[j][2 * r] = fma2<PK>(kv[r].x, uu, mul2<PK>(cc, S[j][2 * r]));
            S[j][2 * r + 1] = fma2<PK>(kv[r].y, uu, mul2<PK>(cc, S[j][2 * r + 1]));
          }
          if (live[j] && sub == 0) orow[col[j]] = fmaf(u, cf[tt * 4 + 2], c1 * qt);
        }
        continue;
      }
      f32x2 dx[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) { const float x = c2 * v[j]; dx[j] = pack2(x, x); }
      if (phase == 1) {
#pragma unroll
        for (int r = 0; r < RPT / 4; ++r) {
          const ulonglong2 bv = k4[r];
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            S[j][2 * r] = fma2<PK>(cc, S[j][2 * r], mul2<PK>(bv.x, dx[j]));
            S[j][2 * r + 1] = fma2<PK>(cc, S[j][2 * r + 1], mul2<PK>(bv.y, dx[j]));
          }
        }
        Pd[0] = mul2<PK>(Pd[0], cc);
        continue;
      }
#pragma unroll
      for (int r = 0; r < RPT / 4; ++r) {
        const ulonglong2 bv = k4[r], qv = q4[r];
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          S[j][2 * r] = fma2<PK>(cc, S[j][2 * r], mul2<PK>(bv.x, dx[j]));
          S[j][2 * r + 1] = fma2<PK>(cc, S[j][2 * r + 1], mul2<PK>(bv.y, dx[j]));
          os[j][0] = fma2<PK>(qv.x, S[j][2 * r], os[j][0]);
          os[j][1] = fma2<PK>(qv.y, S[j][2 * r + 1], os[j][1]);
        }
      }
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        float ot = total(os[j]);
        if (memory) {
          ot *= o.f0;
          if (col[j] == dv && sub == 0)       // the normaliser's column: what the head's read-out is divided by
            reinterpret_cast<float*>(o.norm_out)[(size_t)(t0 + tt) * o.norm_ld + h] = fmaxf(fabsf(ot), cf[tt * 4 + 2]) + o.norm_eps;
          if (col[j] < dv && sub == 0) orow[col[j]] = ot;
        } else {
          ot = fmaf(D, v[j], ot);
          if (live[j] && sub == 0) orow[col[j]] = ot;
        }
      }
    }
    __syncthreads();
  }
  if (phase == 1) {       // this piece's own contribution becomes the next piece's start (after the carry pass); its decay product
    float* nx = X + ((size_t)(zc + 1) * H + h) * hstate;
#pragma unroll
    for (int j = 0; j < CPT; ++j)
#pragma unroll
      for (int r = 0; r < RPT; ++r) { const int i = sub * RPT + r; if (live[j] && i < dk) nx[(size_t)i * sv + col[j]] = r & 1 ? hi2(S[j][r / 2]) : lo2(S[j][r / 2]); }
    if (blockIdx.x == 0 && cl == 0) {
      float* pz = P + ((size_t)zc * H + h) * dk;
#pragma unroll
      for (int r = 0; r < RPT; ++r) { const int i = sub * RPT + r; if (i < dk) pz[i] = NV == 3 && (r & 1) ? hi2(Pd[NV == 3 ? r / 2 : 0]) : lo2(Pd[NV == 3 ? r / 2 : 0]); }
    }
    return;
  }
  if (!last_piece) return;
  float* nst = reinterpret_cast<float*>(o.C2) + (size_t)h * hstate;
#pragma unroll
  for (int j = 0; j < CPT; ++j)
#pragma unroll
    for (int r = 0; r < RPT; ++r) { const int i = sub * RPT + r; if (live[j] && i < dk) nst[(size_t)i * sv + col[j]] = r & 1 ? hi2(S[j][r / 2]) : lo2(S[j][r / 2]); }
}

// grid (ceil(H * dk * sv / 256)), sv state columns: X[0] = the carried state; X[z + 1] = P[z] X[z] + X[z + 1] for the pieces in order.
__global__ void __launch_bounds__(256) fq3s_mstate_carry_kernel(const fq3c_op o, const int pieces, float* X, const float* P, const int sv) {
  const size_t n = (size_t)o.i0 * o.i2 * sv, e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= n) return;
  const size_t hi = e / sv;        // (head, state row)
  float R = reinterpret_cast<const float*>(o.p0)[e];
  X[e] = R;
  for (int z = 0; z + 1 < pieces; ++z) {
    R = fmaf(P[(size_t)z * o.i0 * o.i2 + hi], R, X[(size_t)(z + 1) * n + e]);
    X[(size_t)(z + 1) * n + e] = R;
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Both delta rules over many rows, in blocks of CD_C tokens, every sum in f32.  Inside a block that starts from the state S0, with b_t the sum of
// the decays' logarithms from the block's first token to token t (per key channel; one number per head in mode 0) and G_t = e^(b_t),
//   S_t = diag(G_t) S0 + sum_(s <= t) (k_s e^(b_t - b_s)) u_s^T
//   u_t = beta_t (v_t - S0^T (G_t k_t) - sum_(s < t) A_ts u_s),   A_ts = sum_c k_t k_s e^(b_t - b_s)
//   o_t = S0^T (G_t q_t) + sum_(s <= t) B_ts u_s,                 B_ts = sum_c q_t k_s e^(b_t - b_s)
// so with the unit lower triangle I + diag(beta) A and T = (I + diag(beta) A)^-1 diag(beta):
//   U = T (V - Kt S0),   O = Qt S0 + B U,   S <- diag(G_last) S0 + Kb^T U,   Kt = G_t k_t, Qt = G_t q_t, Kb = k_s e^(b_last - b_s).
// Every exponent is a sum of decays between two tokens, hence never positive; the sums are kept as two floats, so that a difference of two large
// ones is as good as the sum it stands for.  Three launches: the decays' logarithms row by row (fq3s_mstate_cdelta_prep_kernel; mode 0: none), the
// records [Kt | Qt | Kb | G_last | T | B] of all (block, head) pairs at once, and one walk over the blocks per (head, DVT state columns): three
// small dense products per block of tokens instead of a chain of dependent steps per token.  Tokens beyond the last row are empty (k = q = v = 0,
// beta = 0, no decay).
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int CD_C = 16;           // tokens per block
constexpr int CD_TP = CD_C + 4;    // pitch of T and B
constexpr int CD_TILES = CD_C / 2 * (CD_C / 2 + 1) / 2, CD_REC_THREADS = (CD_TILES * 4 + 31) / 32 * 32;      // 2 x 2 tiles of (t, s) pairs, four threads each
constexpr int CD_MIN_ROWS = 32;    // fewer rows are walked token by token
constexpr int CD_MAX_DK = 256;
__host__ __device__ constexpr int cd_rows(int dk) { return (dk + 31) & ~31; }       // state rows, padded with zeros
__host__ __device__ constexpr int cd_pitch(int dk) { return cd_rows(dk) + 4; }
__host__ __device__ constexpr int cd_record(int dk) { return 3 * CD_C * cd_pitch(dk) + cd_rows(dk) + 2 * CD_C * CD_TP; }      // floats, a multiple of four
__host__ __device__ inline long long cd_log_floats(int M, int H, int dk, bool channels) { return channels ? (long long)M * ((H * dk + 3) & ~3) : 0; }
__host__ __device__ inline long long cd_ws_floats(int M, int H, int dk, bool channels) {
  return cd_log_floats(M, H, dk, channels) + (long long)((M + CD_C - 1) / CD_C) * H * cd_record(dk);
}
constexpr float LOG2E_F = 1.4426950408889634f;
__device__ __forceinline__ float pow2_f(const float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
// grid (blocks of tokens, H), CD_REC_THREADS threads; dynamic shared memory: sums (two floats), q and k, [CD_C][pitch] each
__global__ void __launch_bounds__(CD_REC_THREADS) fq3s_cdelta_record_kernel(const fq3c_op o) {
  extern __shared__ __align__(16) float cr[];
  __shared__ float beta[CD_C], N[CD_C][CD_C], fq[CD_C], fk[CD_C];
  const int H = o.i0, G = o.i1, dk = o.i2, h = blockIdx.y, g = h / (H / G), t0 = blockIdx.x * CD_C, tid = threadIdx.x;
  const int D = cd_rows(dk), P = cd_pitch(dk), nt = min(CD_C, o.M - t0);
  const bool channels = o.taps == 6;
  float* bh = cr;
  float* bl = bh + CD_C * P;
  float* qs = bl + CD_C * P;
  float* ks = qs + CD_C * P;
  const float* raw = reinterpret_cast<const float*>(o.res) + (size_t)t0 * o.ldr;
  const float* rows = reinterpret_cast<const float*>(o.A) + (size_t)t0 * o.lda;
  const int lp = (H * dk + 3) & ~3;
  if (tid < CD_C) beta[tid] = tid < nt ? sigmoid_f(raw[(size_t)tid * o.ldr + o.m_begin + h]) : 0.f;
  const float rate = channels ? 0.f : LOG2E_F * expf(reinterpret_cast<const float*>(o.scale)[h]);
  const float dtb = (!channels && o.bias) ? reinterpret_cast<const float*>(o.bias)[h] : 0.f;
  for (int c = tid; c < D; c += CD_REC_THREADS) {
    float hi = 0.f, lo = 0.f, l[CD_C];
#pragma unroll
    for (int t = 0; t < CD_C; ++t) {
      const bool ok = t < nt && c < dk;
      l[t] = !ok ? 0.f : channels ? reinterpret_cast<const float*>(o.ws)[(size_t)(t0 + t) * lp + h * dk + c]
                                  : -rate * softplus_f(raw[(size_t)t * o.ldr + o.col_mod + h] + dtb);
      qs[t * P + c] = ok ? rows[(size_t)t * o.lda + g * dk + c] : 0.f;
      ks[t * P + c] = ok ? rows[(size_t)t * o.lda + o.K + g * dk + c] : 0.f;
    }
#pragma unroll
    for (int t = 0; t < CD_C; ++t) {       // the exact sum of two floats is again two floats; the small part collects
      const float x = fmaxf(l[t], -1000.f), s = hi + x, bb = s - hi;
      lo += (hi - (s - bb)) + (x - bb);
      hi = s;
      bh[t * P + c] = hi;
      bl[t * P + c] = lo;
    }
  }
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31;
  for (int v = warp; v < 2 * CD_C; v += CD_REC_THREADS / 32) {
    const float* x = (v < CD_C ? qs : ks) + (v & (CD_C - 1)) * P;
    float ss = 0.f;
    for (int c = lane; c < dk; c += 32) ss = fmaf(x[c], x[c], ss);
    ss = warp_sum(ss);
    if (lane == 0) (v < CD_C ? fq : fk)[v & (CD_C - 1)] = (v < CD_C ? 1.f / sqrtf((float)dk) : 1.f) / sqrtf(ss + 1e-6f);
  }
  __syncthreads();
  float* rec = reinterpret_cast<float*>(o.ws) + cd_log_floats(o.M, H, dk, channels) + ((size_t)blockIdx.x * H + h) * cd_record(dk);
  for (int i = tid; i < CD_C * (D >> 2); i += CD_REC_THREADS) {
    const int t = i / (D >> 2), c = (i - t * (D >> 2)) * 4, at = t * P + c;
    const float4 hi = ld4(bh + at), lo = ld4(bl + at), eh = ld4(bh + (CD_C - 1) * P + c), el = ld4(bl + (CD_C - 1) * P + c);
    float4 q = ld4(qs + at), k = ld4(ks + at);
    q.x *= fq[t]; q.y *= fq[t]; q.z *= fq[t]; q.w *= fq[t];
    k.x *= fk[t]; k.y *= fk[t]; k.z *= fk[t]; k.w *= fk[t];
    *reinterpret_cast<float4*>(qs + at) = q;
    *reinterpret_cast<float4*>(ks + at) = k;
    const float4 d = make_float4(pow2_f(hi.x), pow2_f(hi.y), pow2_f(hi.z), pow2_f(hi.w));
    *reinterpret_cast<float4*>(rec + at) = make_float4(k.x * d.x, k.y * d.y, k.z * d.z, k.w * d.w);
    *reinterpret_cast<float4*>(rec + CD_C * P + at) = make_float4(q.x * d.x, q.y * d.y, q.z * d.z, q.w * d.w);
    *reinterpret_cast<float4*>(rec + 2 * CD_C * P + at) =
        make_float4(k.x * pow2_f((eh.x - hi.x) + (el.x - lo.x)), k.y * pow2_f((eh.y - hi.y) + (el.y - lo.y)),
                    k.z * pow2_f((eh.z - hi.z) + (el.z - lo.z)), k.w * pow2_f((eh.w - hi.w) + (el.w - lo.w)));
    if (t == CD_C - 1) *reinterpret_cast<float4*>(rec + 3 * CD_C * P + c) = d;
  }
  __syncthreads();
  float* Tm = rec + 3 * CD_C * P + D;
  float* Bm = Tm + CD_C * CD_TP;
  if (tid < CD_TILES * 4) {       // 2 x 2 pairs (t, s): rows 2 ti and next, columns 2 si and next; a quarter of the channels per thread
    const int tile = tid >> 2;
    int ti = (int)((sqrtf(8.f * (float)tile + 1.f) - 1.f) * 0.5f);
    while ((ti + 1) * (ti + 2) / 2 <= tile) ++ti;
    while (ti * (ti + 1) / 2 > tile) --ti;
    const int si = tile - ti * (ti + 1) / 2;
    const unsigned lanes = (warp + 1) * 32 <= CD_TILES * 4 ? 0xffffffffu : (1u << (CD_TILES * 4 % 32)) - 1u;      // the last warp has fewer
    float a[2][2] = {{0.f, 0.f}, {0.f, 0.f}}, b[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
    for (int c = (tid & 3) * 4; c < D; c += 16) {
      float4 ht[2], lt[2], kt[2], qt[2];
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int at = (2 * ti + x) * P + c;
        ht[x] = ld4(bh + at); lt[x] = ld4(bl + at); kt[x] = ld4(ks + at); qt[x] = ld4(qs + at);
      }
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const int at = (2 * si + y) * P + c;
        const float4 hs = ld4(bh + at), ls = ld4(bl + at), k = ld4(ks + at);
#pragma unroll
        for (int x = 0; x < 2; ++x) {      // (above the diagonal the exponent is positive and may overflow: not stored)
          const float e0 = k.x * pow2_f((ht[x].x - hs.x) + (lt[x].x - ls.x)), e1 = k.y * pow2_f((ht[x].y - hs.y) + (lt[x].y - ls.y));
          const float e2 = k.z * pow2_f((ht[x].z - hs.z) + (lt[x].z - ls.z)), e3 = k.w * pow2_f((ht[x].w - hs.w) + (lt[x].w - ls.w));
          a[x][y] = fmaf(kt[x].x, e0, a[x][y]); b[x][y] = fmaf(qt[x].x, e0, b[x][y]);
          a[x][y] = fmaf(kt[x].y, e1, a[x][y]); b[x][y] = fmaf(qt[x].y, e1, b[x][y]);
          a[x][y] = fmaf(kt[x].z, e2, a[x][y]); b[x][y] = fmaf(qt[x].z, e2, b[x][y]);
          a[x][y] = fmaf(kt[x].w, e3, a[x][y]); b[x][y] = fmaf(qt[x].w, e3, b[x][y]);
        }
      }
    }
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        a[x][y] += __shfl_xor_sync(lanes, a[x][y], 1); b[x][y] += __shfl_xor_sync(lanes, b[x][y], 1);
        a[x][y] += __shfl_xor_sync(lanes, a[x][y], 2); b[x][y] += __shfl_xor_sync(lanes, b[x][y], 2);
        const int t = 2 * ti + x, s = 2 * si + y;
        if ((tid & 3) == 2 * x + y) {        // one of the tile's four threads keeps it
          if (s <= t) {
            N[t][s] = beta[t] * a[x][y];
            Bm[t * CD_TP + s] = b[x][y];
          }
          if (s != t) Tm[(s < t ? s : t) * CD_TP + (s < t ? t : s)] = 0.f, Bm[(s < t ? s : t) * CD_TP + (s < t ? t : s)] = 0.f;
        }
      }
  }
  __syncthreads();
  if (tid < CD_C) {       // column tid of T by forward substitution
    float x[CD_C];
#pragma unroll
    for (int t = 0; t < CD_C; ++t) {
      float v = t == tid ? beta[t] : 0.f;
#pragma unroll
      for (int s = 0; s < t; ++s) v = fmaf(-N[t][s], x[s], v);
      x[t] = v;
      if (t >= tid) Tm[t * CD_TP + tid] = v;
    }
  }
}

// set by a kernel whose bounded wait for its own copy ran out; its outputs are then NaN
__device__ int seq_wait_error;
// true when the barrier's phase completed, false when the limit ran out (about a second)
__device__ __forceinline__ bool mbar_wait_bounded(const uint32_t bar, const uint32_t parity) {
  for (int i = 0; i < (1 << 20); ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if (i > 64) __nanosleep(256);
  }
  return false;
}
// grid (ceil(dv / DVT), H), 160 threads: four warps compute, the fifth asks for the records, one bulk copy per block of tokens, one block ahead.
// The state tile [D rows, DVT columns] lives in registers (four rows x two columns x RQ per thread) and, as the operand of the next block's
// products, transposed in shared memory.  [Kt; Qt] S0: a warp takes a quarter of the state rows for all 2 CD_C x DVT sums (a lane: rows r, r + 8,
// r + 16, r + 24 and four columns; with eight columns the half-warps split the quarter once more and exchange halves of their sums), the quarters
// are added where the sums are used.  U and O: a lane per (token, column).
constexpr int CD_WALK_THREADS = 160;
template <int DVT>
__host__ __device__ constexpr int cd_walk_floats(int dk) {
  return 2 * cd_record(dk) + DVT * cd_pitch(dk) + 4 * 2 * CD_C * (DVT + 1) + DVT * CD_TP + 4;
}
template <int DVT, int RQ>
__global__ void __launch_bounds__(CD_WALK_THREADS, 1) fq3s_cdelta_walk_kernel(const fq3c_op o) {
  extern __shared__ __align__(128) float cw[];
  __shared__ __align__(8) unsigned long long full[2];
  constexpr int NCP = DVT / 2, QS = 128 / NCP, CG = DVT / 4, KH = 4 / CG, PP = DVT + 1, JW = DVT / 4;
  const int H = o.i0, dk = o.i2, dv = o.cin, h = blockIdx.y, j0 = blockIdx.x * DVT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = cd_rows(dk), P = cd_pitch(dk), REC = cd_record(dk), nblk = (o.M + CD_C - 1) / CD_C;
  float* St = cw + 2 * REC;                          // [DVT][P]
  float* Xs = St + DVT * P;                          // [DVT][CD_TP]: V - Kt S0, then U
  float* Pp = Xs + DVT * CD_TP;                      // [4][2 CD_C][PP]
  const float* recs = reinterpret_cast<const float*>(o.ws) + cd_log_floats(o.M, H, dk, o.taps == 6) + (size_t)h * REC;
  auto fetch = [&](const int n) {       // one thread
    const uint32_t bar = smem_u32(&full[n & 1]);
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"((uint32_t)REC * 4u) : "memory");
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(cw + (n & 1) * REC)),
                 "l"(recs + (size_t)n * H * REC), "r"((uint32_t)REC * 4u), "r"(bar)
                 : "memory");
  };
  if (tid == 128) {
    mbar_init(smem_u32(&full[0]), 1);
    mbar_init(smem_u32(&full[1]), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    fetch(0);
  }
  __syncthreads();             // the barriers are initialised
  if (warp == 4) {
    for (int n = 0; n < nblk; ++n) {
      if (__syncthreads_or(0)) return;       // the four warps gave up
      if (lane == 0 && n + 1 < nblk) fetch(n + 1);
      __syncthreads();
      __syncthreads();
    }
    return;
  }
  // this thread's part of the state: rows rq + q QS (quads), columns 2 cp, 2 cp + 1
  const int cp = tid % NCP, rq = tid / NCP;
  f32x2 S[RQ][2][2];          // [quad][column][row pair]
  const float* st = reinterpret_cast<const float*>(o.p0) + (size_t)h * dk * dv;
#pragma unroll
  for (int q = 0; q < RQ; ++q)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int r = (rq + q * QS) * 4, c = j0 + 2 * cp + j;
      float v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = (r + e < dk && c < dv) ? st[(size_t)(r + e) * dv + c] : 0.f;
      S[q][j][0] = pack2(v[0], v[1]);
      S[q][j][1] = pack2(v[2], v[3]);
      if (r < D) *reinterpret_cast<float4*>(St + (2 * cp + j) * P + r) = make_float4(v[0], v[1], v[2], v[3]);
    }
  // this thread's (token, column) pairs of U and O: token lane % 16, columns warp JW + lane / 16 (+ 2)
  const int t = lane & (CD_C - 1), jb = warp * JW + (lane >> 4);
  const float* vrow = reinterpret_cast<const float*>(o.A) + o.a_rows + (size_t)h * dv + j0;
  float vn[JW / 2];
  auto load_v = [&](const int n) {
#pragma unroll
    for (int e = 0; e < JW / 2; ++e) {
      const int m = n * CD_C + t, j = jb + 2 * e;
      vn[e] = (m < o.M && j0 + j < dv) ? __ldg(vrow + (size_t)m * o.lda + j) : 0.f;
    }
  };
  load_v(0);
  const int rl = lane & 7, cl = (lane >> 3) % CG, kh = (lane >> 3) / CG, KW = (D >> 2) / KH;      // products: rows rl + 8 i of [Kt; Qt], columns cl + CG i
  for (int n = 0; n < nblk; ++n) {
    const bool there = mbar_wait_bounded(smem_u32(&full[n & 1]), (uint32_t)((n >> 1) & 1));
    // the record is there, the transposed state too; everyone is done with the other buffer
    if (__syncthreads_or(!there)) {
      if (tid == 0) { seq_wait_error = 1; mbar_wait_bounded(smem_u32(&full[n & 1]), (uint32_t)((n >> 1) & 1)); }
      for (int i = tid; i < o.M * DVT; i += 128)
        if (j0 + i % DVT < dv) reinterpret_cast<float*>(o.C)[(size_t)(i / DVT) * o.ldc + (size_t)h * dv + j0 + i % DVT] = __int_as_float(0x7fc00000);
      return;
    }
    const float* rec = cw + (n & 1) * REC;
    {
      f32x2 acc[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0ull;
      const float* kr = rec + rl * P + (warp * KH + kh) * KW;
      const float* sr = St + cl * P + (warp * KH + kh) * KW;
#pragma unroll 2
      for (int k = 0; k < KW; k += 4) {
        ulonglong2 a[4], b[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const ulonglong2*>(kr + 8 * i * P + k);
#pragma unroll
        for (int j = 0; j < 4; ++j) b[j] = *reinterpret_cast<const ulonglong2*>(sr + CG * j * P + k);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            acc[i][j] = fma2<true>(a[i].x, b[j].x, acc[i][j]);
            acc[i][j] = fma2<true>(a[i].y, b[j].y, acc[i][j]);
          }
      }
      float* pw = Pp + warp * 2 * CD_C * PP;
#pragma unroll
      for (int i = 0; i < 4; i += KH)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          float v = lo2(acc[i][j]) + hi2(acc[i][j]);
          if (KH == 2) {       // a half-warp keeps every other row of its four
            const float w = lo2(acc[i + KH - 1][j]) + hi2(acc[i + KH - 1][j]);
            v = (kh ? w : v) + __shfl_xor_sync(0xffffffffu, kh ? v : w, 16);
          }
          pw[(rl + 8 * (i + (KH == 2 ? kh : 0))) * PP + cl + CG * j] = v;
        }
    }
    __syncthreads();
    const float* Tm = rec + 3 * CD_C * P + D;
    const float* Bm = Tm + CD_C * CD_TP;
    auto quarters = [&](const int r, const int j) {
      const float* p = Pp + r * PP + j;
      return (p[0] + p[2 * CD_C * PP]) + (p[4 * CD_C * PP] + p[6 * CD_C * PP]);
    };
    auto row_times = [&](const float* m, const int j) {       // sum_s m[t][s] Xs[j][s]
      const float* x = Xs + j * CD_TP;
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int s = 0; s < CD_C; s += 4) {
        const float4 mv = ld4(m + t * CD_TP + s), xv = ld4(x + s);
        a = fmaf(mv.x, xv.x, a); b = fmaf(mv.y, xv.y, b);
        a = fmaf(mv.z, xv.z, a); b = fmaf(mv.w, xv.w, b);
      }
      return a + b;
    };
    float u[JW / 2];
#pragma unroll
    for (int e = 0; e < JW / 2; ++e) Xs[(jb + 2 * e) * CD_TP + t] = vn[e] - quarters(t, jb + 2 * e);
    __syncwarp();
#pragma unroll
    for (int e = 0; e < JW / 2; ++e) u[e] = row_times(Tm, jb + 2 * e);
    __syncwarp();
#pragma unroll
    for (int e = 0; e < JW / 2; ++e) Xs[(jb + 2 * e) * CD_TP + t] = u[e];
    if (n + 1 < nblk) load_v(n + 1);
    __syncthreads();
    {   // S <- diag(G_last) S + Kb^T U
      const float* Kb = rec + 2 * CD_C * P;
      const float* Gl = rec + 3 * CD_C * P;
      const float* u0 = Xs + 2 * cp * CD_TP;
#pragma unroll
      for (int q = 0; q < RQ; ++q) {
        const int r = (rq + q * QS) * 4;
        if (r >= D) continue;
        const ulonglong2 gl = *reinterpret_cast<const ulonglong2*>(Gl + r);
#pragma unroll
        for (int j = 0; j < 2; ++j) { S[q][j][0] = mul2<true>(gl.x, S[q][j][0]); S[q][j][1] = mul2<true>(gl.y, S[q][j][1]); }
#pragma unroll
        for (int s = 0; s < CD_C; s += 4) {
          ulonglong2 kb[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) kb[e] = *reinterpret_cast<const ulonglong2*>(Kb + (s + e) * P + r);
          const float4 ua = ld4(u0 + s), ub = ld4(u0 + CD_TP + s);
          const float uv[2][4] = {{ua.x, ua.y, ua.z, ua.w}, {ub.x, ub.y, ub.z, ub.w}};
#pragma unroll
          for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
              const f32x2 uu = pack2(uv[j][e], uv[j][e]);
              S[q][j][0] = fma2<true>(kb[e].x, uu, S[q][j][0]);
              S[q][j][1] = fma2<true>(kb[e].y, uu, S[q][j][1]);
            }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
          *reinterpret_cast<ulonglong2*>(St + (2 * cp + j) * P + r) = make_ulonglong2(S[q][j][0], S[q][j][1]);
      }
    }
#pragma unroll
    for (int e = 0; e < JW / 2; ++e) {       // O = Qt S0 + B U
      const int j = jb + 2 * e, m = n * CD_C + t;
      const float ov = quarters(CD_C + t, j) + row_times(Bm, j);
      if (m < o.M && j0 + j < dv) reinterpret_cast<float*>(o.C)[(size_t)m * o.ldc + (size_t)h * dv + j0 + j] = ov;
    }
  }
  float* nst = reinterpret_cast<float*>(o.C2) + (size_t)h * dk * dv;
#pragma unroll
  for (int q = 0; q < RQ; ++q)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int r = (rq + q * QS) * 4, c = j0 + 2 * cp + j;
      const float v[4] = {lo2(S[q][j][0]), hi2(S[q][j][0]), lo2(S[q][j][1]), hi2(S[q][j][1])};
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (r + e < dk && c < dv) nst[(size_t)(r + e) * dv + c] = v[e];
    }
}

// ===========================================================================================================================
// ABI 8 (kinds 30-31): several residual streams with learned read / write / mixing weights, and the gated unit of routed experts
// whose weight multiplies the expert's input.
// ===========================================================================================================================
constexpr int HY_MAX = 16;      // streams; the kernel comes in an 8- and a 16-stream variant (register arrays of that size)
// grid (M), 256 threads, dynamic shared memory N floats (the row's read-out u).  One pass writes the streams back (when a
// sublayer's output is given) and forms u; a second one norms it.  Everything f32.
template <int MAXS>
__global__ void __launch_bounds__(256) fq3s_hyper_kernel(const fq3c_op o) {
  extern __shared__ float hsm[];
  __shared__ float red[32];
  const int m = blockIdx.x, S = o.i0;
  float* X = const_cast<float*>(reinterpret_cast<const float*>(o.A)) + (size_t)m * o.lda;
  const float* y = o.res ? reinterpret_cast<const float*>(o.res) + (size_t)m * o.ldr : nullptr;
  const float* mix = reinterpret_cast<const float*>(o.p0);
  const float* wo = reinterpret_cast<const float*>(o.p1);
  const float* wi = reinterpret_cast<const float*>(o.bias);
  float ss = 0.f;
  for (int c = threadIdx.x; c < o.N; c += blockDim.x) {
    float xs[MAXS], xn[MAXS];
#pragma unroll
    for (int s = 0; s < MAXS; ++s) xs[s] = s < S ? X[(size_t)s * (size_t)o.K + c] : 0.f;
    if (y) {
      const float yv = o.f1 * y[c];
#pragma unroll
      for (int t = 0; t < MAXS; ++t) {
        if (t >= S) continue;
        float acc = wo[t] * yv;
#pragma unroll
        for (int s = 0; s < MAXS; ++s)
          if (s < S) acc = fmaf(mix[s * S + t], xs[s], acc);
        xn[t] = acc;
        X[(size_t)t * (size_t)o.K + c] = acc;
      }
    } else {
#pragma unroll
      for (int t = 0; t < MAXS; ++t) xn[t] = xs[t];
    }
    if (o.C) {
      float u = 0.f;
#pragma unroll
      for (int t = 0; t < MAXS; ++t)
        if (t < S) u = fmaf(wi[t], xn[t], u);
      hsm[c] = u;
      ss = fmaf(u, u, ss);
    }
  }
  if (!o.C) return;
  const float* w = reinterpret_cast<const float*>(o.scale);
  float rs = 1.f;
  if (w) rs = 1.f / sqrtf(seq_block_sum(ss, red) / (float)o.N + o.f0);
  for (int c = threadIdx.x; c < o.N; c += blockDim.x) {      // a thread reads back what it wrote itself
    const float v = w ? hsm[c] * rs * w[c] : hsm[c];
    if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[(size_t)m * o.ldc + c] = v;
    else reinterpret_cast<bf16*>(o.C)[(size_t)m * o.ldc + c] = __float2bfloat16_rn(v);
  }
}

// grid (ceil(N / 256), M)
__global__ void __launch_bounds__(256) fq3s_glu_kernel(const fq3c_op o) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, q = blockIdx.y;
  if (c >= o.N) return;
  const int r = o.ws ? reinterpret_cast<const int*>(o.ws)[q] : q;
  if (r < 0) return;
  const float w = o.p1 ? reinterpret_cast<const float*>(o.p1)[q] : 1.f;
  const float* a = reinterpret_cast<const float*>(o.A) + (size_t)r * o.lda;
  const float g = w * a[c], u = w * a[o.N + c];
  const float v = g / (1.f + expf(-g)) * u;
  if (o.flags & FQ3C_OUT_F32) reinterpret_cast<float*>(o.C)[(size_t)r * o.ldc + c] = v;
  else reinterpret_cast<bf16*>(o.C)[(size_t)r * o.ldc + c] = __float2bfloat16_rn(v);
}

// ===========================================================================================================================
// ABI 9 (kind 32): the residual sum of a layer whose sublayers run side by side on one normed input, fused with the norm that
// reads the finished stream (a layer norm without bias, or an RMS norm).
// ===========================================================================================================================
// grid (M), 256 threads (up to 1024 for a few rows), dynamic shared memory N floats (the finished row).  Pass 1 forms the weighted sum of the slices, writes it
// and keeps it; passes 2 and 3 take the mean and the mean squared deviation from the kept row; pass 4 writes the normed row.
// A thread only ever reads back entries it wrote itself, and C may be slice 0 (every entry is read before it is written).
__global__ void __launch_bounds__(1024) fq3s_sum_norm_kernel(const fq3c_op o) {
  extern __shared__ float snm[];
  __shared__ float red[32];
  const int m = blockIdx.x;
  const float* a = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda;
  const float* w = reinterpret_cast<const float*>(o.p0);
  float* c = reinterpret_cast<float*>(o.C) + (size_t)m * o.ldc;
  const bool post = (o.flags & FQ3C_POST) != 0;
  const float* nb = reinterpret_cast<const float*>(o.bias);
  float sm = 0.f;
  for (int i = threadIdx.x; i < o.N; i += blockDim.x) {
    float v = 0.f;
    for (int j = 0; j < o.i0; j += 4) {       // four slices' loads in flight
      float wv[4], av[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) { const bool ok = j + q < o.i0; wv[q] = ok ? w[j + q] : 0.f; av[q] = ok ? a[(size_t)(j + q) * (size_t)o.K + i] : 0.f; }
#pragma unroll
      for (int q = 0; q < 4; ++q)
        if (j + q < o.i0) v = fmaf(wv[q], av[q], v);
    }
    if (!post) c[i] = v;
    if (o.C2) reinterpret_cast<bf16*>(o.C2)[(size_t)m * o.ldc + i] = __float2bfloat16_rn(v);
    snm[i] = v;
    sm += v;
  }
  if (!o.norm_out && !post) return;
  if (!o.norm_w) {       // no norm: the finished row itself, in the product operands' type
    for (int i = threadIdx.x; i < o.N; i += blockDim.x) {
      if (o.flags & FQ3C_F32) reinterpret_cast<float*>(o.norm_out)[(size_t)m * o.norm_ld + i] = snm[i];
      else reinterpret_cast<bf16*>(o.norm_out)[(size_t)m * o.norm_ld + i] = __float2bfloat16_rn(snm[i]);
    }
    return;
  }
  float mean = 0.f;
  if (o.flags & FQ3C_CENTER) mean = seq_block_sum(sm, red) / (float)o.N;
  float ss = 0.f;
  for (int i = threadIdx.x; i < o.N; i += blockDim.x) { const float d = snm[i] - mean; ss = fmaf(d, d, ss); }
  const float rs = 1.f / sqrtf(seq_block_sum(ss, red) / (float)o.N + o.norm_eps);
  const float* nw = reinterpret_cast<const float*>(o.norm_w);
  for (int i = threadIdx.x; i < o.N; i += blockDim.x) {
    float n = (snm[i] - mean) * rs * nw[i];
    if (nb) n += nb[i];
    if (post) c[i] = n;
    if (!o.norm_out) continue;
    if (o.flags & FQ3C_F32) reinterpret_cast<float*>(o.norm_out)[(size_t)m * o.norm_ld + i] = n;
    else reinterpret_cast<bf16*>(o.norm_out)[(size_t)m * o.norm_ld + i] = __float2bfloat16_rn(n);
  }
}

// The same for rows of whole 16-byte pieces: the row stays in registers.  grid (M), up to 256 threads.
constexpr int SN_VECS = 4;
__global__ void __launch_bounds__(256) fq3s_sum_norm_vec_kernel(const fq3c_op o) {
  __shared__ float red[32];
  const int m = blockIdx.x, tid = threadIdx.x, nth = blockDim.x;
  const float* a = reinterpret_cast<const float*>(o.A) + (size_t)m * o.lda;
  const float* w = reinterpret_cast<const float*>(o.p0);
  float* c = reinterpret_cast<float*>(o.C) + (size_t)m * o.ldc;
  const bool post = (o.flags & FQ3C_POST) != 0;
  float v[SN_VECS][4];
#pragma unroll
  for (int q = 0; q < SN_VECS; ++q) { v[q][0] = 0.f; v[q][1] = 0.f; v[q][2] = 0.f; v[q][3] = 0.f; }
  for (int j = 0; j < o.i0; j += 2) {       // two slices' loads in flight
    float4 s0[SN_VECS], s1[SN_VECS];
    const bool two = j + 1 < o.i0;
    const float w0 = w[j], w1 = two ? w[j + 1] : 0.f;
#pragma unroll
    for (int q = 0; q < SN_VECS; ++q) {
      const int i = (q * nth + tid) * 4;
      if (i < o.N) {
        s0[q] = ld4(a + (size_t)j * (size_t)o.K + i);
        if (two) s1[q] = ld4(a + (size_t)(j + 1) * (size_t)o.K + i);
      }
    }
#pragma unroll
    for (int q = 0; q < SN_VECS; ++q) {
      if ((q * nth + tid) * 4 >= o.N) continue;
      v[q][0] = fmaf(w0, s0[q].x, v[q][0]); v[q][1] = fmaf(w0, s0[q].y, v[q][1]); v[q][2] = fmaf(w0, s0[q].z, v[q][2]); v[q][3] = fmaf(w0, s0[q].w, v[q][3]);
      if (two) { v[q][0] = fmaf(w1, s1[q].x, v[q][0]); v[q][1] = fmaf(w1, s1[q].y, v[q][1]); v[q][2] = fmaf(w1, s1[q].z, v[q][2]); v[q][3] = fmaf(w1, s1[q].w, v[q][3]); }
    }
  }
  float sm = 0.f;
#pragma unroll
  for (int q = 0; q < SN_VECS; ++q) {
    const int i = (q * nth + tid) * 4;
    if (i >= o.N) continue;
    if (!post) st4(c + i, v[q]);
    sm += (v[q][0] + v[q][1]) + (v[q][2] + v[q][3]);
  }
  if (!o.norm_out && !post) return;
  float rs = 1.f, mean = 0.f;
  if (o.norm_w) {
    if (o.flags & FQ3C_CENTER) mean = seq_block_sum(sm, red) / (float)o.N;
    float ss = 0.f;
#pragma unroll
    for (int q = 0; q < SN_VECS; ++q) {
      if ((q * nth + tid) * 4 >= o.N) continue;
#pragma unroll
      for (int e = 0; e < 4; ++e) { const float d = v[q][e] - mean; ss = fmaf(d, d, ss); }
    }
    rs = 1.f / sqrtf(seq_block_sum(ss, red) / (float)o.N + o.norm_eps);
  }
#pragma unroll
  for (int q = 0; q < SN_VECS; ++q) {
    const int i = (q * nth + tid) * 4;
    if (i >= o.N) continue;
    if (o.norm_w) {
      const float4 nw = ld4(reinterpret_cast<const float*>(o.norm_w) + i);
      v[q][0] = (v[q][0] - mean) * rs * nw.x; v[q][1] = (v[q][1] - mean) * rs * nw.y; v[q][2] = (v[q][2] - mean) * rs * nw.z; v[q][3] = (v[q][3] - mean) * rs * nw.w;
      if (o.bias) {
        const float4 nb = ld4(reinterpret_cast<const float*>(o.bias) + i);
        v[q][0] += nb.x; v[q][1] += nb.y; v[q][2] += nb.z; v[q][3] += nb.w;
      }
      if (post) st4(c + i, v[q]);
      if (!o.norm_out) continue;
    }
    if (o.flags & FQ3C_F32) st4(reinterpret_cast<float*>(o.norm_out) + (size_t)m * o.norm_ld + i, v[q]);
    else st4(reinterpret_cast<bf16*>(o.norm_out) + (size_t)m * o.norm_ld + i, v[q]);
  }
}
