// Per-head RMSNorm on q and k, rotary position encoding on q and k, and the write of k and v
// into the request's cache pages: one pass over the [T, (H+2G)*hd] output of the QKV product.
//
// FeLLM does this as separate ops: rmsnorm_group (oxide_kernels.rs:165), rope_batch (323),
// kv_write_batch (4227) twice; formulas in crates/backend-cpu/src/kernels/norm.rs:6-39 and
// rope.rs:28-62.  Angle = float32(position) * inv_freq[i]; a' = a*c - b*s, b' = a*s + b*c on
// pairs (2i, 2i+1) (pairing 0, "adjacent") or (i, i+rot_dim/2) (pairing 1, "split_half") of the
// first rot_dim <= hd elements of a head (rope.rs:37-44: rope_dim <= head_dim); the elements
// behind rot_dim are normed and not rotated.  inv_freq has rot_dim/2 entries.
//
// Cache pool layout (one pool per cache group, shared by the group's layers):
//   [page][layer in group][k=0 / v=1][kv head][token in page][hd]
// so that the [page_tokens, hd] tile of one kv head is contiguous.
#include "common.cuh"

template <typename TA, typename TC>
__global__ void qk_rope_write_kernel(const TA* __restrict__ qkv, const float* __restrict__ q_w,
                                     const float* __restrict__ k_w, float eps,
                                     const float* __restrict__ inv_freq, int pairing,
                                     const int* __restrict__ positions, const int* __restrict__ row_slot,
                                     const int* __restrict__ block_table, int max_pages,
                                     TC* __restrict__ pool, int layer, int layers_in_group,
                                     int page_tokens, TA* __restrict__ q_out, int T, int H, int G, int hd,
                                     int rot_dim, int write_kv, int* __restrict__ status) {
  FELLM_TRACE_SCOPE(TRACE_QK_ROPE_WRITE);
  pdl_launch_dependents();
  pdl_wait(); FELLM_TRACE_WAITED();
  int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  int lane = threadIdx.x & 31;
  int heads_total = H + 2 * G;
  if (warp >= T * heads_total) return;
  int row = warp / heads_total, head = warp - row * heads_total;
  const TA* src = qkv + (size_t)row * heads_total * hd + (size_t)head * hd;
  int pos = positions[row];
  bool is_q = head < H, is_k = !is_q && head < H + G;
  if (!is_q && !write_kv) return;

  TC* dst_c = nullptr;
  if (!is_q) {
    int g = is_k ? head - H : head - H - G;
    int page = block_table[(size_t)row_slot[row] * max_pages + pos / page_tokens];
    if (page < 0) {                      // never write outside the pool: record and skip
      if (lane == 0 && status) atomicExch(status, 2);
      return;
    }
    size_t off = ((((size_t)page * layers_in_group + layer) * 2 + (is_k ? 0 : 1)) * G + g) * page_tokens
                 + (pos % page_tokens);
    dst_c = pool + off * hd;
  }
  if (!is_q && !is_k) {                  // v: copied as it is
    for (int e = lane; e < hd; e += 32) dst_c[e] = from_f<TC>(to_f(src[e]));
    return;
  }
  const float* nw = is_q ? q_w : k_w;
  int half = rot_dim >> 1;
  float scale = 1.f;
  if (nw) {
    float ss = 0.f;
    for (int e = lane; e < hd; e += 32) { float v = to_f(src[e]); ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    scale = 1.0f / sqrtf(ss / (float)hd + eps);
  }
  for (int e = rot_dim + lane; e < hd; e += 32) {      // behind the rotated part: normed, not rotated
    float a = to_f(src[e]);
    if (nw) a = (a * scale) * nw[e];
    if (is_q) q_out[((size_t)row * H + head) * hd + e] = from_f<TA>(a);
    else dst_c[e] = from_f<TC>(a);
  }
  for (int p = lane; p < half; p += 32) {
    int i0 = pairing == 0 ? 2 * p : p;
    int i1 = pairing == 0 ? 2 * p + 1 : p + half;
    float a = to_f(src[i0]), b = to_f(src[i1]);
    if (nw) { a = (a * scale) * nw[i0]; b = (b * scale) * nw[i1]; }
    if (inv_freq) {
      float ang = (float)pos * inv_freq[p];
      float sn, cs;
      sincosf(ang, &sn, &cs);
      float a2 = a * cs - b * sn, b2 = a * sn + b * cs;
      a = a2; b = b2;
    }
    if (is_q) {
      TA* q = q_out + ((size_t)row * H + head) * hd;
      q[i0] = from_f<TA>(a); q[i1] = from_f<TA>(b);
    } else {
      dst_c[i0] = from_f<TC>(a); dst_c[i1] = from_f<TC>(b);
    }
  }
}

// bfloat16, hd % 16 == 0: a head is taken by hd/16 lanes of a group of GL lanes (GL the next power
// of two), each with 16 elements = 8 pairs in two 16-byte loads: elements [16l, 16l+16) when pairs
// are adjacent, [8l, 8l+8) and [hd/2 + 8l, hd/2 + 8l + 8) when they are (i, i + hd/2).
__device__ __forceinline__ void rw_unpack8(uint4 v, float* f) {
  const __nv_bfloat162* h = (const __nv_bfloat162*)&v;
#pragma unroll
  for (int i = 0; i < 4; ++i) { float2 t = __bfloat1622float2(h[i]); f[2 * i] = t.x; f[2 * i + 1] = t.y; }
}
__device__ __forceinline__ uint4 rw_pack8(const float* f) {
  uint4 v;
  __nv_bfloat162 p0 = __floats2bfloat162_rn(f[0], f[1]), p1 = __floats2bfloat162_rn(f[2], f[3]);
  __nv_bfloat162 p2 = __floats2bfloat162_rn(f[4], f[5]), p3 = __floats2bfloat162_rn(f[6], f[7]);
  v.x = *(unsigned*)&p0; v.y = *(unsigned*)&p1; v.z = *(unsigned*)&p2; v.w = *(unsigned*)&p3;
  return v;
}

template <int GL>
__global__ void qk_rope_write_vec_kernel(const bf16* __restrict__ qkv, const float* __restrict__ q_w,
                                         const float* __restrict__ k_w, float eps,
                                         const float* __restrict__ inv_freq, int pairing,
                                         const int* __restrict__ positions, const int* __restrict__ row_slot,
                                         const int* __restrict__ block_table, int max_pages,
                                         bf16* __restrict__ pool, int layer, int layers_in_group,
                                         int page_tokens, bf16* __restrict__ q_out, int T, int H, int G, int hd,
                                         int write_kv, int* __restrict__ status) {
  FELLM_TRACE_SCOPE(TRACE_QK_ROPE_WRITE_VEC);
  pdl_launch_dependents();
  pdl_wait(); FELLM_TRACE_WAITED();
  const long long gid = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / GL;
  const int l = threadIdx.x % GL;
  const int heads_total = H + 2 * G;
  const bool live = gid < (long long)T * heads_total;         // every lane stays for the shuffles
  const int row = live ? (int)(gid / heads_total) : 0, head = live ? (int)(gid - (long long)row * heads_total) : 0;
  const bool is_q = head < H, is_k = !is_q && head < H + G;
  const bool lane_on = live && l * 16 < hd && (is_q || write_kv);
  const int half = hd >> 1;
  const int o0 = pairing == 0 ? 16 * l : 8 * l;               // the lane's two runs of 8 elements
  const int o1 = pairing == 0 ? 16 * l + 8 : half + 8 * l;
  const bf16* src = qkv + ((size_t)row * heads_total + head) * hd;
  const int pos = positions[row];

  bf16* dst = nullptr;
  bool ok = lane_on;
  if (lane_on) {
    if (is_q) dst = q_out + ((size_t)row * H + head) * hd;
    else {
      int g = is_k ? head - H : head - H - G;
      int page = block_table[(size_t)row_slot[row] * max_pages + pos / page_tokens];
      if (page < 0) {                      // never write outside the pool: record and skip
        if (l == 0 && status) atomicExch(status, 2);
        ok = false;
      } else {
        size_t off = ((((size_t)page * layers_in_group + layer) * 2 + (is_k ? 0 : 1)) * G + g) * page_tokens
                     + (pos % page_tokens);
        dst = pool + off * hd;
      }
    }
  }
  uint4 r0 = make_uint4(0, 0, 0, 0), r1 = r0;
  if (lane_on) { r0 = *(const uint4*)(src + o0); r1 = *(const uint4*)(src + o1); }
  const bool is_v = !is_q && !is_k;
  if (is_v) {                              // v: copied as it is; the lanes stay for the warp's shuffles
    if (ok) { *(uint4*)(dst + o0) = r0; *(uint4*)(dst + o1) = r1; }
    ok = false;
  }
  float a[8], b[8];
  rw_unpack8(r0, a); rw_unpack8(r1, b);
  const float* nw = is_q ? q_w : k_w;
  if (nw) {
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(a[e], a[e], ss);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(b[e], b[e], ss);
#pragma unroll
    for (int o = GL / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float scale = 1.0f / sqrtf(ss / (float)hd + eps);
    if (ok) {
#pragma unroll
      for (int e = 0; e < 8; ++e) { a[e] = (a[e] * scale) * nw[o0 + e]; b[e] = (b[e] * scale) * nw[o1 + e]; }
    }
  }
  if (!ok) return;
  if (inv_freq) {
    if (pairing == 0) {                    // pairs (2i, 2i+1): inside each run
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        float sn, cs;
        sincosf((float)pos * inv_freq[(o0 + e) >> 1], &sn, &cs);
        float x = a[e], y = a[e + 1];
        a[e] = x * cs - y * sn; a[e + 1] = x * sn + y * cs;
        sincosf((float)pos * inv_freq[(o1 + e) >> 1], &sn, &cs);
        x = b[e]; y = b[e + 1];
        b[e] = x * cs - y * sn; b[e + 1] = x * sn + y * cs;
      }
    } else {                               // pairs (i, i + hd/2): run a against run b
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float sn, cs;
        sincosf((float)pos * inv_freq[o0 + e], &sn, &cs);
        float x = a[e], y = b[e];
        a[e] = x * cs - y * sn; b[e] = x * sn + y * cs;
      }
    }
  }
  *(uint4*)(dst + o0) = rw_pack8(a);
  *(uint4*)(dst + o1) = rw_pack8(b);
}

FELLM_API int fellm_qk_rope_write(const void* qkv, int act_bf16, const float* q_w, const float* k_w,
                                  float eps, const float* inv_freq, int pairing, const int* positions,
                                  const int* row_slot, const int* block_table, int max_pages, void* pool,
                                  int cache_bf16, int layer, int layers_in_group, int page_tokens,
                                  void* q_out, int T, int H, int G, int hd, int rot_dim, int write_kv,
                                  int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (hd < 2 || (hd & 1)) return FELLM_ERR_SIZE;
  if (!inv_freq) rot_dim = 0;
  if (rot_dim < 0 || rot_dim > hd || (rot_dim & 1)) return FELLM_ERR_SIZE;
  if (!qkv || !q_out || !positions || !row_slot || (write_kv && (!pool || !block_table))) return FELLM_ERR_ARG;
  if (act_bf16 != cache_bf16) return FELLM_ERR_ARG;
  long long warps = (long long)T * (H + 2 * G);
  int threads = 128;
  long long blocks = (warps * 32 + threads - 1) / threads;
  if (act_bf16 && hd % 16 == 0 && hd <= 256 && (rot_dim == hd || rot_dim == 0)) {
    int lanes = hd / 16, gl = 1;
    while (gl < lanes) gl <<= 1;
    long long nthreads = warps * gl;
    dim3 vgrid((unsigned)((nthreads + threads - 1) / threads));
#define RW_VEC(GL_) launch_k_class(launch_class_for_rows(T, 2), qk_rope_write_vec_kernel<GL_>, vgrid, dim3(threads), 0, stream, 1, (const bf16*)qkv, q_w, k_w, \
                             eps, inv_freq, pairing, positions, row_slot, block_table, max_pages, (bf16*)pool, layer,     \
                             layers_in_group, page_tokens, (bf16*)q_out, T, H, G, hd, write_kv, status)
    switch (gl) {
      case 1: return RW_VEC(1);
      case 2: return RW_VEC(2);
      case 4: return RW_VEC(4);
      case 8: return RW_VEC(8);
      default: return RW_VEC(16);
    }
#undef RW_VEC
  }
  if (act_bf16)
    return launch_k_class(launch_class_for_rows(T, 2), qk_rope_write_kernel<bf16, bf16>, dim3((unsigned)blocks), dim3(threads), 0, stream, 1,
                    (const bf16*)qkv, q_w, k_w, eps, inv_freq, pairing, positions, row_slot, block_table, max_pages,
                    (bf16*)pool, layer, layers_in_group, page_tokens, (bf16*)q_out, T, H, G, hd, rot_dim, write_kv, status);
  return launch_k_class(launch_class_for_rows(T, 2), qk_rope_write_kernel<float, float>, dim3((unsigned)blocks), dim3(threads), 0, stream, 1,
                  (const float*)qkv, q_w, k_w, eps, inv_freq, pairing, positions, row_slot, block_table, max_pages,
                  (float*)pool, layer, layers_in_group, page_tokens, (float*)q_out, T, H, G, hd, rot_dim, write_kv, status);
}

// ---------------------------------------------------------------- rotation and unit norm in place
// For layers whose keys and values differ in size (or that read another layer's pages): the heads of q (n_q at column
// 0 of a row) and of k (n_k at column k_off) are rotated on their first rot_dim elements and then, unit_norm, divided
// by their root mean square over hd (no weight), where they lie; the cache write and the attention read them from
// there.  A warp a (row, head); a head's values stay in registers between the sum and the scaling, so a bfloat16 value
// is rounded once.  hd <= 512.
#define RN_MAXP 8      // pairs a lane: rot_dim <= 512
#define RN_MAXT 16     // unrotated elements a lane
template <typename TA>
__global__ void __launch_bounds__(128)
qk_rotate_norm_kernel(TA* __restrict__ qkv, int ld, int T, int n_q, int n_k, int k_off, int hd, int rot_dim,
                      const float* __restrict__ inv_freq, int pairing, const int* __restrict__ positions, float eps,
                      int unit_norm) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  const int heads = n_q + n_k;
  if (warp >= T * heads) return;
  const int row = warp / heads, head = warp - row * heads;
  TA* p = qkv + (size_t)row * ld + (head < n_q ? (size_t)head * hd : (size_t)k_off + (size_t)(head - n_q) * hd);
  const float pos = (float)positions[row];
  const int half = rot_dim >> 1;
  float ra[RN_MAXP], rb[RN_MAXP], tl[RN_MAXT];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < RN_MAXP; ++j) {
    const int i = lane + 32 * j;
    ra[j] = rb[j] = 0.f;
    if (i < half) {
      const int ia = pairing ? i : 2 * i, ib = pairing ? i + half : 2 * i + 1;
      float sn, cs;
      sincosf(pos * inv_freq[i], &sn, &cs);
      const float a = to_f(p[ia]), b = to_f(p[ib]);
      ra[j] = a * cs - b * sn; rb[j] = b * cs + a * sn;
      ss = fmaf(ra[j], ra[j], fmaf(rb[j], rb[j], ss));
    }
  }
#pragma unroll
  for (int j = 0; j < RN_MAXT; ++j) {
    const int i = rot_dim + lane + 32 * j;
    tl[j] = 0.f;
    if (i < hd) { tl[j] = to_f(p[i]); ss = fmaf(tl[j], tl[j], ss); }
  }
  float scale = 1.0f;
  if (unit_norm) scale = 1.0f / sqrtf(warp_sum(ss) / (float)hd + eps);
#pragma unroll
  for (int j = 0; j < RN_MAXP; ++j) {
    const int i = lane + 32 * j;
    if (i < half) {
      const int ia = pairing ? i : 2 * i, ib = pairing ? i + half : 2 * i + 1;
      p[ia] = from_f<TA>(ra[j] * scale); p[ib] = from_f<TA>(rb[j] * scale);
    }
  }
  if (unit_norm) {
#pragma unroll
    for (int j = 0; j < RN_MAXT; ++j) {
      const int i = rot_dim + lane + 32 * j;
      if (i < hd) p[i] = from_f<TA>(tl[j] * scale);
    }
  }
}

// bfloat16, heads of 32, 64, 128 or 256, pairs (i, i + rot_dim/2), rot_dim a multiple of 16: hd / 8 lanes a head, a lane
// eight consecutive elements (one 16-byte load, and one more for the eight it is paired with); a head's sum of squares
// goes round its lanes by shuffles.  All loads of a warp lie in front of its stores.
template <int LANES>
__global__ void __launch_bounds__(128)
qk_rotate_norm_vec_kernel(bf16* __restrict__ qkv, int ld, int T, int n_q, int n_k, int k_off, int rot_dim,
                          const float* __restrict__ inv_freq, const int* __restrict__ positions, float eps, int unit_norm) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int hd = LANES * 8;
  const long long slot = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / LANES;
  const int c = threadIdx.x % LANES;                       // this lane's chunk of eight in the head
  const int heads = n_q + n_k;
  const bool live = slot < (long long)T * heads;
  const int row = live ? (int)(slot / heads) : 0, head = live ? (int)(slot - (long long)row * heads) : 0;
  bf16* p = qkv + (size_t)row * ld + (head < n_q ? (size_t)head * hd : (size_t)k_off + (size_t)(head - n_q) * hd);
  const int half = rot_dim >> 1, hc = half >> 3;           // chunks of a half
  float v[8], w[8];
  uint4 mine = make_uint4(0, 0, 0, 0), other = make_uint4(0, 0, 0, 0);
  const bool rotated = c < 2 * hc, first = c < hc;
  if (live) {
    mine = *(const uint4*)(p + 8 * c);
    if (rotated) other = *(const uint4*)(p + 8 * (first ? c + hc : c - hc));
  }
  __syncwarp();
  {
    const __nv_bfloat162* m2 = (const __nv_bfloat162*)&mine; const __nv_bfloat162* o2 = (const __nv_bfloat162*)&other;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 a = __bfloat1622float2(m2[e]), b = __bfloat1622float2(o2[e]);
      v[2 * e] = a.x; v[2 * e + 1] = a.y; w[2 * e] = b.x; w[2 * e + 1] = b.y;
    }
  }
  float ss = 0.f;
  if (rotated && live) {
    const float pos = (float)positions[row];
    const int f0 = 8 * (first ? c : c - hc);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float sn, cs;
      sincosf(pos * inv_freq[f0 + e], &sn, &cs);
      v[e] = first ? v[e] * cs - w[e] * sn : v[e] * cs + w[e] * sn;
    }
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float scale = unit_norm ? 1.0f / sqrtf(ss / (float)hd + eps) : 1.0f;
  if (live && (rotated || unit_norm)) {
    uint4 out; __nv_bfloat162* o2 = (__nv_bfloat162*)&out;
#pragma unroll
    for (int e = 0; e < 4; ++e) o2[e] = __floats2bfloat162_rn(v[2 * e] * scale, v[2 * e + 1] * scale);
    *(uint4*)(p + 8 * c) = out;
  }
}

FELLM_API int fellm_qk_rotate_norm(void* qkv, int is_bf16, int ld, int T, int n_q, int n_k, int k_off, int hd, int rot_dim,
                                   const float* inv_freq, int pairing, const int* positions, float eps, int unit_norm,
                                   cudaStream_t stream) {
  if (T <= 0 || n_q + n_k <= 0) return 0;
  if (!inv_freq) rot_dim = 0;
  if (hd < 1 || hd > 32 * RN_MAXT || rot_dim < 0 || rot_dim > hd || (rot_dim & 1) || rot_dim > 64 * RN_MAXP) return FELLM_ERR_SIZE;
  if (!qkv || !positions || n_q < 0 || n_k < 0) return FELLM_ERR_ARG;
  if (!rot_dim && !unit_norm) return 0;
  const long long warps = (long long)T * (n_q + n_k);
  const int cls = launch_class_for_rows(T, 2);
  if (is_bf16 && pairing == 1 && (hd == 32 || hd == 64 || hd == 128 || hd == 256) && rot_dim % 16 == 0 && ld % 8 == 0 &&
      k_off % 8 == 0 && ((uintptr_t)qkv & 15) == 0) {
    const int lanes = hd / 8;
    dim3 vgrid((unsigned)((warps * lanes + 127) / 128));
#define RN_VEC(L_) launch_k_class(cls, qk_rotate_norm_vec_kernel<L_>, vgrid, dim3(128), 0, stream, 1, (bf16*)qkv, ld, T, n_q, n_k, k_off, \
                                  rot_dim, inv_freq, positions, eps, unit_norm)
    switch (lanes) {
      case 4: return RN_VEC(4);
      case 8: return RN_VEC(8);
      case 16: return RN_VEC(16);
      default: return RN_VEC(32);
    }
#undef RN_VEC
  }
  dim3 grid((unsigned)((warps + 3) / 4));
  if (is_bf16) return launch_k_class(cls, qk_rotate_norm_kernel<bf16>, grid, dim3(128), 0, stream, 1, (bf16*)qkv, ld, T, n_q, n_k, k_off, hd,
                                     rot_dim, inv_freq, pairing, positions, eps, unit_norm);
  return launch_k_class(cls, qk_rotate_norm_kernel<float>, grid, dim3(128), 0, stream, 1, (float*)qkv, ld, T, n_q, n_k, k_off, hd,
                        rot_dim, inv_freq, pairing, positions, eps, unit_norm);
}

// ---------------------------------------------------------------- rotation, value mixing and the cache write in one
// For layers whose keys and values differ in size, whose cos and sin carry a magnitude, or whose values are mixed with
// an earlier layer's: the rows of the input product are [q (H hd) | k (G hd) | v (G vd)], ld elements apart.  q is
// rotated where it lies; k, rotated, and v, or (1 - lam) v + lam v0 (v0: the same rows' values of the layer mixed with,
// ldv0 elements apart; lam: one float on the device), go into the row's page.  A page-layer record is the keys
// [G][page_tokens][hd], then the values [G][page_tokens][vd].  Rotation: the first rot_dim elements of a head, angle =
// float(position) * inv_freq[i], cos and sin times mag; float32 throughout, rounded once.  A block a row: the row's
// sines and cosines once for all heads, and its page's number, before the wait for the product.
#define RWM_HALF 256      // pairs of a head in shared memory: rot_dim <= 512

struct RotateWriteArgs {
  int ld, H, G, hd, vd, rot_dim, pairing, ldv0, max_pages, page_tokens, layer, layers_in_group;
  float mag;
  const float* inv_freq; const float* lam;
  const int* positions; const int* row_slot; const int* block_table;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(128)
qkv_rotate_write_kernel(T* __restrict__ qkv, const T* __restrict__ v0, T* __restrict__ pool, RotateWriteArgs a) {
  __shared__ float sn_s[RWM_HALF], cs_s[RWM_HALF];
  pdl_launch_dependents();
  const int row = blockIdx.x, pos = a.positions[row], half = a.rot_dim >> 1;
  const int page = a.block_table[(size_t)a.row_slot[row] * a.max_pages + pos / a.page_tokens];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, cs;
    sincosf((float)pos * a.inv_freq[i], &sn, &cs);
    sn_s[i] = sn * a.mag; cs_s[i] = cs * a.mag;
  }
  __syncthreads();
  pdl_wait();
  T* p = qkv + (size_t)row * a.ld;
  for (int u = threadIdx.x; u < a.H * half; u += blockDim.x) {
    const int h = u / half, i = u - h * half;
    T* q = p + (size_t)h * a.hd;
    const int ia = a.pairing ? i : 2 * i, ib = a.pairing ? i + half : 2 * i + 1;
    const float x = to_f(q[ia]), y = to_f(q[ib]);
    q[ia] = from_f<T>(x * cs_s[i] - y * sn_s[i]); q[ib] = from_f<T>(y * cs_s[i] + x * sn_s[i]);
  }
  if (page < 0) {                        // never write outside the pool: record and skip
    if (threadIdx.x == 0 && a.status) atomicExch(a.status, 2);
    return;
  }
  const int in_page = pos % a.page_tokens;
  T* rec = pool + ((size_t)page * a.layers_in_group + a.layer) * ((size_t)a.G * a.page_tokens * (a.hd + a.vd));
  const T* kp = p + (size_t)a.H * a.hd;
  const int per_k = a.hd - half;         // a pair, or one element behind the rotated part
  for (int u = threadIdx.x; u < a.G * per_k; u += blockDim.x) {
    const int g = u / per_k, i = u - g * per_k;
    const T* k = kp + (size_t)g * a.hd;
    T* dst = rec + ((size_t)g * a.page_tokens + in_page) * a.hd;
    if (i < half) {
      const int ia = a.pairing ? i : 2 * i, ib = a.pairing ? i + half : 2 * i + 1;
      const float x = to_f(k[ia]), y = to_f(k[ib]);
      dst[ia] = from_f<T>(x * cs_s[i] - y * sn_s[i]); dst[ib] = from_f<T>(y * cs_s[i] + x * sn_s[i]);
    } else {
      dst[i + half] = k[i + half];
    }
  }
  const T* vp = kp + (size_t)a.G * a.hd;
  T* vrec = rec + (size_t)a.G * a.page_tokens * a.hd;
  const float lam = v0 ? *a.lam : 0.f;
  for (int u = threadIdx.x; u < a.G * a.vd; u += blockDim.x) {
    const int g = u / a.vd, c = u - g * a.vd;
    T* dst = vrec + ((size_t)g * a.page_tokens + in_page) * a.vd + c;
    if (v0) *dst = from_f<T>((1.0f - lam) * to_f(vp[u]) + lam * to_f(v0[(size_t)row * a.ldv0 + u]));
    else *dst = vp[u];
  }
}

// bfloat16, pairs (i, i + rot_dim/2), hd and vd multiples of 8, rot_dim of 16, rows on 16-byte boundaries: a thread eight
// elements (and the eight they are paired with) by 16-byte loads and stores.
__global__ void __launch_bounds__(128)
qkv_rotate_write_vec_kernel(bf16* __restrict__ qkv, const bf16* __restrict__ v0, bf16* __restrict__ pool, RotateWriteArgs a) {
  __shared__ float sn_s[RWM_HALF], cs_s[RWM_HALF];
  pdl_launch_dependents();
  const int row = blockIdx.x, pos = a.positions[row], half = a.rot_dim >> 1;
  const int page = a.block_table[(size_t)a.row_slot[row] * a.max_pages + pos / a.page_tokens];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, cs;
    sincosf((float)pos * a.inv_freq[i], &sn, &cs);
    sn_s[i] = sn * a.mag; cs_s[i] = cs * a.mag;
  }
  __syncthreads();
  pdl_wait();
  bf16* p = qkv + (size_t)row * a.ld;
  const int hc = half >> 3, kc = (a.hd >> 3) - hc, vc = a.vd >> 3;      // units of a query head, a key head, a value
  const int n_q = a.H * hc, n_k = a.G * kc, n_v = a.G * vc;
  const int in_page = pos % a.page_tokens;
  if (page < 0 && threadIdx.x == 0 && a.status) atomicExch(a.status, 2);          // never write outside the pool: record and skip
  bf16* rec = pool + ((size_t)max(page, 0) * a.layers_in_group + a.layer) * ((size_t)a.G * a.page_tokens * (a.hd + a.vd));
  const int n_units = page < 0 ? n_q : n_q + n_k + n_v;
  const float lam = v0 ? *a.lam : 0.f;
  for (int u = threadIdx.x; u < n_units; u += blockDim.x) {
    if (u < n_q + n_k) {
      const bool is_q = u < n_q;
      const int w = is_q ? u : u - n_q, per = is_q ? hc : kc, head = w / per, c = w - head * per;
      const bf16* src = p + (is_q ? (size_t)head * a.hd : (size_t)(a.H + head) * a.hd);
      bf16* dst = is_q ? const_cast<bf16*>(src) : rec + ((size_t)head * a.page_tokens + in_page) * a.hd;
      if (c < hc) {
        float x[8], y[8];
        rw_unpack8(*(const uint4*)(src + 8 * c), x); rw_unpack8(*(const uint4*)(src + half + 8 * c), y);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float sn = sn_s[8 * c + e], cs = cs_s[8 * c + e], xe = x[e];
          x[e] = xe * cs - y[e] * sn; y[e] = y[e] * cs + xe * sn;
        }
        *(uint4*)(dst + 8 * c) = rw_pack8(x); *(uint4*)(dst + half + 8 * c) = rw_pack8(y);
      } else {
        *(uint4*)(dst + half + 8 * c) = *(const uint4*)(src + half + 8 * c);
      }
    } else {
      const int w = u - n_q - n_k, g = w / vc, c = w - g * vc;
      uint4 val = *(const uint4*)(p + (size_t)(a.H + a.G) * a.hd + 8 * w);
      if (v0) {
        float x[8], y[8];
        rw_unpack8(val, x); rw_unpack8(*(const uint4*)(v0 + (size_t)row * a.ldv0 + 8 * w), y);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = (1.0f - lam) * x[e] + lam * y[e];
        val = rw_pack8(x);
      }
      *(uint4*)(rec + (size_t)a.G * a.page_tokens * a.hd + ((size_t)g * a.page_tokens + in_page) * a.vd + 8 * c) = val;
    }
  }
}

FELLM_API int fellm_qkv_rotate_write(void* qkv, int is_bf16, int ld, int T, int H, int G, int hd, int vd, int rot_dim,
                                     const float* inv_freq, int pairing, float mag, const void* v0, int ldv0, const float* lam,
                                     const int* positions, const int* row_slot, const int* block_table, int max_pages,
                                     void* pool, int cache_bf16, int page_tokens, int layer, int layers_in_group, int* status,
                                     cudaStream_t stream) {
  if (T <= 0) return 0;
  if (!inv_freq) rot_dim = 0;
  if (H < 1 || G < 1 || hd < 1 || vd < 1 || rot_dim < 0 || rot_dim > hd || (rot_dim & 1) || rot_dim > 2 * RWM_HALF || page_tokens < 1) return FELLM_ERR_SIZE;
  if (ld < H * hd + G * (hd + vd) || (v0 && ldv0 < G * vd)) return FELLM_ERR_SIZE;
  if (!qkv || !positions || !row_slot || !block_table || !pool || (v0 && !lam) || is_bf16 != cache_bf16) return FELLM_ERR_ARG;
  RotateWriteArgs a;
  a.ld = ld; a.H = H; a.G = G; a.hd = hd; a.vd = vd; a.rot_dim = rot_dim; a.pairing = pairing; a.ldv0 = ldv0; a.max_pages = max_pages;
  a.page_tokens = page_tokens; a.layer = layer; a.layers_in_group = layers_in_group; a.mag = mag; a.inv_freq = inv_freq; a.lam = lam;
  a.positions = positions; a.row_slot = row_slot; a.block_table = block_table; a.status = status;
  const int cls = launch_class_for_rows(T, 2);
  const bool vec = is_bf16 && (pairing == 1 || rot_dim == 0) && hd % 8 == 0 && vd % 8 == 0 && rot_dim % 16 == 0 && ld % 8 == 0 &&
                   (!v0 || (ldv0 % 8 == 0 && ((uintptr_t)v0 & 15) == 0)) && (((uintptr_t)qkv | (uintptr_t)pool) & 15) == 0;
  if (vec) return launch_k_class(cls, qkv_rotate_write_vec_kernel, dim3(T), dim3(128), 0, stream, 1, (bf16*)qkv, (const bf16*)v0, (bf16*)pool, a);
  if (is_bf16) return launch_k_class(cls, qkv_rotate_write_kernel<bf16>, dim3(T), dim3(128), 0, stream, 1, (bf16*)qkv, (const bf16*)v0, (bf16*)pool, a);
  return launch_k_class(cls, qkv_rotate_write_kernel<float>, dim3(T), dim3(128), 0, stream, 1, (float*)qkv, (const float*)v0, (float*)pool, a);
}

// ---------------------------------------------------------------- norm over the whole projection, rotation and the cache write
// The rows of the input product are [q (H hd) | k (G hd) | v (G vd) | ...], ld elements apart.  All of a row's q, and all
// of its k, are divided by their root mean square (eps inside the root) and multiplied by a weight per row element (qw
// [H hd], kw [G hd]); then every head is rotated on its first rot_dim elements (pairs (2i, 2i + 1) or (i, i + rot_dim/2)).
// q stays where it lies; k and v go into the row's page, a page-layer record being the keys [G][page_tokens][hd], then
// the values [G][page_tokens][vd].  G = 0: the rows hold no k and v (the layer reads another layer's pages).  A block a
// row; the row's sines and cosines and its page's number before the wait for the product; float32 throughout, rounded
// once; the sums' order depends on the sizes alone.
#define NRW_THREADS 256

struct NormRotateWriteArgs {
  int ld, H, G, hd, vd, rot_dim, pairing, max_pages, page_tokens, layer, layers_in_group;
  float eps;
  const float* inv_freq; const float* qw; const float* kw;
  const int* positions; const int* row_slot; const int* block_table;
  int* status;
};

// The block's sums of two values, the same in every thread: warps in order.
__device__ __forceinline__ void nrw_block_sums(float& x, float& y, float (*red)[NRW_THREADS / 32]) {
  const int warp = threadIdx.x >> 5;
  x = warp_sum(x); y = warp_sum(y);
  if ((threadIdx.x & 31) == 0) { red[0][warp] = x; red[1][warp] = y; }
  __syncthreads();
  x = y = 0.f;
#pragma unroll
  for (int w = 0; w < NRW_THREADS / 32; ++w) { x += red[0][w]; y += red[1][w]; }
}

template <typename T>
__global__ void __launch_bounds__(NRW_THREADS)
qkv_norm_rotate_write_kernel(T* __restrict__ qkv, T* __restrict__ pool, NormRotateWriteArgs a) {
  __shared__ float sn_s[RWM_HALF], cs_s[RWM_HALF], red[2][NRW_THREADS / 32];
  pdl_launch_dependents();
  const int row = blockIdx.x, pos = a.positions[row], half = a.rot_dim >> 1;
  const int page = a.G ? a.block_table[(size_t)a.row_slot[row] * a.max_pages + pos / a.page_tokens] : 0;
  for (int i = threadIdx.x; i < half; i += NRW_THREADS) sincosf((float)pos * a.inv_freq[i], &sn_s[i], &cs_s[i]);
  pdl_wait();
  T* p = qkv + (size_t)row * a.ld;
  const int nq = a.H * a.hd, nk = a.G * a.hd;
  float sq = 0.f, sk = 0.f;
  for (int e = threadIdx.x; e < nq; e += NRW_THREADS) { const float v = to_f(p[e]); sq = fmaf(v, v, sq); }
  for (int e = threadIdx.x; e < nk; e += NRW_THREADS) { const float v = to_f(p[nq + e]); sk = fmaf(v, v, sk); }
  nrw_block_sums(sq, sk, red);                       // (its barrier is also the one behind the sines and cosines)
  const float rq = 1.0f / sqrtf(sq / (float)nq + a.eps), rk = nk ? 1.0f / sqrtf(sk / (float)nk + a.eps) : 0.f;
  if (a.G && page < 0 && threadIdx.x == 0 && a.status) atomicExch(a.status, 2);          // never write outside the pool: record and skip
  const bool write = a.G && page >= 0;
  const int in_page = pos % a.page_tokens;
  T* rec = write ? pool + ((size_t)page * a.layers_in_group + a.layer) * ((size_t)a.G * a.page_tokens * (a.hd + a.vd)) : nullptr;
  const int per = a.hd - half, heads = a.H + (write ? a.G : 0);       // a pair, or one element behind the rotated part
  for (int u = threadIdx.x; u < heads * per; u += NRW_THREADS) {
    const int h = u / per, i = u - h * per;
    const bool is_q = h < a.H;
    const T* src = p + (size_t)h * a.hd;
    T* dst = is_q ? p + (size_t)h * a.hd : rec + ((size_t)(h - a.H) * a.page_tokens + in_page) * a.hd;
    const float* w = is_q ? a.qw + (size_t)h * a.hd : a.kw + (size_t)(h - a.H) * a.hd;
    const float r = is_q ? rq : rk;
    if (i < half) {
      const int ia = a.pairing ? i : 2 * i, ib = a.pairing ? i + half : 2 * i + 1;
      const float x = to_f(src[ia]) * r * w[ia], y = to_f(src[ib]) * r * w[ib];
      dst[ia] = from_f<T>(x * cs_s[i] - y * sn_s[i]); dst[ib] = from_f<T>(y * cs_s[i] + x * sn_s[i]);
    } else {
      dst[i + half] = from_f<T>(to_f(src[i + half]) * r * w[i + half]);
    }
  }
  if (!write) return;
  const T* vp = p + nq + nk;
  T* vrec = rec + (size_t)a.G * a.page_tokens * a.hd;
  for (int u = threadIdx.x; u < a.G * a.vd; u += NRW_THREADS) {
    const int g = u / a.vd, c = u - g * a.vd;
    vrec[((size_t)g * a.page_tokens + in_page) * a.vd + c] = vp[u];
  }
}

// bfloat16, hd and vd multiples of 8, rot_dim of 8 (pairs of neighbours: SPLIT false) or 16, rows on 16-byte boundaries:
// a thread eight elements by 16-byte loads and stores (and, SPLIT, the eight they are paired with).
template <bool SPLIT>
__global__ void __launch_bounds__(NRW_THREADS)
qkv_norm_rotate_write_vec_kernel(bf16* __restrict__ qkv, bf16* __restrict__ pool, NormRotateWriteArgs a) {
  __shared__ float sn_s[RWM_HALF], cs_s[RWM_HALF], red[2][NRW_THREADS / 32];
  pdl_launch_dependents();
  const int row = blockIdx.x, pos = a.positions[row], half = a.rot_dim >> 1;
  const int page = a.G ? a.block_table[(size_t)a.row_slot[row] * a.max_pages + pos / a.page_tokens] : 0;
  for (int i = threadIdx.x; i < half; i += NRW_THREADS) sincosf((float)pos * a.inv_freq[i], &sn_s[i], &cs_s[i]);
  pdl_wait();
  bf16* p = qkv + (size_t)row * a.ld;
  const int nq = a.H * a.hd, nk = a.G * a.hd;
  float sq = 0.f, sk = 0.f;
  for (int u = threadIdx.x; u < (nq + nk) >> 3; u += NRW_THREADS) {
    float x[8], s = 0.f;
    rw_unpack8(*(const uint4*)(p + 8 * u), x);
#pragma unroll
    for (int e = 0; e < 8; ++e) s = fmaf(x[e], x[e], s);
    if (8 * u < nq) sq += s; else sk += s;
  }
  nrw_block_sums(sq, sk, red);                       // (its barrier is also the one behind the sines and cosines)
  const float rq = 1.0f / sqrtf(sq / (float)nq + a.eps), rk = nk ? 1.0f / sqrtf(sk / (float)nk + a.eps) : 0.f;
  if (a.G && page < 0 && threadIdx.x == 0 && a.status) atomicExch(a.status, 2);          // never write outside the pool: record and skip
  const bool write = a.G && page >= 0;
  const int in_page = pos % a.page_tokens;
  bf16* rec = write ? pool + ((size_t)page * a.layers_in_group + a.layer) * ((size_t)a.G * a.page_tokens * (a.hd + a.vd)) : nullptr;
  const int hc = SPLIT ? half >> 3 : 0, per = (a.hd >> 3) - hc, vc = a.vd >> 3;
  const int n_heads = a.H * per + (write ? a.G * per : 0), n_units = n_heads + (write ? a.G * vc : 0);
  for (int u = threadIdx.x; u < n_units; u += NRW_THREADS) {
    if (u < n_heads) {
      const int h = u / per, c = u - h * per;
      const bool is_q = h < a.H;
      const bf16* src = p + (size_t)h * a.hd;
      bf16* dst = is_q ? p + (size_t)h * a.hd : rec + ((size_t)(h - a.H) * a.page_tokens + in_page) * a.hd;
      const float* w = is_q ? a.qw + (size_t)h * a.hd : a.kw + (size_t)(h - a.H) * a.hd;
      const float r = is_q ? rq : rk;
      const int at = (SPLIT && c >= hc) ? 8 * c + half : 8 * c;        // behind the rotated part, SPLIT skips its second half
      float x[8];
      rw_unpack8(*(const uint4*)(src + at), x);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = x[e] * r * w[at + e];
      if (SPLIT && c < hc) {
        float y[8];
        rw_unpack8(*(const uint4*)(src + half + at), y);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float sn = sn_s[at + e], cs = cs_s[at + e], xe = x[e], ye = y[e] * r * w[half + at + e];
          x[e] = xe * cs - ye * sn; y[e] = ye * cs + xe * sn;
        }
        *(uint4*)(dst + half + at) = rw_pack8(y);
      } else if (!SPLIT && at < a.rot_dim) {
#pragma unroll
        for (int e = 0; e < 8; e += 2) {
          const float sn = sn_s[(at + e) >> 1], cs = cs_s[(at + e) >> 1], xe = x[e], ye = x[e + 1];
          x[e] = xe * cs - ye * sn; x[e + 1] = ye * cs + xe * sn;
        }
      }
      *(uint4*)(dst + at) = rw_pack8(x);
    } else {
      const int w = u - n_heads, g = w / vc, c = w - g * vc;
      *(uint4*)(rec + (size_t)a.G * a.page_tokens * a.hd + ((size_t)g * a.page_tokens + in_page) * a.vd + 8 * c) =
          *(const uint4*)(p + nq + nk + 8 * w);
    }
  }
}

FELLM_API int fellm_qkv_norm_rotate_write(void* qkv, int is_bf16, int ld, int T, int H, int G, int hd, int vd, const float* qw,
                                          const float* kw, float eps, int rot_dim, const float* inv_freq, int pairing,
                                          const int* positions, const int* row_slot, const int* block_table, int max_pages,
                                          void* pool, int cache_bf16, int page_tokens, int layer, int layers_in_group, int* status,
                                          cudaStream_t stream) {
  if (T <= 0) return 0;
  if (!inv_freq) rot_dim = 0;
  if (H < 1 || G < 0 || hd < 1 || vd < 1 || rot_dim < 0 || rot_dim > hd || (rot_dim & 1) || rot_dim > 2 * RWM_HALF || page_tokens < 1) return FELLM_ERR_SIZE;
  if (ld < H * hd + G * (hd + vd)) return FELLM_ERR_SIZE;
  if (!qkv || !positions || !qw || (G && (!kw || !row_slot || !block_table || !pool || is_bf16 != cache_bf16))) return FELLM_ERR_ARG;
  NormRotateWriteArgs a;
  a.ld = ld; a.H = H; a.G = G; a.hd = hd; a.vd = vd; a.rot_dim = rot_dim; a.pairing = pairing; a.max_pages = max_pages;
  a.page_tokens = page_tokens; a.layer = layer; a.layers_in_group = layers_in_group; a.eps = eps; a.inv_freq = inv_freq;
  a.qw = qw; a.kw = kw; a.positions = positions; a.row_slot = row_slot; a.block_table = block_table; a.status = status;
  const int cls = launch_class_for_rows(T, 2);
  const bool vec = is_bf16 && hd % 8 == 0 && vd % 8 == 0 && rot_dim % (pairing ? 16 : 8) == 0 && ld % 8 == 0 &&
                   (((uintptr_t)qkv | (uintptr_t)pool) & 15) == 0;
  if (vec && pairing) return launch_k_class(cls, qkv_norm_rotate_write_vec_kernel<true>, dim3(T), dim3(NRW_THREADS), 0, stream, 1, (bf16*)qkv, (bf16*)pool, a);
  if (vec) return launch_k_class(cls, qkv_norm_rotate_write_vec_kernel<false>, dim3(T), dim3(NRW_THREADS), 0, stream, 1, (bf16*)qkv, (bf16*)pool, a);
  if (is_bf16) return launch_k_class(cls, qkv_norm_rotate_write_kernel<bf16>, dim3(T), dim3(NRW_THREADS), 0, stream, 1, (bf16*)qkv, (bf16*)pool, a);
  return launch_k_class(cls, qkv_norm_rotate_write_kernel<float>, dim3(T), dim3(NRW_THREADS), 0, stream, 1, (float*)qkv, (float*)pool, a);
}
