// Decayed sums (REC_DECAY of recurrent_mixers.cuh: S <- c S + k v^T, o = S^T q with one constant c per head) of prompt portions in
// matrix form on the tensor cores, bf16 engines.  A chunk is up to 64 consecutive tokens of one run; with the state S before it and
// its rows counted from 0,
//
//   o_i = c^(i+1) S^T q_i + sum_{j <= i} c^(i-j) <q_i, k_j> v_j          S <- c^n S + sum_j c^(n-1-j) k_j v_j^T
//
// decayed_chunks_kernel   one CTA per (run, head, 16 value columns) walks the run's chunks in order.  Warps 0-3 take 16 query rows each
//                         (S^T q, then the masked products), warps 4-7 hold the state (fp32 accumulators of mma.sync m16n8k16) and add the
//                         chunk to it at the same time.  q, k, v are the bf16 values of the projections; everything else is fp32: where an
//                         fp32 operand (the state, the decayed products, the decayed values) enters an MMA it goes in as TWO bf16 parts,
//                         hi = bf16(x) and lo = bf16(x - hi), so a product keeps 17 bits of it; powers of c are taken by powf.
//
// Chunks are counted from the start of the portion, so how a prompt is cut changes the order of the additions and nothing else.
#pragma once

#include "multi_attention.cuh"
#include "recurrent_mixers.cuh"

namespace mtx {

constexpr int kDcTokens = 64, kDcCols = 16, kDcThreads = 256, kDcVPitch = kDcCols + 8;

struct DecayedChunksArgs {
  const void* src;     // [rows, ld]: q at q_col, k at k_col, v at v_col (heads x dim, heads x dim, heads x vdim), SRC = bf16 or fp32 that holds bf16 values
  long long ld;
  int q_col, k_col, v_col;
  float* o;            // [rows, heads * vdim]
  float* state;        // [slots, heads, vdim, dim]
  const float* head_decay;
  const int* run_row0;
  const int* group;
  const int* pos;
  int heads, dim, vdim;
  float q_scale;
  int vec8;            // SRC = bf16: ld, the columns, dim and vdim are multiples of 8 and src is 16-byte aligned
};

// stage s: Q [64][dp + 8], K [64][dp + 8], V [64][24]; then the state [hi, lo][16][dp + 8], the decayed values [hi, lo][64][24], the powers [65]
inline size_t decayed_chunks_smem_bytes(int dim) {
  const size_t dp = size_t(mat_pad16(dim)) + 8;
  return sizeof(bf16) * (2 * (2 * kDcTokens * dp + kDcTokens * kDcVPitch) + 2 * kDcCols * dp + 2 * kDcTokens * kDcVPitch) + sizeof(float) * (kDcTokens + 4);
}

// x = hi + lo + (what 16 bits do not hold)
__device__ __forceinline__ void dc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = smax_pack_bf16(x - f.x, y - f.y);
}

__device__ __forceinline__ void dc_cp_async_16(bf16* dst, const bf16* src, bool ok) {
  const int n = ok ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(n) : "memory");
}

// MT: 16-channel tiles of the state per warp of warps 4-7 (dim <= 64 MT)
template <typename SRC, int MT>
__global__ void __launch_bounds__(kDcThreads) decayed_chunks_kernel(const DecayedChunksArgs a) {
  extern __shared__ __align__(16) unsigned char dc_raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int d = a.dim, dv = a.vdim, H = a.heads, dp = (d + 15) & ~15, DP = dp + 8;
  const int stage_elems = 2 * kDcTokens * DP + kDcTokens * kDcVPitch;
  bf16* const stage0 = reinterpret_cast<bf16*>(dc_raw);
  bf16* const sS = stage0 + 2 * stage_elems;         // state, transposed: [hi, lo][16 columns][DP]
  bf16* const sW = sS + 2 * kDcCols * DP;            // decayed values [hi, lo][64][24]
  float* const pw = reinterpret_cast<float*>(sW + 2 * kDcTokens * kDcVPitch);  // c^0 .. c^64
  griddep_wait();
  const int r0 = a.run_row0[blockIdx.x], nr = a.run_row0[blockIdx.x + 1] - r0, h = blockIdx.y, col0 = int(blockIdx.z) * kDcCols;
  if (nr <= 0) return;
  const float decay = a.head_decay[h];
  if (tid <= kDcTokens) pw[tid] = tid == 0 ? 1.0f : powf(decay, float(tid));
  const int n_chunks = (nr + kDcTokens - 1) / kDcTokens;
  const SRC* const src = static_cast<const SRC*>(a.src) + size_t(r0) * a.ld;

  auto load_chunk = [&](int c, int stage) {
    bf16* sq = stage0 + size_t(stage) * stage_elems;
    bf16* sk = sq + kDcTokens * DP;
    bf16* sv = sk + kDcTokens * DP;
    const int t0 = c * kDcTokens;
    if constexpr (sizeof(SRC) == 2) {
      if (a.vec8) {
        const int ch = dp / 8;
        for (int e = tid; e < kDcTokens * ch; e += kDcThreads) {
          const int i = e / ch, x = (e % ch) * 8;
          const bool ok = t0 + i < nr && x < d;
          const SRC* row = src + size_t(ok ? t0 + i : 0) * a.ld + h * d + (ok ? x : 0);
          dc_cp_async_16(sq + i * DP + x, row + a.q_col, ok);
          dc_cp_async_16(sk + i * DP + x, row + a.k_col, ok);
        }
        for (int e = tid; e < kDcTokens * 2; e += kDcThreads) {
          const int i = e >> 1, x = (e & 1) * 8;
          const bool ok = t0 + i < nr && col0 + x < dv;
          dc_cp_async_16(sv + i * kDcVPitch + x, src + size_t(ok ? t0 + i : 0) * a.ld + a.v_col + h * dv + (ok ? col0 + x : 0), ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        return;
      }
    }
    for (int e = tid; e < kDcTokens * dp; e += kDcThreads) {
      const int i = e / dp, x = e % dp;
      const bool ok = t0 + i < nr && x < d;
      const SRC* row = src + size_t(ok ? t0 + i : 0) * a.ld + h * d + (ok ? x : 0);
      sq[i * DP + x] = __float2bfloat16_rn(ok ? act_f32(row[a.q_col]) : 0.0f);
      sk[i * DP + x] = __float2bfloat16_rn(ok ? act_f32(row[a.k_col]) : 0.0f);
    }
    for (int e = tid; e < kDcTokens * kDcCols; e += kDcThreads) {
      const int i = e / kDcCols, x = e % kDcCols;
      const bool ok = t0 + i < nr && col0 + x < dv;
      sv[i * kDcVPitch + x] = __float2bfloat16_rn(ok ? act_f32(src[size_t(t0 + i) * a.ld + a.v_col + h * dv + col0 + x]) : 0.0f);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // warps 4-7: the state's channel tiles m = (warp - 4) + 4 u; S[u][nt]: channels 16 m + g / + 8, columns col0 + 8 nt + 2 t / + 1
  const bool fresh = a.pos[r0] == 0;
  float* const gs = a.state + (size_t(a.group[r0]) * H + h) * dv * d;
  float S[MT][2][4];
  auto state_at = [&](int u, int nt, int e, int& ch, int& col) {
    ch = ((warp & 3) + 4 * u) * 16 + g + (e & 2) * 4;
    col = col0 + nt * 8 + 2 * t + (e & 1);
    return warp >= 4 && ch < d && col < dv;
  };
#pragma unroll
  for (int u = 0; u < MT; ++u)
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        int ch, col;
        const bool ok = state_at(u, nt, e, ch, col) && !fresh;
        S[u][nt][e] = ok ? gs[size_t(col) * d + ch] : 0.0f;
      }
  load_chunk(0, 0);
  for (int c = 0; c < n_chunks; ++c) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // chunk c has landed; everybody is done with chunk c - 1
    if (c + 1 < n_chunks) load_chunk(c + 1, (c + 1) & 1);
    const bf16* sq = stage0 + size_t(c & 1) * stage_elems;
    const bf16* sk = sq + kDcTokens * DP;
    const bf16* sv = sk + kDcTokens * DP;
    const int t0 = c * kDcTokens, n = nr - t0 < kDcTokens ? nr - t0 : kDcTokens;
    if (warp >= 4) {  // the state before the chunk, as an operand
#pragma unroll
      for (int u = 0; u < MT; ++u) {
        const int ch = ((warp & 3) + 4 * u) * 16 + g;
        if (ch < dp) {
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float x = S[u][nt][e];
              const bf16 hi = __float2bfloat16_rn(x);
              bf16* dst = sS + (nt * 8 + 2 * t + (e & 1)) * DP + ch + (e & 2) * 4;
              dst[0] = hi;
              dst[kDcCols * DP] = __float2bfloat16_rn(x - __bfloat162float(hi));
            }
        }
      }
    } else {  // the values, each decayed to the end of the chunk (rows beyond the run: zero)
      for (int e = tid; e < kDcTokens * (kDcCols / 2); e += 128) {
        const int i = e >> 3, x = (e & 7) * 2;
        const float w = i < n ? pw[n - 1 - i] : 0.0f;
        const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sv + i * kDcVPitch + x));
        uint32_t hi, lo;
        dc_split(w * v.x, w * v.y, hi, lo);
        *reinterpret_cast<uint32_t*>(sW + i * kDcVPitch + x) = hi;
        *reinterpret_cast<uint32_t*>(sW + (kDcTokens + i) * kDcVPitch + x) = lo;
      }
    }
    __syncthreads();
    if (warp >= 4) {
      const float keep = pw[n];
      const int kts = (n + 15) >> 4;
#pragma unroll
      for (int u = 0; u < MT; ++u) {
        const int m = (warp & 3) + 4 * u;
        if (m * 16 < dp) {
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[u][nt][e] *= keep;
          for (int kt = 0; kt < kts; ++kt) {
            uint32_t kf[4], wh[4], wl[4];
            mat_ldsm_x4_trans(kf, sk + (kt * 16 + (lane & 7) + (lane >> 4) * 8) * DP + m * 16 + ((lane >> 3) & 1) * 8);
            const bf16* w0 = sW + (kt * 16 + (lane & 15)) * kDcVPitch + (lane >> 4) * 8;
            mat_ldsm_x4_trans(wh, w0);
            mat_ldsm_x4_trans(wl, w0 + kDcTokens * kDcVPitch);
            mma_bf16_16816(S[u][0], kf, wh[0], wh[1]);
            mma_bf16_16816(S[u][1], kf, wh[2], wh[3]);
            mma_bf16_16816(S[u][0], kf, wl[0], wl[1]);
            mma_bf16_16816(S[u][1], kf, wl[2], wl[3]);
          }
        }
      }
    } else if (warp * 16 < n) {
      const int i0 = warp * 16 + g, i1 = i0 + 8;  // this thread's rows of the chunk
      float o[2][4], p[8][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[nt][e] = 0.0f;
#pragma unroll
      for (int nb = 0; nb < 8; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) p[nb][e] = 0.0f;
      const bf16* qa = sq + (warp * 16 + (lane & 15)) * DP + (lane >> 4) * 8;
      const int brow = (lane & 7) + (lane >> 4) * 8, bcol = ((lane >> 3) & 1) * 8;
#pragma unroll 2
      for (int k0 = 0; k0 < dp; k0 += 16) {
        uint32_t qf[4], bf[4];
        mat_ldsm_x4(qf, qa + k0);
        mat_ldsm_x4(bf, sS + brow * DP + bcol + k0);
        mma_bf16_16816(o[0], qf, bf[0], bf[1]);
        mma_bf16_16816(o[1], qf, bf[2], bf[3]);
        mat_ldsm_x4(bf, sS + (kDcCols + brow) * DP + bcol + k0);
        mma_bf16_16816(o[0], qf, bf[0], bf[1]);
        mma_bf16_16816(o[1], qf, bf[2], bf[3]);
#pragma unroll
        for (int kb = 0; kb < 4; ++kb)
          if (kb <= warp) {  // keys after the warp's last row are not seen
            mat_ldsm_x4(bf, sk + (kb * 16 + brow) * DP + bcol + k0);
            mma_bf16_16816(p[2 * kb], qf, bf[0], bf[1]);
            mma_bf16_16816(p[2 * kb + 1], qf, bf[2], bf[3]);
          }
      }
      const float c0 = pw[i0 + 1], c1 = pw[i1 + 1];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        o[nt][0] *= c0;
        o[nt][1] *= c0;
        o[nt][2] *= c1;
        o[nt][3] *= c1;
      }
#pragma unroll
      for (int kb = 0; kb < 4; ++kb)
        if (kb <= warp) {
          uint32_t ph[4], pl[4], vf[4];
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            float* q = p[2 * kb + half];
            const int j = kb * 16 + half * 8 + 2 * t;
            q[0] = j <= i0 ? q[0] * pw[i0 - j] : 0.0f;
            q[1] = j + 1 <= i0 ? q[1] * pw[i0 - j - 1] : 0.0f;
            q[2] = j <= i1 ? q[2] * pw[i1 - j] : 0.0f;
            q[3] = j + 1 <= i1 ? q[3] * pw[i1 - j - 1] : 0.0f;
            dc_split(q[0], q[1], ph[2 * half], pl[2 * half]);
            dc_split(q[2], q[3], ph[2 * half + 1], pl[2 * half + 1]);
          }
          mat_ldsm_x4_trans(vf, sv + (kb * 16 + (lane & 15)) * kDcVPitch + (lane >> 4) * 8);
          mma_bf16_16816(o[0], ph, vf[0], vf[1]);
          mma_bf16_16816(o[1], ph, vf[2], vf[3]);
          mma_bf16_16816(o[0], pl, vf[0], vf[1]);
          mma_bf16_16816(o[1], pl, vf[2], vf[3]);
        }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = (e & 2) ? i1 : i0, col = col0 + nt * 8 + 2 * t + (e & 1);
          if (i < n && col < dv) a.o[size_t(r0 + t0 + i) * H * dv + h * dv + col] = o[nt][e] * a.q_scale;
        }
    }
  }
#pragma unroll
  for (int u = 0; u < MT; ++u)
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        int ch, col;
        if (state_at(u, nt, e, ch, col)) gs[size_t(col) * d + ch] = S[u][nt][e];
      }
}

}  // namespace mtx
