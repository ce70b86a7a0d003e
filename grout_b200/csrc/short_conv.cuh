// Short causal convolutions over time, one filter per channel, on the rows of a step: shared by
// the mixers that keep the last taps - 1 inputs of every sequence beside a recurrent state.
//
//   y_t = sum_j w[c, taps - 1 - j] x_{t - j}      (zeros in front of the sequence's start, no bias)
//
// An input lies in the step's rows, or, behind them, in the sequence's kept tail [taps - 1, Cc]
// (entry s: the input taps - 1 - s rows in front of the step's first).
#pragma once
#include "common.cuh"

#define SHORT_CONV_TAPS 8     // taps fetched together; more are walked in turns

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// Channel c of row t, the r-th its sequence brings.  `proj` rows are `ld` floats apart, channel c
// is column c; without a tail (a padding row) what lies in front of the step is zeros.
__device__ __forceinline__ float short_conv_silu(const float* proj, long long ld, const float* conv_w, int taps,
                                                 const float* tail, int Cc, int t, int r, int c) {
  float acc = 0.f;
  for (int j0 = 0; j0 < taps; j0 += SHORT_CONV_TAPS) {
    float x[SHORT_CONV_TAPS], w[SHORT_CONV_TAPS];
#pragma unroll
    for (int jj = 0; jj < SHORT_CONV_TAPS; ++jj) {     // all loads first: one trip to memory
      const int j = j0 + jj, rr = r - j;               // the input j tokens back
      x[jj] = 0.f, w[jj] = 0.f;
      if (j < taps) {
        w[jj] = conv_w[(size_t)c * taps + taps - 1 - j];
        if (rr >= 0) x[jj] = proj[(size_t)(t - j) * ld + c];
        else if (tail) x[jj] = tail[(size_t)(taps - 1 + rr) * Cc + c];
      }
    }
#pragma unroll
    for (int jj = 0; jj < SHORT_CONV_TAPS; ++jj) acc = fmaf(w[jj], x[jj], acc);
  }
  return silu_f(acc);
}

// The new tail of a sequence of n rows from row0 on: entry s becomes the input at n - (taps - 1) + s
// rows from the step's first; an entry that stays is read (at n + s > s) before anything at or above
// it is written.  The caller's threads share the channels: first, first + step, ...; every reader of
// the old tail must have finished.
__device__ __forceinline__ void short_conv_keep_tail(const float* proj, long long ld, int taps, float* tail, int Cc,
                                                     int row0, int n, int first, int step) {
  for (int c = first; c < Cc; c += step) {
    for (int s0 = 0; s0 < taps - 1; s0 += 8) {         // up to eight entries are read before any is written
      float v[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const int s = s0 + u, rr = n - (taps - 1) + s;
        v[u] = 0.f;
        if (s < taps - 1) v[u] = rr >= 0 ? proj[(size_t)(row0 + rr) * ld + c] : tail[(size_t)(taps - 1 + rr) * Cc + c];
      }
#pragma unroll
      for (int u = 0; u < 8; ++u)
        if (s0 + u < taps - 1) tail[(size_t)(s0 + u) * Cc + c] = v[u];
    }
  }
}

// Rows in runs of R (never fewer than taps - 1) that start at each sequence's first row: only a
// sequence's first run looks back behind the step, so the thread that owns a channel there can
// read the kept inputs and replace them afterwards.  Sequence s's runs are given the blocks
// cu_q[s] / R + s up to those of s + 1, which are never fewer than it needs and are found by
// bisection (the host need not know how rows divide into sequences); T / R + n_seqs blocks in all.
// `one_row`: every sequence brings one row, and block i is sequence i.
__device__ __forceinline__ void run_of_block(const int* cu_q, int n_seqs, int R, bool one_row, int block, int& seq,
                                             int& run) {
  seq = block, run = 0;
  if (one_row) return;
  int lo = 0, hi = n_seqs - 1;
  while (lo < hi) {                  // the last sequence whose first block is not behind this one
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] / R + mid <= block) lo = mid; else hi = mid - 1;
  }
  seq = lo, run = block - (cu_q[lo] / R + lo);
}
