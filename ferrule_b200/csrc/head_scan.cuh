// Parameters of the head-decay scan kernels (head_scan.cu, head_scan_chunk.cu).
#pragma once
#include "common.cuh"

namespace fb {

template <typename T>
struct HeadScanParams {
  const T* xbc;
  long long ldx;
  int off_b, off_c;
  const T* dt;
  const T* z;
  long long ldp;
  const float* dt_bias;
  const float* a_neg;
  const float* d_skip;
  float* states;
  const int* seq_start;
  const int* state_in;
  const int* state_out;
  T* out;
  long long ldo;
  int rows, n_seqs, heads, vdim, state, groups, n_states, out_cols;
  int skip_single;                  // sequences with one row are another launch's
  DeviceStatus* status;
};

// state buffers of a sequence; false: the indices are out of range
template <typename T>
__device__ __forceinline__ bool scan_bind(const HeadScanParams<T>& p, int seq, int& sin, int& sout) {
  sin = p.state_in[seq];
  sout = p.state_out[seq];
  return sin < p.n_states && sout < p.n_states && !(sin >= 0 && sin == sout);
}

// whether the chunked form takes a mixer of these sizes
inline bool head_scan_chunk_ok(int vdim, int state, int groups) {
  return vdim % 8 == 0 && state <= 128 && (state % 8 == 0 || groups == 1);
}
int run_head_scan_chunk(const HeadScanParams<__nv_bfloat16>& p, cudaStream_t stream);

}  // namespace fb
