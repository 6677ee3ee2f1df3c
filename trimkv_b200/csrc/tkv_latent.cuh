// Latent attention: keys and values of all heads are linear maps of one latent vector per position, plus one rotated key part
// that the heads share.  Score = (q_plain . k_plain + q_turned . k_turned) * scale over a sliding window.
//
// A position is held as one row of lw = cpad + rpad elements: the normed latent c zero-padded to cpad, the rotated key part
// zero-padded to rpad (multiples of 64).  Two storages: ring [slots, rows, lw], position p in row p mod rows; linear
// [rows, lw], one step's tokens, each request's part preceded by the positions its window still reaches.
#pragma once
#include "tkv_elem.cuh"

namespace tkv {

// Attention with keys in two parts, of any layout.  Rows are linear (kv_start) or of a ring (slots, ring_rows > 0, one token
// per request); head strides of 0 share a part between the heads.
struct TwoPartAttn {
  const void* q1; int64_t q1_token, q1_head; int d1;
  const void* q2; int64_t q2_token, q2_head; int d2;
  const void* k1; int64_t k1_row, k1_head;
  const void* k2; int64_t k2_row;
  const void* v; int64_t v_row, v_head; int vdim;
  void* out; int64_t out_token, out_head;
  const int32_t* slots; int ring_rows;
  const int32_t* kv_start; const int32_t* cu; const int32_t* pos0;
  int batch, tokens, heads, window;
  float scale;
  int32_t* status;
};

int launch_two_part_any(const char* what, const TwoPartAttn& p, int dtype, cudaStream_t st);
// The tcgen05 form for prompts (tkv_latent_tc.cu): shapes it takes.
bool two_part_tc_shape(const TwoPartAttn& p, int dtype);
int launch_two_part_tc(const TwoPartAttn& p, int64_t kv_rows, int max_tokens, cudaStream_t st);

}  // namespace tkv
