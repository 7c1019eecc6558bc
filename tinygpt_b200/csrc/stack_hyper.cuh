// stack_hyper.cuh — hyper-connected blocks (stack_hyper.cu): `streams` copies of the residual stream that every sublayer reads
// as a weighted sum and writes back through a small matrix, the pre-norm and the short input convolution behind it, and the
// token shift (each row blended with the row before it) a time-mixing mixer reads.  The copies, the norms and the convolution
// are fp32; T = bf16 or fp32 is the type of the operand rows that leave.
#pragma once
#include "stack.cuh"

namespace b200 {

constexpr int kMaxStreams = 8;
constexpr int kConvMaxTaps = 16;
constexpr int kShiftMixes = 5;

// What a mixer's input convolution and token shift need.  h_t = n_t + Σ_j w[taps − 1 − j]·n_(t − j) over the normed rows n
// (zeros before the sequence); with mu:  mix_s = h_t + (h_(t−1) − h_t)·mu_s for kShiftMixes vectors mu_s.
// The slot keeps the last `taps` normed rows, oldest first ([taps][width] fp32): h_(t−1) is built from them again, so a
// decoded token sees exactly the value a prompt would have used.
struct InputConv {
  int taps = 1;
  const float* w = nullptr;      // [taps][width], last row meets the current token; null: no convolution (h = n)
  const float* mu = nullptr;     // [kShiftMixes][width] or null
  void* h = nullptr;             // [n_tok, width] T, or null when only the mixes are read
  void* mix = nullptr;           // [kShiftMixes][n_tok][width] T
  float* state = nullptr;        // slot 0's rows; slot s is s·slot_stride floats further
  int64_t slot_stride = 0;
};

// One pass over the rows of the stream:
//   x_d <- Σ_s mix[s][d]·x_s + mult·out[d]·y       (y given: the previous sublayer's output; else the copies stay)
//   u = Σ_s in[s]·x_s                               (in null: the plain sum)
//   n = u·rsqrt(mean(u²) + eps)·(offset + norm_w)   (norm_w null: n = u)
// and n leaves as T (h), as fp32 (hn), or — `conv`, every row its sequence's only new row — through the input convolution.
struct HyperStep {
  int streams = 1, width = 0, n_tok = 0;
  float* x = nullptr;            // [n_tok][streams][width]
  const void* y = nullptr;       // [n_tok, width] fp32 or bf16
  bool y_bf16 = false;
  b200_hyper_desc prev{};        // of the sublayer that produced y (null pointers: plain residual, one stream)
  float mult = 1.f;
  const float* in = nullptr;
  const float* norm_w = nullptr;
  float eps = 1e-5f, offset = 0.f;
  void* h = nullptr;
  float* hn = nullptr;
  bool conv = false;
  InputConv c{};
  const int32_t* slot = nullptr;
  const int32_t* pos = nullptr;
};
int launch_hyper_step(const HyperStep& p, int dtype, cudaStream_t st);
// x[t][s][:] = float(embed[tok[t], :])·scale for every copy s
int launch_hyper_embed(float* x, const void* embed, const int32_t* tok, int64_t n_tok, int vocab, int width, int streams, float scale,
                       int dtype, cudaStream_t st);
// The input convolution (and token shift) of a step's rows hn [n_tok, width]; the state is only read (launch_shift_state moves
// it on).
int launch_input_conv(const InputConv& c, const float* hn, const int32_t* slot, const int32_t* pos, int n_tok, int width, int dtype,
                      cudaStream_t st);

// Moves "last `keep` input rows" states on, after everything that reads them has been launched: for every sequence of the
// step (rows [row0, row0 + count)) entry i becomes the row keep − 1 − i positions before its last one, from the step's rows
// or from the old entries (zeros before the sequence).
struct ShiftSource {
  const void* rows = nullptr;    // [n_tok, ld], T or fp32
  bool f32 = false;
  int64_t ld = 0;
  int channels = 0, keep = 0;
  float* state = nullptr;        // slot 0's [keep][channels]
};
constexpr int kShiftSources = 4;
struct ShiftState {
  ShiftSource src[kShiftSources];
  int n_src = 0;
  const int32_t* seg_row0 = nullptr;
  const int32_t* seg_count = nullptr;
  const int32_t* slot = nullptr;
  const int32_t* pos = nullptr;
  int n_seg = 0;
  int64_t slot_stride = 0;
};
int launch_shift_state(const ShiftState& p, int dtype, cudaStream_t st);

#ifdef __CUDACC__
// Row t − j of the step is position pos[t] − j of the same sequence exactly when it has the same slot and that position: the
// rows of a sequence lie side by side, in order.
__device__ __forceinline__ bool row_same_seq(const int32_t* slot, const int32_t* pos, int t, int j) {
  return t - j >= 0 && slot[t - j] == slot[t] && pos[t - j] == pos[t] - j;
}
// rows [t0, t1) are one sequence's, in order (a sequence's rows lie side by side in a step, so the ends tell)
__device__ __forceinline__ bool rows_one_seq(const int32_t* slot, const int32_t* pos, int t0, int t1) {
  return slot[t0] == slot[t1 - 1] && pos[t1 - 1] - pos[t0] == t1 - 1 - t0;
}
// rows of this sequence in front of row t, counted up to `most`
__device__ __forceinline__ int rows_in_front(const int32_t* slot, const int32_t* pos, int t, int most) {
  int n = 0;
  while (n < most && row_same_seq(slot, pos, t, n + 1)) ++n;
  return n;
}
#endif

}  // namespace b200
