// The sampler's binding, part of both torch modules.
#pragma once
#include "binding_util.h"
#include "kernels/api.h"

namespace {

void sample_tokens(const Tensor& logits, const OptTensor& history, const OptTensor& allow_mask, double temperature,
                   int64_t top_k, double top_p, double repetition_penalty, int64_t seed, Tensor& out_tokens,
                   OptTensor out_logprob) {
  const bool f32 = logits.scalar_type() == F32;
  chk(logits, f32 ? F32 : BF16, "logits");
  chk_c(out_tokens, I32, "out_tokens");
  TORCH_CHECK(logits.dim() == 2 && logits.stride(1) == 1, "sample_tokens: logits must be [rows, vocab]");
  const int* hist = nullptr;
  int hist_len = 0;
  if (history.has_value()) {
    chk_c(*history, I32, "history");
    hist = history->data_ptr<int>();
    hist_len = (int)history->size(1);
  }
  mb::SamplerArgs a{(float)temperature, (float)top_p, (float)repetition_penalty, (int)top_k,
                    (unsigned long long)seed};
  c10::cuda::CUDAGuard guard(logits.device());
  mb::sample_tokens(logits.data_ptr(), logits.stride(0), (int)logits.size(0), (int)logits.size(1), hist, hist_len,
                    allow_mask.has_value() ? allow_mask->data_ptr<unsigned char>() : nullptr, a,
                    out_tokens.data_ptr<int>(), out_logprob.has_value() ? out_logprob->data_ptr<float>() : nullptr,
                    nullptr, cur_stream(), f32);
}

}  // namespace
