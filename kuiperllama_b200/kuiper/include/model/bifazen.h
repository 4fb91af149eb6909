// Bifazen: a decoder-only family served by the sequence-batch engine.
//
//   the residual is config "streams" rows x_1 .. x_S, all equal to embed[token] at the start (hyper-connections);
//   layers in the order config "layers" lists them, each with a mixer and an optional feed-forward.  A sublayer reads
//       u = sum_s in_s x_s,    y = sublayer(RMS(u) (1 + norm)),    and    x_t <- sum_s mix_st x_s + out_t y
//   mixer 'latent_attention':  queries W_q h, per head [dim plain | rot_dim rotated]; keys and values through a latent of
//       kv_rank (RMS norm, then W_uk / W_uv per head) and one rotated key part shared by all heads; neighbouring coordinates
//       are rotated together; a sliding window; W_o
//   mixer 'attention':  W_q h + b, W_k h + b, W_v h + b; one RMS norm over all query rows and one over all key rows; no
//       positions; a sliding window; in layers with v_mix, v <- (1 - lambda) v + lambda v_first, v_first being the values of
//       the first such layer; a sigmoid gate per head (W_g h); W_o + b
//   ff 'dense': down(gelu(gate h) * up h), the tanh form of gelu
//   logits = embed . (RMS(sum_s x_s) (1 + final.norm))
//
// The class only translates config.json and the tensor names into the engine's layer descriptors; every size and
// constant comes from the configuration or from a tensor's shape.
#ifndef KLLM_KUIPER_MODEL_BIFAZEN_H_
#define KLLM_KUIPER_MODEL_BIFAZEN_H_
#include "sequence_model.h"

namespace model {
class BifazenModel final : public SequenceModel {
 protected:
  base::Status build(const json::Value& config, const SafetensorsFile& weights) override;
  base::Status check_folder(const json::Value& config, const SafetensorsFile& weights) override;

 private:
  base::Status build_latent(const json::Value& mixer, const SafetensorsFile& w, const std::string& prefix, kllm_seq_latent* out);
  // `v_blend`: KLLM_SEQ_VBLEND_*
  base::Status build_attention(const json::Value& mixer, const SafetensorsFile& w, const std::string& prefix, int32_t v_blend,
                               kllm_seq_attention* out);
  base::Status build_dense(const json::Value& mlp, const SafetensorsFile& w, const std::string& prefix, kllm_seq_dense* out);
  // RMS norm over the model width whose stored weight is the distance from one
  base::Status centred_norm(const SafetensorsFile& w, const std::string& name, kllm_seq_norm* out);
  base::Status hyper(const SafetensorsFile& w, const std::string& prefix, kllm_seq_hyper* out);
};
}  // namespace model
#endif  // KLLM_KUIPER_MODEL_BIFAZEN_H_
