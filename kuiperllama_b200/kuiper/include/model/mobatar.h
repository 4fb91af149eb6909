// Mobatar: a decoder-only family served by the sequence-batch engine.
//
//   x = embed[token] + bigram[(previous * mul_prev + token * mul_cur) mod buckets]     (first token: the row behind the buckets)
//   layers in the order config "layers" lists them; an entry with "weights_of" runs an earlier entry's weights again, with a
//   cache and a state of its own.  A layer has no norm ahead of its sublayers; each sublayer's OUTPUT is normed:
//       x += RMS(mixer(x)) (1 + norm1);   x += RMS(ff(x)) (1 + norm2)                  (the feed-forward is optional)
//   mixer 'attention':  rotary positions (halves paired) whose frequencies are kept, divided or blended by wavelength; q and k
//       divided by their root mean square AFTER the rotation; causal softmax with one added to the denominator; W_o
//   mixer 'parallel':   left_scale * A(x) + right_scale * R(x) with
//       A  softmax attention inside chunks of mask.size positions: one RMS norm over all query rows and one over all key rows,
//          rotary positions with divided frequencies, a sigmoid gate per head (W_g x), W_o
//       R  retention: rotated q and k, k * dim^-1/2, S <- decay_h S + k v^T, o = S^T q, each head's o divided by its root mean
//          square, times silu(W_g x), W_o
//   mixer 'latent_attention':  queries W_q x, per head [dim plain | rot_dim rotated]; keys and values through a latent of
//       kv_rank (RMS norm, then W_uk / W_uv per head) and one rotated key part shared by all heads; neighbouring coordinates are
//       rotated together; a sliding window; W_o
//   ff 'dense': g = min(gate x + b, limit), u = clamp(up x + b, -limit, limit): down(g sigmoid(1.702 g) (u + 1)) + b
//   logits = head . (RMS(x) (1 + final.norm))
//
// The class only translates config.json and the tensor names into the engine's layer descriptors; every size and
// constant comes from the configuration or from a tensor's shape.
#ifndef KLLM_KUIPER_MODEL_MOBATAR_H_
#define KLLM_KUIPER_MODEL_MOBATAR_H_
#include "sequence_model.h"

namespace model {
class MobatarModel final : public SequenceModel {
 protected:
  base::Status build(const json::Value& config, const SafetensorsFile& weights) override;
  base::Status check_folder(const json::Value& config, const SafetensorsFile& weights) override;

 private:
  // the sizes, projections, rotation and mask that every softmax attention of the family has
  base::Status build_attention(const json::Value& mixer, const SafetensorsFile& w, const std::string& prefix, bool gated,
                               kllm_seq_attention* out);
  base::Status build_retention(const json::Value& mixer, const SafetensorsFile& w, const std::string& prefix,
                               kllm_seq_linear* out);
  base::Status build_latent(const json::Value& mixer, const SafetensorsFile& w, const std::string& prefix, kllm_seq_latent* out);
  base::Status build_dense(const json::Value& mlp, const SafetensorsFile& w, const std::string& prefix, kllm_seq_dense* out);
  // a "rot" entry: dims, base and, on the device, the angle per position of every pair
  base::Status build_rotation(const json::Value& mixer, const std::string& prefix, int32_t limit, int32_t* dims, float* base,
                              const float** freq);
  // RMS norm over the model width whose stored weight is the distance from one
  base::Status centred_norm(const SafetensorsFile& w, const std::string& name, kllm_seq_norm* out);
};
}  // namespace model
#endif  // KLLM_KUIPER_MODEL_MOBATAR_H_
