#include <torch/types.h>
namespace tk {
using OptT = c10::optional<torch::Tensor>;
bool latent_decode_tc(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, double, const torch::Tensor&, const OptT&, torch::Tensor&) { return false; }
}
