"""The "norm" of blocks whose sublayers read tanh(alpha x) * w + b of an fp32 residual stream: no mean, no variance, nothing of the row enters but
the value itself.

    x <- x + (outputs of the previous layer's sublayers)        (a plain fp32 sum; the outputs arrive in the activation dtype or fp32)
    out = tanh(alpha x) * w + b                                 (the input of every sublayer of this layer, in the activation dtype)

in one pass (csrc/ragged/latent_ops.cu `stream_tanh_norm`).  alpha (one number), w, b and the stream are fp32 whatever the activation dtype is."""
from typing import Optional, Sequence

import torch

from .... import kernels as K
from ....inference_parameter import InferenceParameter
from ....inference_utils import DtypeEnum, NormTypeEnum
from ...configs import DSNormConfig
from ...interfaces import DSPreNormBase, DSPreNormRegistry


@DSPreNormRegistry.register_module
class DSDynamicTanhNorm(DSPreNormBase):

    @staticmethod
    def name() -> str:
        return "cuda_dynamic_tanh"

    @staticmethod
    def supports_config(config: DSNormConfig) -> bool:
        return (NormTypeEnum(config.type) == NormTypeEnum.DynamicTanh and config.shared_input and DtypeEnum(config.residual_dtype) == DtypeEnum.fp32 and
                config.weight_offset == 0.0 and DtypeEnum(config.input_dtype) in (DtypeEnum.bf16, DtypeEnum.fp32) and
                DtypeEnum(config.output_dtype) in (DtypeEnum.bf16, DtypeEnum.fp32))

    def transform_param(self, param: torch.Tensor) -> InferenceParameter:
        """Weight, shift and alpha (a scalar: stored as one entry)."""
        return InferenceParameter.initialize(param.to(torch.float32).reshape(-1).contiguous())

    def forward(self, residual: torch.Tensor, hidden_states: Optional[Sequence[torch.Tensor]], gamma: Optional[torch.Tensor],
                beta: Optional[torch.Tensor] = None, alpha: Optional[torch.Tensor] = None, fp32_branch: Optional[torch.Tensor] = None,
                fp32_copy: bool = False):
        """residual: fp32 stream (updated in place).  hidden_states: the finished sublayers' outputs in the activation dtype (a tensor, up to
        two tensors, or None); fp32_branch: one more output that is already fp32.  gamma / beta / alpha: weight, shift and slope, None when only
        the sum is wanted.  Returns (residual, result or None); with `fp32_copy` a third value: the result before its rounding."""
        branches = () if hidden_states is None else ((hidden_states, ) if torch.is_tensor(hidden_states) else tuple(hidden_states))
        out = K.stream_tanh_norm(residual, branches, fp32_branch, alpha, gamma, beta, out_dtype=DtypeEnum(self._config.output_dtype).value, fp32_copy=fp32_copy)
        if fp32_copy:
            return residual, out[0], out[1]
        return residual, out
