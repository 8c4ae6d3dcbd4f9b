"""The norm of blocks whose residual is a small set of parallel fp32 streams ("hyper-connections"):

    x_t <- sum_s mix[s, t] x_s + w_out[t] * scale * (branch + bias)      (the finished sublayer joins: all streams at once from the old ones)
    out = rms_norm(sum_s w_in[s] x_s) * w                                (what the next sublayer reads, in the activation dtype)

in one pass over the token's row (csrc/ragged/hyper_ops.cu `stream_mix_norm`).  Streams, sums, statistic and all weights are fp32 whatever the
activation dtype is.  The streams start equal: until the first join they are ONE row per token, afterwards a [tokens, streams, width] tensor."""
from typing import Optional, Tuple

import torch

from .... import kernels as K
from ....inference_parameter import InferenceParameter
from ....inference_utils import DtypeEnum, NormTypeEnum
from ...configs import DSNormConfig
from ...interfaces import DSPreNormBase, DSPreNormRegistry


@DSPreNormRegistry.register_module
class DSStreamMixRMSNorm(DSPreNormBase):

    @staticmethod
    def name() -> str:
        return "cuda_stream_mix_rms"

    @staticmethod
    def supports_config(config: DSNormConfig) -> bool:
        return (NormTypeEnum(config.type) == NormTypeEnum.RMSNorm and config.streams >= 1 and DtypeEnum(config.residual_dtype) == DtypeEnum.fp32 and
                config.weight_offset == 0.0 and DtypeEnum(config.input_dtype) in (DtypeEnum.bf16, DtypeEnum.fp32) and
                DtypeEnum(config.output_dtype) in (DtypeEnum.bf16, DtypeEnum.fp32))

    def transform_param(self, param: torch.Tensor) -> InferenceParameter:
        return InferenceParameter.initialize(param.to(torch.float32).contiguous())

    def forward(self, residual: torch.Tensor, hidden_states: Optional[Tuple], gamma: Optional[torch.Tensor], beta: Optional[torch.Tensor] = None,
                read: Optional[torch.Tensor] = None):
        """residual: fp32 streams [T, streams, width], or [T, width] while they are equal.  hidden_states: what has not joined them yet, (output,
        bias or None, scale, mix, w_out) as `kernels.stream_mix_norm` takes it, or None.  gamma: weight of the norm that feeds the next sublayer
        (None: only the join), read: the weights of the streams it reads.  Returns (streams, normed input or None)."""
        c = self._config
        assert beta is None, "RMS norms have no shift"
        return K.stream_mix_norm(residual, c.streams, hidden_states, read, gamma, c.eps, out_dtype=DtypeEnum(c.output_dtype).value)
