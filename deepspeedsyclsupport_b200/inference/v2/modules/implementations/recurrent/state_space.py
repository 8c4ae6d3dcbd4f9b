"""State-space mixer with one decay per head (state-space duality).

Per layer and step, from the fused projection: `ssd_prepare` (convolution with bias and silu over x | B | C, step sizes and log decays per head),
`conv_state_update` (the last taps - 1 rows become the sequence's state), the recurrence, and `gated_group_norm` (times silu(z), RMS norm in
equal parts, weight).  csrc/ragged/ssd_ops.cu.

Two forms of the recurrence.  `ssd_scan`: token by token with the state in registers, any sizes, fp32 arithmetic for both activation dtypes --
decode steps, short portions, fp32.  `ssd_chunk` (csrc/ragged/ssd_chunk.cu): chunks of 128 tokens as matrix products on the tensor cores, bf16
with state rows up to 128 and columns up to 64 -- the sequences of a step that bring at least CHUNK_MIN tokens.  The state of a
head lives in the state manager's slots as fp32 [state_size, value_size] and starts at zero (a sequence at position 0 ignores what its slot
held)."""
from typing import Any, Dict, List, Type

import torch

from .... import kernels as K
from ....inference_parameter import InferenceParameter
from ....inference_utils import DtypeEnum
from ....ragged.state_slots import StateBufferSpec
from ...configs import DSStateSpaceConfig
from ...interfaces import DSRecurrentMixerBase, DSRecurrentRegistry

CHUNK_MIN = 32  # new tokens of a sequence from which on the chunked form is the faster one


@DSRecurrentRegistry.register_module
class DSStateSpace(DSRecurrentMixerBase):

    @staticmethod
    def name() -> str:
        return "state_space"

    @staticmethod
    def config_class() -> Type[DSStateSpaceConfig]:
        return DSStateSpaceConfig

    @staticmethod
    def supports_config(config) -> bool:
        return (isinstance(config, DSStateSpaceConfig) and config.input_dtype == config.output_dtype and
                DtypeEnum(config.input_dtype) in (DtypeEnum.bf16, DtypeEnum.fp32) and config.state_size <= (1024 if config.value_size % 4 == 0 else 512))

    def __init__(self, config: DSStateSpaceConfig, implementation_config: Dict[str, Any] = None) -> None:
        super().__init__(config, implementation_config)
        self._dtype = DtypeEnum(config.input_dtype).value

    @property
    def inner(self) -> int:
        return self._config.n_heads * self._config.value_size

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self._config.n_groups * self._config.state_size

    @property
    def in_width(self) -> int:
        """Columns of the input projection: z | x | B | C | step sizes."""
        return self.inner + self.conv_channels + self._config.n_heads

    def state_specs(self, prefix: str) -> List[StateBufferSpec]:
        c = self._config
        specs = [StateBufferSpec(prefix + ".S", (c.n_heads, c.state_size, c.value_size), torch.float32)]
        if c.conv_taps > 1:
            specs.append(StateBufferSpec(prefix + ".conv", (c.conv_taps - 1, self.conv_channels), self._dtype))
        return specs

    def transform_fp32_param(self, param: torch.Tensor) -> InferenceParameter:
        """Convolution bias, step-size biases, skip weights and norm weight stay fp32."""
        return InferenceParameter.initialize(param.to(torch.float32).contiguous())

    def transform_conv_param(self, param: torch.Tensor) -> InferenceParameter:
        """[channels, taps] -> fp32 [taps, channels]: the lanes of a warp read one stretch."""
        return InferenceParameter.initialize(param.to(torch.float32).t().contiguous())

    def transform_rate_param(self, param: torch.Tensor) -> InferenceParameter:
        """Stored as the logarithm of the decay rate; the kernels read the rate (formed in double, rounded once)."""
        return InferenceParameter.initialize(param.to(torch.float64).exp().to(torch.float32).contiguous())

    def forward(self, proj: torch.Tensor, col0: int, conv_w: torch.Tensor, conv_b: torch.Tensor, dt_bias: torch.Tensor, rate: torch.Tensor,
                skip: torch.Tensor, norm_w: torch.Tensor, batch, state_manager, prefix: str, out: torch.Tensor) -> torch.Tensor:
        """proj [T, N]: the fused projection with (z | x | B | C | step sizes) from column col0.  out: [T, inner] view."""
        c = self._config
        H, P, N, G, C = c.n_heads, c.value_size, c.state_size, c.n_groups, self.conv_channels
        desc, n_seqs = batch.seq_desc(), batch.current_sequences
        conv_state = state_manager.get_state(prefix + ".conv") if c.conv_taps > 1 else None
        x0 = col0 + self.inner
        xbc, dt, la = K.ssd_prepare(proj, x0, x0 + C, conv_w, conv_b, conv_state, desc, batch.tok_seq(), dt_bias, rate, C, H, c.conv_taps)
        if conv_state is not None:
            K.conv_state_update(proj, x0, C, conv_state, 0, desc, n_seqs, c.conv_taps)
        state = state_manager.get_state(prefix + ".S")
        y = torch.empty(proj.shape[0], self.inner, dtype=torch.float32, device=proj.device)
        longest, shortest = batch.portion_range
        chunked = longest >= CHUNK_MIN and K.ssd_chunk_ok(xbc, H, G, N, P)
        if chunked:
            K.ssd_chunk(xbc, dt, la, skip, desc, n_seqs, state, y, H, G, N, P, min_new=CHUNK_MIN)
        if not chunked or shortest < CHUNK_MIN:
            K.ssd_scan(xbc, dt, la, skip, desc, n_seqs, state, H, G, N, P, out=y, **({"max_new": CHUNK_MIN - 1} if chunked else {}))
        return K.gated_group_norm(y, proj[:, col0:col0 + self.inner], norm_w, out, c.norm_groups, c.eps)
