"""Containers of the Ritalorn family: tensor names of its checkpoints -> parameters of the inference model.

Every layer has, for its mixer, `l<i>.norm1`, `l<i>.ls1` and `l<i>.hc1.{in, out, mix}` and, with a feed-forward, the same with 2; the mixer itself
lies under `l<i>.mix.`:
  attention         {q, k, v, o} with biases `<name>.b`, {q, k, v}.conv, g  -- a layer that reads another's keys and values lacks those of k and v
  latent_attention  {q, dkv, dkv.norm, uk, uv, o}
The feed-forward is `l<i>.mlp.{gate, up, down}`.  Outside the layers: `embed`, `final.norm`, `head`.  Linear weights have shape [out, in]."""
from typing import Optional

import torch

from ..common_parameters import EmbeddingParameter, NormParameter, UnembedParameter
from ..layer_container_base import LayerContainer
from ..parameter_base import ParameterBase


class DenseParameter(ParameterBase):
    """A linear weight in the activation dtype."""
    params: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_dense_param(self.params)


class Fp32Parameter(ParameterBase):
    """Small tensors that enter norms, stream sums or layer scales: kept fp32."""
    params: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_fp32_param(self.params)


class AttentionInputParameter(ParameterBase):
    """(query | key | value) and output-gate projections of an attention mixer, stacked."""
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    g: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_gated_input_param((self.q, self.k, self.v), self.g)


class QueryInputParameter(ParameterBase):
    """Query and output-gate projections of an attention mixer without keys and values of its own, stacked."""
    q: torch.Tensor
    g: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_gated_input_param((self.q, ), self.g)


class StackedFp32Parameter(ParameterBase):
    """Per-channel fp32 tensors of the query, key and value projections (their biases), stacked."""
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_fp32_param(torch.cat([self.q, self.k, self.v], dim=0))


class ConvTapsParameter(ParameterBase):
    """Convolution taps [channels, taps] of the query, key and value projections -> one fp32 tensor [taps, all channels]: the layout the
    prepare kernel reads (the lanes of a warp read neighbouring channels of one tap)."""
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_fp32_param(torch.cat([self.q, self.k, self.v], dim=0).t())


class QueryTapsParameter(ParameterBase):
    """The same of a mixer that has queries only."""
    q: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_fp32_param(self.q.t())


class LatentInputParameter(ParameterBase):
    """(queries | low-rank row) projections of a latent-attention mixer, stacked."""
    q: torch.Tensor
    dkv: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_dense_param(torch.cat([self.q, self.dkv], dim=0))


class KeyUpParameter(ParameterBase):
    params: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_key_up_param(self.params, self.layer_index)


class ValueUpParameter(ParameterBase):
    params: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_value_up_param(self.params, self.layer_index)


class FeedForwardInputParameter(ParameterBase):
    """(gate | up) projections of a dense feed-forward, stacked."""
    gate: torch.Tensor
    up: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_dense_param(torch.cat([self.gate, self.up], dim=0))


class _RitalornLayerContainer(LayerContainer):
    norm1_w: NormParameter
    scale1: Fp32Parameter
    read1: Fp32Parameter
    write1: Fp32Parameter
    mix1: Fp32Parameter
    norm2_w: Optional[NormParameter]
    scale2: Optional[Fp32Parameter]
    read2: Optional[Fp32Parameter]
    write2: Optional[Fp32Parameter]
    mix2: Optional[Fp32Parameter]
    o_w: DenseParameter
    ff_in_w: Optional[FeedForwardInputParameter]
    ff_down_w: Optional[DenseParameter]

    PARAM_MAPPING = {
        "norm1": "norm1_w.params",
        "ls1": "scale1.params",
        "hc1.in": "read1.params",
        "hc1.out": "write1.params",
        "hc1.mix": "mix1.params",
        "norm2": "norm2_w.params",
        "ls2": "scale2.params",
        "hc2.in": "read2.params",
        "hc2.out": "write2.params",
        "hc2.mix": "mix2.params",
        "mix.o": "o_w.params",
        "mlp.gate": "ff_in_w.gate",
        "mlp.up": "ff_in_w.up",
        "mlp.down": "ff_down_w.params",
    }

    def __init__(self, model, layer_index: int) -> None:
        self.layer_index = layer_index
        super().__init__(model)
        for p in self._params.values():
            p.layer_index = layer_index


class RitalornAttentionContainer(_RitalornLayerContainer):
    in_w: AttentionInputParameter
    in_bias: StackedFp32Parameter
    conv_w: Optional[ConvTapsParameter]
    o_bias: Fp32Parameter

    PARAM_MAPPING = {
        "mix.q": "in_w.q",
        "mix.k": "in_w.k",
        "mix.v": "in_w.v",
        "mix.g": "in_w.g",
        "mix.q.b": "in_bias.q",
        "mix.k.b": "in_bias.k",
        "mix.v.b": "in_bias.v",
        "mix.q.conv": "conv_w.q",
        "mix.k.conv": "conv_w.k",
        "mix.v.conv": "conv_w.v",
        "mix.o.b": "o_bias.params",
    }


class RitalornQueryContainer(_RitalornLayerContainer):
    """An attention mixer that reads another layer's keys and values: queries only."""
    in_w: QueryInputParameter
    in_bias: Fp32Parameter
    conv_w: Optional[QueryTapsParameter]
    o_bias: Fp32Parameter

    PARAM_MAPPING = {
        "mix.q": "in_w.q",
        "mix.g": "in_w.g",
        "mix.q.b": "in_bias.params",
        "mix.q.conv": "conv_w.q",
        "mix.o.b": "o_bias.params",
    }


class RitalornLatentContainer(_RitalornLayerContainer):
    in_w: LatentInputParameter
    kv_norm: Fp32Parameter
    key_up: KeyUpParameter
    value_up: ValueUpParameter

    PARAM_MAPPING = {
        "mix.q": "in_w.q",
        "mix.dkv": "in_w.dkv",
        "mix.dkv.norm": "kv_norm.params",
        "mix.uk": "key_up.params",
        "mix.uv": "value_up.params",
    }


class RitalornNonTransformerContainer(LayerContainer):
    embed: EmbeddingParameter
    final_norm_w: NormParameter
    lm_head: UnembedParameter

    PARAM_MAPPING = {"embed": "embed.params", "final.norm": "final_norm_w.params", "head": "lm_head.params"}
