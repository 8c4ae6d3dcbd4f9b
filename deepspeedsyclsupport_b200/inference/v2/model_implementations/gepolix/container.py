"""Containers of the Gepolix family: tensor names of its checkpoints -> parameters of the inference model.

Every layer has `l<i>.norm1` (with `.alpha` and `.b`) and a mixer under `l<i>.mix.`:
  attention   {q, k, v} with biases `<name>.b`, o   -- a layer that reads another layer's keys and values has only q, q.b and o
  mamba2      in, conv, conv.b, dt_bias, A_log, D, norm, o
A dense feed-forward is `l<i>.mlp.{gate, up, down}`; a mixture of experts `l<i>.mlp.{router, router.b, e<j>.gate, e<j>.up, e<j>.down}` and, with a
shared expert, `l<i>.mlp.shared.{gate, up, down, sg}`.  Outside the layers: `embed`, `final.norm` (with `.alpha` and `.b`), `head`.  Linear
weights have shape [out, in]."""
from typing import Optional

import torch

from ..common_parameters import (EmbeddingParameter, MoEGatingWeightParameter, NormParameter, UnembedParameter, UnfusedMoEGatedMLPParameter,
                                 UnfusedMoEMLP2Parameter)
from ..layer_container_base import LayerContainer
from ..parameter_base import ParameterBase


class DenseParameter(ParameterBase):
    """A linear weight in the activation dtype."""
    params: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_dense_param(self.params)


class Fp32Parameter(ParameterBase):
    """Small tensors that enter norms, routers or a recurrence: kept fp32 (a scalar as one entry)."""
    params: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_fp32_param(self.params)


class ConvParameter(ParameterBase):
    """Taps of a short convolution, re-laid-out for the kernel."""
    params: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_conv_param(self.params, self.layer_index)


class DecayRateParameter(ParameterBase):
    """Decay rates, stored as their logarithms."""
    params: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_rate_param(self.params, self.layer_index)


class AttentionInputParameter(ParameterBase):
    """(query | key | value) projections of an attention mixer, stacked."""
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_dense_param(torch.cat([self.q, self.k, self.v], dim=0))


class GatedPairParameter(ParameterBase):
    """(gate | up) projections of a gated feed-forward, stacked."""
    gate: torch.Tensor
    up: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_dense_param(torch.cat([self.gate, self.up], dim=0))


class GatedPairWithRowGateParameter(ParameterBase):
    """(gate | up | one row whose output gates the whole feed-forward per token), stacked."""
    gate: torch.Tensor
    up: torch.Tensor
    sg: torch.Tensor

    def finalize(self) -> torch.Tensor:
        return self.inference_model.transform_dense_param(torch.cat([self.gate, self.up, self.sg], dim=0))


class _GepolixLayerContainer(LayerContainer):
    norm1_w: NormParameter
    norm1_alpha: Fp32Parameter
    norm1_b: Fp32Parameter
    o_w: DenseParameter
    ff_in_w: Optional[GatedPairParameter]
    ff_down_w: Optional[DenseParameter]
    router_w: Optional[MoEGatingWeightParameter]
    router_b: Optional[Fp32Parameter]
    experts_gu: Optional[UnfusedMoEGatedMLPParameter]
    experts_dn: Optional[UnfusedMoEMLP2Parameter]
    shared_in_w: Optional[GatedPairWithRowGateParameter]
    shared_down_w: Optional[DenseParameter]

    PARAM_MAPPING = {
        "norm1": "norm1_w.params",
        "norm1.alpha": "norm1_alpha.params",
        "norm1.b": "norm1_b.params",
        "mix.o": "o_w.params",
        "mlp.gate": "ff_in_w.gate",
        "mlp.up": "ff_in_w.up",
        "mlp.down": "ff_down_w.params",
        "mlp.router": "router_w.params",
        "mlp.router.b": "router_b.params",
        "mlp.e*.gate": "experts_gu.gating_experts",
        "mlp.e*.up": "experts_gu.up_experts",
        "mlp.e*.down": "experts_dn.experts",
        "mlp.shared.gate": "shared_in_w.gate",
        "mlp.shared.up": "shared_in_w.up",
        "mlp.shared.sg": "shared_in_w.sg",
        "mlp.shared.down": "shared_down_w.params",
    }

    def __init__(self, model, layer_index: int) -> None:
        self.layer_index = layer_index
        model._loading_layer = layer_index  # the expert lists are sized per layer
        super().__init__(model)
        for p in self._params.values():
            p.layer_index = layer_index


class GepolixAttentionContainer(_GepolixLayerContainer):
    mix_in_w: AttentionInputParameter
    bias_q: Optional[Fp32Parameter]
    bias_k: Optional[Fp32Parameter]
    bias_v: Optional[Fp32Parameter]

    PARAM_MAPPING = {
        "mix.q": "mix_in_w.q",
        "mix.k": "mix_in_w.k",
        "mix.v": "mix_in_w.v",
        "mix.q.b": "bias_q.params",
        "mix.k.b": "bias_k.params",
        "mix.v.b": "bias_v.params",
    }


class GepolixQueryContainer(_GepolixLayerContainer):
    """An attention layer that reads another layer's keys and values."""
    mix_in_w: DenseParameter
    bias_q: Optional[Fp32Parameter]

    PARAM_MAPPING = {"mix.q": "mix_in_w.params", "mix.q.b": "bias_q.params"}


class GepolixStateSpaceContainer(_GepolixLayerContainer):
    mix_in_w: DenseParameter
    conv_w: ConvParameter
    conv_b: Fp32Parameter
    dt_bias: Fp32Parameter
    rate: DecayRateParameter
    skip: Fp32Parameter
    mix_norm: Fp32Parameter

    PARAM_MAPPING = {
        "mix.in": "mix_in_w.params",
        "mix.conv": "conv_w.params",
        "mix.conv.b": "conv_b.params",
        "mix.dt_bias": "dt_bias.params",
        "mix.A_log": "rate.params",
        "mix.D": "skip.params",
        "mix.norm": "mix_norm.params",
    }


class GepolixNonTransformerContainer(LayerContainer):
    embed: EmbeddingParameter
    final_norm_w: NormParameter
    final_norm_alpha: Fp32Parameter
    final_norm_b: Fp32Parameter
    lm_head: UnembedParameter

    PARAM_MAPPING = {
        "embed": "embed.params",
        "final.norm": "final_norm_w.params",
        "final.norm.alpha": "final_norm_alpha.params",
        "final.norm.b": "final_norm_b.params",
        "head": "lm_head.params",
    }
