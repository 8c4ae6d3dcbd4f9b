"""Ritalorn: a decoder-only family built from
  * a residual of several parallel fp32 streams ("hyper-connections") that all start as the token embedding: a sublayer reads the RMS norm of a
    weighted sum of them, and its output, times one weight per channel (layer scale), joins every stream while the streams are mixed with one
    another; the model's output reads their sum,
  * 'attention' mixers: query / key / value projections with biases behind a short causal convolution, weightless RMS norms of queries and keys per
    head, no rotation -- every head's scores lose a fixed amount per position of distance -- and a mask by fixed chunks of the sequence; a sigmoid
    gate on the concatenated heads and an output projection with a bias; query / key and value heads may differ in size; a layer may read an
    earlier attention layer's cached keys and values instead of having its own,
  * 'latent_attention' mixers: keys and values are per-head up-projections of one cached, normed low-rank latent per token; beside it one rotated
    key part that all heads share (neighbouring entries are paired); a sliding window,
  * feed-forwards that are absent or dense (gated by the tanh form of gelu),
  * a final norm, the unembedding and a soft cap on the logits.
Every size may differ from layer to layer; all of them, the order of layers and the constants come from config.json.

The class reuses the ragged engine's plumbing from `RaggedTransformer` (containers and streamed loading, decode-step CUDA graphs, the state
manager's paged cache and block tables) and replaces the module set and the layer loop.  Attention layers of both kinds with keys and values of
their own get cache tensors, all sharing a sequence's block ids; layers that read another's are pointed at its tensors.  Convolution tails live in
the state manager's per-sequence slots, described by `state_config`.

Fused steps: all projections that read a mixer's input are ONE GEMM (queries | keys | values | output gate; queries | low-rank row), as are gate |
up; a sublayer's output bias, layer scale and join, the mixing of the streams, the next sublayer's weighted sum and its norm are ONE kernel (the last
join happens inside the final norm, for the wanted rows only); bias + convolution + head norms + cache append are one kernel, as are rotation +
latent norm + cache append; the attention kernel applies the output gate to its fp32 result; the value up-projection leaves the heads side by side."""
from dataclasses import dataclass, field
from typing import List, Optional

import torch

from ...inference_utils import DtypeEnum, NormTypeEnum
from ...modules import heuristics
from ...modules.configs import (DSConvSinkAttentionConfig, DSEmbeddingsConfig, DSLinearConfig, DSNormConfig, DSRotaryLatentAttentionConfig,
                                DSUnembedConfig)
from ...ragged.manager_configs import KVCacheConfig
from ... import kernels as K
from ..inference_model_base import DSInferenceModelBase
from ..ragged_transformer import RaggedTransformer

ROW_ALIGN = 8  # the parts of a fused projection start at multiples of this many columns (16 bytes of bf16: vector accesses everywhere)


@dataclass
class RitalornAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    chunk: int  # 0 = the whole history
    kv_from: Optional[int]  # the layer whose keys and values this one reads; None = its own


@dataclass
class RitalornLatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_dims: int
    rot_base: float
    window: int  # 0 = the whole history


@dataclass
class RitalornLayerSpec:
    kind: str  # "attention" | "latent_attention"
    attn: Optional[RitalornAttentionSpec] = None
    latent: Optional[RitalornLatentSpec] = None
    ff: int = 0  # hidden size of the feed-forward; 0 = the layer has none


@dataclass
class RitalornSpec:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    streams: int
    logit_softcap: float  # 0 = no cap
    layers: List[RitalornLayerSpec] = field(default_factory=list)
    family: str = "ritalorn"

    @property
    def num_layers(self):
        return len(self.layers)

    @classmethod
    def from_config(cls, c: dict) -> "RitalornSpec":
        layers = []
        for i, lc in enumerate(c["layers"]):
            m, f = lc["mixer"], lc.get("mlp")
            if f is not None and f.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind '{f.get('kind')}'")
            ff = int(f["ff"]) if f is not None else 0
            size = int((m.get("mask") or {}).get("size") or 0)
            if lc["type"] == "attention":
                src, heads = m.get("kv_from"), int(m["heads"])
                a = RitalornAttentionSpec(heads=heads, kv_heads=int(m.get("kv_heads", heads)), dim=int(m["dim"]), vdim=int(m.get("vdim", m["dim"])),
                                          conv=int(m.get("conv") or 1), scale=float(m["scale"]), chunk=size, kv_from=None if src is None else int(src))
                if a.kv_from is not None:
                    owner = layers[a.kv_from].attn if 0 <= a.kv_from < i else None
                    if owner is None or owner.kv_from is not None:
                        raise ValueError(f"layer {i}: layer {src} has no keys and values of its own in front of it")
                    if (owner.kv_heads, owner.dim, owner.vdim) != (a.kv_heads, a.dim, a.vdim):
                        raise ValueError(f"layer {i}: its key / value heads ({a.kv_heads} of {a.dim} / {a.vdim}) differ from layer {src}'s")
                layers.append(RitalornLayerSpec("attention", attn=a, ff=ff))
            elif lc["type"] == "latent_attention":
                rot = m.get("rot") or {}
                layers.append(RitalornLayerSpec("latent_attention", ff=ff, latent=RitalornLatentSpec(
                    heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                    scale=float(m["scale"]), rot_dims=int(rot.get("dims", m["rot_dim"])), rot_base=float(rot.get("base", 10000.0)), window=size)))
            else:
                raise ValueError(f"layer {i}: unknown mixer type '{lc['type']}'")
        return cls(vocab_size=int(c["vocab"]), hidden_size=int(c["width"]), norm_eps=float(c["norm"]["eps"]), streams=int(c.get("streams") or 1),
                   logit_softcap=float(c.get("logit_softcap") or 0.0), layers=layers)


class RitalornInferenceModel(RaggedTransformer, DSInferenceModelBase):
    describes_own_cache = True  # the engine builds its paged cache from `kv_cache_config` below

    def __init__(self, spec: RitalornSpec, tp_group=None, dtype=torch.bfloat16, device=None, engine_config=None, quantization_mode=""):
        from .container import RitalornAttentionContainer, RitalornLatentContainer, RitalornNonTransformerContainer, RitalornQueryContainer
        assert dtype in (torch.bfloat16, torch.float32), "Ritalorn runs with bf16 or fp32 activations"
        assert not quantization_mode, "Ritalorn has no quantised linears"
        self._init_plumbing(spec, tp_group, dtype, device, engine_config)
        assert self.tp == 1, "Ritalorn is served on one GPU per replica (its latent mixers are not sharded for tensor parallelism)"
        self.hq = self.hkv = 0
        self.vocab_padded = spec.vocab_size
        self._build_modules()

        def container_of(L):
            if L.kind == "latent_attention":
                return RitalornLatentContainer
            return RitalornAttentionContainer if L.attn.kv_from is None else RitalornQueryContainer

        self.layers = [container_of(L)(self, i) for i, L in enumerate(spec.layers)]
        self.non_transformer = RitalornNonTransformerContainer(self)
        # cache tensors of every layer with keys and values of its own: the latent row, one two-plane tensor or a (key, value) pair; layers
        # that read another layer's keys and values share its entry
        self._cache_index, n = {}, 0
        for i, L in enumerate(spec.layers):
            if L.attn is not None and L.attn.kv_from is not None:
                self._cache_index[i] = self._cache_index[L.attn.kv_from]
                continue
            k = len(self.attn_mods[i].cache_shapes())
            self._cache_index[i] = tuple(range(n, n + k))
            n += k
        self._layer_hook = None  # debugging aid: called as hook(layer index, fp32 sum of the streams) after every layer

    # ---- cache and state
    def kv_cache_config(self, block_size: int = 64):
        name = {torch.bfloat16: "bf16", torch.float32: "fp32"}[self.dtype]
        shapes = [s for m in self.attn_mods for s in m.cache_shapes()]
        return KVCacheConfig(block_size=block_size, cache_shape=(len(shapes), max(s[1] for s in shapes), max(s[2] for s in shapes)),
                             cache_dtype=name, layer_shapes=shapes)

    def state_config(self):
        """What a sequence carries between steps besides its cache blocks: `l<i>.mix.conv`, the last projected rows in front of an attention
        layer's convolution."""
        return [s for i, L in enumerate(self.spec.layers) if L.kind == "attention" for s in self.attn_mods[i].state_specs(f"l{i}.mix")]

    # ---- building blocks
    def _build_modules(self):
        s, ec, dt = self.spec, self.engine_config, DtypeEnum(self.dtype)
        sm = getattr(ec, "state_manager", None)
        max_tokens = getattr(sm, "max_ragged_batch_size", 768)
        max_seqs = getattr(sm, "max_ragged_sequence_count", 512)
        D = s.hidden_size
        common = dict(max_tokens=max_tokens, input_dtype=dt, output_dtype=dt)
        self.embed_mod = heuristics.instantiate_embed(DSEmbeddingsConfig(max_tokens=max_tokens, residual_dtype=dt, embedding_dim=D, fp32_stream=True), ec)
        self.norm_mod = heuristics.instantiate_pre_norm(DSNormConfig(type=NormTypeEnum.RMSNorm, channels=D, residual_dtype=DtypeEnum.fp32, eps=s.norm_eps,
                                                                      streams=s.streams, **common), ec)
        self.lin_mod = heuristics.instantiate_linear(DSLinearConfig(in_channels=D, out_channels=D, **common), None)
        self.attn_mods = []
        for L in s.layers:
            if L.kind == "latent_attention":
                a = L.latent
                cfg = DSRotaryLatentAttentionConfig(n_heads=a.heads, qk_dim=a.dim, rot_dim=a.rot_dim, v_dim=a.vdim, kv_rank=a.kv_rank, scale=a.scale,
                                                    rotate_dim=a.rot_dims, interleaved=True, theta_base=a.rot_base, window=a.window, eps=s.norm_eps,
                                                    max_sequences=max_seqs, **common)
            else:
                a = L.attn
                cfg = DSConvSinkAttentionConfig(n_heads_q=a.heads, n_heads_kv=a.kv_heads, head_size=a.dim, value_size=a.vdim, conv_taps=a.conv,
                                                scale=a.scale, part_size=a.chunk, qk_norm_weight=False, linear_bias=True, output_gate=True,
                                                reads_cache=a.kv_from is not None, eps=s.norm_eps, max_sequences=max_seqs, **common)
            self.attn_mods.append(heuristics.instantiate_attention(cfg, ec))
        self.unembed_mod = heuristics.instantiate_unembed(DSUnembedConfig(max_tokens=max_tokens, dtype=dt, norm_type=NormTypeEnum.RMSNorm, model_dim=D,
                                                                          max_sequences=max_seqs, vocab_size=s.vocab_size, eps=s.norm_eps,
                                                                          logit_softcap=s.logit_softcap, residual_fp32=True, streams=s.streams), ec)

    # ---- parameter transforms
    def transform_embedding_param(self, param):
        return self._dev(self.embed_mod.transform_param(param))

    def transform_norm_param(self, param):
        return self._dev(self.norm_mod.transform_param(param))

    def transform_dense_param(self, param):
        return self._dev(self.lin_mod.transform_param(param))

    def transform_gated_input_param(self, parts, gate):
        """[the projections in front of the convolution | output gate]; the gate starts at a multiple of ROW_ALIGN rows (zero rows in between)."""
        w = torch.cat(tuple(parts), dim=0)
        return self.transform_dense_param(torch.cat([torch.nn.functional.pad(w, (0, 0, 0, -w.shape[0] % ROW_ALIGN)), gate], dim=0))

    def transform_fp32_param(self, param):
        return self._dev(param.to(torch.float32).contiguous())

    def transform_key_up_param(self, param, layer_index):
        return self._dev(self.attn_mods[layer_index].transform_key_up_param(param))

    def transform_value_up_param(self, param, layer_index):
        return self._dev(self.attn_mods[layer_index].transform_value_up_param(param))

    def transform_unembed_param(self, param):
        return self._dev(param.to(self.dtype).contiguous())

    def load_canonical(self, sd):
        """State dict with the family's own tensor names."""
        import re
        rx = re.compile(r"^l(\d+)\.(.*)$")
        for name, tensor in sd.items():
            m = rx.match(name)
            ok = self.layers[int(m.group(1))].set_dependency(m.group(2), tensor) if m else self.non_transformer.set_dependency(name, tensor)
            if not ok:
                raise KeyError(f"unexpected parameter '{name}' for family ritalorn")
        self.check_populated()

    def check_populated(self):
        super().check_populated()
        for i, (L, c) in enumerate(zip(self.spec.layers, self.layers)):
            need = ["norm2_w", "scale2", "read2", "write2", "mix2", "ff_in_w", "ff_down_w"] if L.ff else []
            if L.kind == "attention" and L.attn.conv > 1:
                need.append("conv_w")
            if any(k not in c for k in need):
                raise RuntimeError(f"layer {i}: tensors are missing ({[k for k in need if k not in c]})")

    # ---- forward
    def _attention_mixer(self, li, L, W, h, batch, state_manager):
        mod = self.attn_mods[li]
        C = mod.conv_channels
        g0 = C + -C % ROW_ALIGN
        proj = self.lin_mod(h, W["in_w"])  # (queries | keys | values | output gate), or (queries | output gate); biases join in front of the convolution
        caches = [state_manager.get_cache(ci) for ci in self._cache_index[li]]
        n = mod.out_width
        o = torch.empty(h.shape[0], n + -n % ROW_ALIGN, dtype=h.dtype, device=h.device)[:, :n]
        mod(proj, 0, W["in_bias"], self._taps(W, C), None, None, None, None, None, caches[0], caches[1] if len(caches) > 1 else None, batch, state_manager,
            f"l{li}.mix", o, gate=proj[:, g0:g0 + n])
        return self.lin_mod(o, W["o_w"]), W["o_bias"]

    def _taps(self, W, channels):
        """A layer without taps of its own: one tap of weight one."""
        if "conv_w" in W:
            return W["conv_w"]
        ones = getattr(self, "_unit_taps", None)
        if ones is None or ones.shape[1] < channels:
            ones = self._unit_taps = torch.ones(1, channels, dtype=torch.float32, device=self.device)
        return ones[:, :channels]

    def _latent_mixer(self, li, L, W, h, batch, state_manager):
        nq = L.latent.heads * (L.latent.dim + L.latent.rot_dim)
        proj = self.lin_mod(h, W["in_w"])  # (queries | low-rank row)
        o = self.attn_mods[li](proj, (0, nq), state_manager.get_cache(self._cache_index[li][0]), batch, W["kv_norm"], W["key_up"], W["value_up"], None)
        return self.lin_mod(o, W["o_w"]), None

    def _feed_forward(self, L, W, h):
        gu = self.lin_mod(h, W["ff_in_w"])
        a = torch.empty(h.shape[0], L.ff + -L.ff % ROW_ALIGN, dtype=h.dtype, device=h.device)[:, :L.ff]
        return self.lin_mod(K.gelu_gate_cols(gu, 0, L.ff, L.ff, a), W["ff_down_w"])

    def forward(self, batch, state_manager):
        """batch: finalized RaggedBatchWrapper.  Returns fp32 logits [batch.n_logit_rows, vocab]."""
        s, nt = self.spec, self.non_transformer
        x = self.embed_mod(batch, nt.embed)  # fp32 [T, width]: the start of every stream
        pending = None  # the last sublayer's output that has not joined the streams yet: (output, bias, layer scale, mixing matrix, write weights)
        for li, L in enumerate(s.layers):
            W = self.layers[li]
            x, h = self.norm_mod(x, pending, W["norm1_w"], read=W["read1"])
            mixer = self._latent_mixer if L.kind == "latent_attention" else self._attention_mixer
            y, bias = mixer(li, L, W, h, batch, state_manager)
            pending = (y, bias, W["scale1"], W["mix1"], W["write1"])
            if L.ff:
                x, h = self.norm_mod(x, pending, W["norm2_w"], read=W["read2"])
                pending = (self._feed_forward(L, W, h), None, W["scale2"], W["mix2"], W["write2"])
            if self._layer_hook is not None:
                x, _ = self.norm_mod(x, pending, None)
                pending = None
                self._layer_hook(li, x.sum(1))
        return self.unembed_mod(x, nt.lm_head, batch, gamma=nt.final_norm_w, pending=pending)
