"""Gepolix: a decoder-only family built from
  * an fp32 residual stream that starts as the token embedding,
  * layers with ONE norm whose output every sublayer reads -- x += mixer(h) + ff(h), h = norm(x) -- where the norm has no statistic:
    norm(x) = tanh(alpha x) * w + b with one alpha per norm,
  * 'attention' mixers: query / key / value projections with biases, a rotate-half rotation of the first entries of a head, a sliding window,
    the plain softmax; query / key and value heads may differ in size; a layer may read an earlier attention layer's cached keys and values
    instead of having its own,
  * 'mamba2' mixers: state-space recurrences with one decay per head behind a short causal convolution, gated and normed in parts,
  * feed-forwards that are absent, dense (silu-gated), or a mixture of experts whose router has a bias and whose weights are a softmax over the
    chosen logits, with an optional shared expert that a number per token gates,
  * a final norm of the same kind and the unembedding.
Every size may differ from layer to layer; all of them, the order of layers and the constants come from config.json.

The class reuses the ragged engine's plumbing from `RaggedTransformer` (containers and streamed loading, decode-step CUDA graphs, the state
manager's paged cache and block tables) and replaces the module set and the layer loop.  Attention layers with keys and values of their own get
cache tensors (one two-plane tensor -- in bf16 of heads padded to a width the tensor-core kernels take -- or a key and a value tensor when the
head sizes differ), all sharing a sequence's block ids; layers that read another's are pointed at its tensors.  The recurrent layers' states
and convolution tails live in the state manager's per-sequence slots, described by `state_config`.

Fused steps: all projections that read a layer's normed input are ONE GEMM (mixer inputs | dense or shared-expert gate and up | the shared
expert's gate row); the mixer's output projection and the dense / shared-expert down projection are ONE GEMM over the concatenated
[mixer output | activated hidden] rows, which also forms their sum before any rounding (the shared expert's gate multiplies its hidden values);
the sublayers' outputs join the fp32 stream inside the next layer's norm kernel (the last layer's inside the final norm, for the wanted rows
only); biases + rotation + cache append are one kernel, as are convolution + bias + silu + step sizes."""
from dataclasses import dataclass, field
from typing import List, Optional

import torch

from ...inference_utils import ActivationType, DtypeEnum, NormTypeEnum
from ...modules import heuristics
from ...modules.configs import (DSEmbeddingsConfig, DSLinearConfig, DSMoEConfig, DSNormConfig, DSSinkAttentionConfig, DSStateSpaceConfig,
                                DSUnembedConfig)
from ...ragged.manager_configs import KVCacheConfig
from ... import kernels as K
from ..inference_model_base import DSInferenceModelBase
from ..ragged_transformer import RaggedTransformer

ROW_ALIGN = 8  # the fused projection's parts start at multiples of this many columns (16 bytes of bf16: vector accesses everywhere)


@dataclass
class GepolixAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int  # 0 = the whole history
    rot_dims: int
    rot_base: float
    kv_from: Optional[int]  # the layer whose keys and values this one reads; None = its own


@dataclass
class GepolixStateSpaceSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass
class GepolixFeedForwardSpec:
    kind: str  # "dense" | "moe"
    ff: int = 0  # dense: hidden size; moe: hidden size of an expert
    experts: int = 0
    top: int = 0
    shared_ff: int = 0  # 0 = no shared expert


@dataclass
class GepolixLayerSpec:
    kind: str  # "attention" | "mamba2"
    attn: Optional[GepolixAttentionSpec] = None
    ssm: Optional[GepolixStateSpaceSpec] = None
    mlp: Optional[GepolixFeedForwardSpec] = None


@dataclass
class GepolixSpec:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: List[GepolixLayerSpec] = field(default_factory=list)
    family: str = "gepolix"

    @property
    def num_layers(self):
        return len(self.layers)

    @classmethod
    def from_config(cls, c: dict) -> "GepolixSpec":
        layers = []
        for i, lc in enumerate(c["layers"]):
            m = lc["mixer"]
            mlp = None
            f = lc.get("mlp")
            if f is not None:
                if f.get("kind") == "dense":
                    mlp = GepolixFeedForwardSpec("dense", ff=int(f["ff"]))
                elif f.get("kind") == "moe":
                    sh = f.get("shared")
                    mlp = GepolixFeedForwardSpec("moe", ff=int(f["expert"]["ff"]), experts=int(f["router"]["experts"]), top=int(f["router"]["top"]),
                                                 shared_ff=int(sh["ff"]) if sh else 0)
                else:
                    raise ValueError(f"layer {i}: unknown feed-forward kind '{f.get('kind')}'")
            if lc["type"] == "attention":
                rot, src = m.get("rot") or {}, m.get("kv_from")
                attn = GepolixAttentionSpec(heads=int(m["heads"]), kv_heads=int(m.get("kv_heads", m["heads"])), dim=int(m["dim"]),
                                            vdim=int(m.get("vdim", m["dim"])), scale=float(m["scale"]), window=int((m.get("mask") or {}).get("size", 0)),
                                            rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)),
                                            kv_from=None if src is None else int(src))
                if attn.kv_from is not None:
                    owner = layers[attn.kv_from].attn if 0 <= attn.kv_from < i else None
                    if owner is None or owner.kv_from is not None:
                        raise ValueError(f"layer {i}: layer {src} has no keys and values of its own in front of it")
                    if (owner.kv_heads, owner.dim, owner.vdim) != (attn.kv_heads, attn.dim, attn.vdim):
                        raise ValueError(f"layer {i}: its key / value heads ({attn.kv_heads} of {attn.dim} / {attn.vdim}) differ from layer {src}'s")
                layers.append(GepolixLayerSpec("attention", attn=attn, mlp=mlp))
            elif lc["type"] == "mamba2":
                ssm = GepolixStateSpaceSpec(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m.get("groups", 1)),
                                            conv=int(m["conv"]), norm_groups=int(m.get("norm_groups", 1)))
                layers.append(GepolixLayerSpec("mamba2", ssm=ssm, mlp=mlp))
            else:
                raise ValueError(f"layer {i}: unknown mixer type '{lc['type']}'")
        return cls(vocab_size=int(c["vocab"]), hidden_size=int(c["width"]), norm_eps=float(c["norm"]["eps"]), layers=layers)


class GepolixInferenceModel(RaggedTransformer, DSInferenceModelBase):
    describes_own_cache = True  # the engine builds its paged cache from `kv_cache_config` below

    def __init__(self, spec: GepolixSpec, tp_group=None, dtype=torch.bfloat16, device=None, engine_config=None, quantization_mode=""):
        from .container import GepolixAttentionContainer, GepolixNonTransformerContainer, GepolixQueryContainer, GepolixStateSpaceContainer
        assert dtype in (torch.bfloat16, torch.float32), "Gepolix runs with bf16 or fp32 activations"
        assert not quantization_mode, "Gepolix has no quantised linears"
        self._loading_layer = 0
        self._init_plumbing(spec, tp_group, dtype, device, engine_config)
        assert self.tp == 1, "Gepolix is served on one GPU per replica (its recurrent mixers are not sharded for tensor parallelism)"
        self.hq = self.hkv = 0
        self.vocab_padded = spec.vocab_size
        self._build_modules()

        def container_of(L):
            if L.kind == "mamba2":
                return GepolixStateSpaceContainer
            return GepolixAttentionContainer if L.attn.kv_from is None else GepolixQueryContainer

        self.layers = [container_of(L)(self, i) for i, L in enumerate(spec.layers)]
        self.non_transformer = GepolixNonTransformerContainer(self)
        # cache tensors of every attention layer that has keys and values: one two-plane tensor or a (key, value) pair; layers that read
        # another layer's keys and values share its entry
        self._cache_index, n = {}, 0
        for i, L in enumerate(spec.layers):
            if L.kind != "attention":
                continue
            if L.attn.kv_from is not None:
                self._cache_index[i] = self._cache_index[L.attn.kv_from]
                continue
            k = len(self.attn_mods[i].cache_shapes())
            self._cache_index[i] = tuple(range(n, n + k))
            n += k
        self._fused = [None] * len(spec.layers)  # per layer, after loading: (input weight, first column of the feed-forward part, output weight)
        self._layer_hook = None  # debugging aid: called as hook(layer index, fp32 residual) after every layer

    # ---- facts the parameter classes ask for
    @property
    def n_experts(self):
        mlp = self.spec.layers[self._loading_layer].mlp
        return mlp.experts if mlp is not None else 0

    # ---- cache and state
    def kv_cache_config(self, block_size: int = 64):
        name = {torch.bfloat16: "bf16", torch.float32: "fp32"}[self.dtype]
        shapes = [s for m in self.attn_mods if m is not None for s in m.cache_shapes()]
        if not shapes:
            shapes = [(1, 1, 1)]  # a model without attention layers caches nothing per token; the block bookkeeping stays uniform
        return KVCacheConfig(block_size=block_size, cache_shape=(len(shapes), max(s[1] for s in shapes), max(s[2] for s in shapes)),
                             cache_dtype=name, layer_shapes=shapes)

    def state_config(self):
        """What a sequence carries between steps besides its cache blocks: `l<i>.mix.S` (the recurrent layers' states) and `l<i>.mix.conv` (the
        last projected rows in front of their convolutions)."""
        return [s for i, m in enumerate(self.ssm_mods) if m is not None for s in m.state_specs(f"l{i}.mix")]

    # ---- building blocks
    def _build_modules(self):
        s, ec, dt = self.spec, self.engine_config, DtypeEnum(self.dtype)
        sm = getattr(ec, "state_manager", None)
        max_tokens = getattr(sm, "max_ragged_batch_size", 768)
        max_seqs = getattr(sm, "max_ragged_sequence_count", 512)
        D = s.hidden_size
        common = dict(max_tokens=max_tokens, input_dtype=dt, output_dtype=dt)
        self.embed_mod = heuristics.instantiate_embed(DSEmbeddingsConfig(max_tokens=max_tokens, residual_dtype=dt, embedding_dim=D, fp32_stream=True), ec)
        self.norm_mod = heuristics.instantiate_pre_norm(DSNormConfig(type=NormTypeEnum.DynamicTanh, channels=D, residual_dtype=DtypeEnum.fp32, eps=s.norm_eps,
                                                                      shared_input=True, **common), ec)
        self.lin_mod = heuristics.instantiate_linear(DSLinearConfig(in_channels=D, out_channels=D, **common), None)
        self.attn_mods, self.ssm_mods, self.moe_mods = [], [], []
        for L in s.layers:
            attn = ssm = None
            if L.kind == "attention":
                a = L.attn
                attn = heuristics.instantiate_attention(DSSinkAttentionConfig(
                    n_heads_q=a.heads, n_heads_kv=a.kv_heads, head_size=a.dim, value_size=a.vdim, scale=a.scale, sink=0.0, qk_norm=False, v_norm=False,
                    rotate_dim=a.rot_dims, theta_base=a.rot_base, window=a.window, reads_cache=a.kv_from is not None, eps=s.norm_eps,
                    max_sequences=max_seqs, **common), ec)
            else:
                g = L.ssm
                ssm = heuristics.instantiate_recurrent(DSStateSpaceConfig(n_heads=g.heads, value_size=g.vdim, state_size=g.state, n_groups=g.groups,
                                                                          conv_taps=g.conv, norm_groups=g.norm_groups, eps=s.norm_eps,
                                                                          max_sequences=max_seqs, **common), ec)
            self.attn_mods.append(attn)
            self.ssm_mods.append(ssm)
            f = L.mlp
            self.moe_mods.append(None if f is None or f.kind != "moe" else heuristics.instantiate_moe(
                DSMoEConfig(model_dim=D, intermediate_features=f.ff, n_experts=f.experts, top_k=f.top, activation=ActivationType.SiGLU,
                            normalize_scores=True, router_bias=True, fp32_combine=True, **common), ec))
        self.unembed_mod = heuristics.instantiate_unembed(DSUnembedConfig(max_tokens=max_tokens, dtype=dt, norm_type=NormTypeEnum.DynamicTanh, model_dim=D,
                                                                          max_sequences=max_seqs, vocab_size=s.vocab_size, eps=s.norm_eps,
                                                                          residual_fp32=True), ec)

    # ---- parameter transforms
    def transform_embedding_param(self, param):
        return self._dev(self.embed_mod.transform_param(param))

    def transform_norm_param(self, param):
        return self._dev(self.norm_mod.transform_param(param))

    def transform_dense_param(self, param):
        return self._dev(self.lin_mod.transform_param(param))

    def transform_fp32_param(self, param):
        return self._dev(param.to(torch.float32).reshape(-1).contiguous())

    def transform_conv_param(self, param, layer_index):
        return self._dev(self.ssm_mods[layer_index].transform_conv_param(param))

    def transform_rate_param(self, param, layer_index):
        return self._dev(self.ssm_mods[layer_index].transform_rate_param(param))

    def transform_unembed_param(self, param):
        return self._dev(param.to(self.dtype).contiguous())

    def _any_moe(self):
        mods = [m for m in self.moe_mods if m is not None]
        assert mods, "an expert tensor arrived for a model without mixture-of-experts layers"
        return mods[0]

    def transform_moe_gate_param(self, param):
        return self._dev(self._any_moe().transform_gate_param(param))

    def transform_moe_mlp_1_param(self, param, gated=True):
        return self._dev(self._any_moe().transform_moe_mlp_1_param(param))

    def transform_moe_mlp_2_param(self, param):
        return self._dev(self._any_moe().transform_moe_mlp_2_param(param))

    def load_canonical(self, sd):
        """State dict with the family's own tensor names."""
        import re
        rx = re.compile(r"^l(\d+)\.(.*)$")
        for name, tensor in sd.items():
            m = rx.match(name)
            ok = self.layers[int(m.group(1))].set_dependency(m.group(2), tensor) if m else self.non_transformer.set_dependency(name, tensor)
            if not ok:
                raise KeyError(f"unexpected parameter '{name}' for family gepolix")
        self.finish_loading()

    def check_populated(self):
        super().check_populated()
        for i, (L, c) in enumerate(zip(self.spec.layers, self.layers)):
            f = L.mlp
            need = ["bias_q"] + (["bias_k", "bias_v"] if L.attn.kv_from is None else []) if L.kind == "attention" else []
            if f is not None and f.kind == "dense":
                need += ["ff_in_w", "ff_down_w"]
            elif f is not None:
                need += ["router_w", "router_b", "experts_gu", "experts_dn"] + (["shared_in_w", "shared_down_w"] if f.shared_ff else [])
            if any(k not in c for k in need):
                raise RuntimeError(f"layer {i}: tensors are missing ({[k for k in need if k not in c]})")

    def finish_loading(self):
        """All tensors have arrived: check every layer and form its fused weights -- the input weight (mixer projections | dense or shared gate
        and up, and the shared expert's gate row; zero rows fill up to ROW_ALIGN) and the output weight (mixer output | dense or shared down, side
        by side along the input axis)."""
        self.check_populated()
        for i, (L, c) in enumerate(zip(self.spec.layers, self.layers)):
            f = L.mlp
            side_in = side_out = None
            if f is not None and f.kind == "dense":
                side_in, side_out = c["ff_in_w"], c["ff_down_w"]
            elif f is not None and f.shared_ff:
                side_in, side_out = c["shared_in_w"], c["shared_down_w"]
            o_w = c["o_w"]
            if L.kind == "attention":  # zero weights meet the padding the attention kernels leave between heads
                o_w = self.attn_mods[i].layout_output_weight(o_w)
            parts = [self._fill_rows(c["mix_in_w"])] + ([self._fill_rows(side_in)] if side_in is not None else [])
            w_in = torch.cat(parts, dim=0).contiguous()
            w_out = o_w if side_out is None else torch.cat([o_w, side_out], dim=1)
            self._fused[i] = (w_in, parts[0].shape[0], w_out.contiguous())

    @staticmethod
    def _fill_rows(w):
        n = -w.shape[0] % ROW_ALIGN
        return torch.nn.functional.pad(w, (0, 0, 0, n)) if n else w

    # ---- forward
    @staticmethod
    def _side_hidden(L):
        """Hidden size of the feed-forward part that shares the layer's two fused GEMMs (dense, or the shared expert); 0 = none."""
        f = L.mlp
        if f is None:
            return 0
        return f.ff if f.kind == "dense" else f.shared_ff

    def forward(self, batch, state_manager):
        """batch: finalized RaggedBatchWrapper.  Returns fp32 logits [batch.n_logit_rows, vocab]."""
        s, nt = self.spec, self.non_transformer
        x = self.embed_mod(batch, nt.embed)  # fp32 residual stream [T, width]
        pending = None  # outputs of the previous layer's sublayers that have not joined the stream yet: ((activation dtype, ...), fp32 or None)
        for li, L in enumerate(s.layers):
            W = self.layers[li]
            w_in, ff0, w_out = self._fused[li]
            moe = self.moe_mods[li]
            branches, fp32_branch = pending if pending is not None else (None, None)
            h32 = None
            if moe is not None:
                _, h, h32 = self.norm_mod(x, branches, W["norm1_w"], W["norm1_b"], W["norm1_alpha"], fp32_branch=fp32_branch, fp32_copy=True)
            else:
                _, h = self.norm_mod(x, branches, W["norm1_w"], W["norm1_b"], W["norm1_alpha"], fp32_branch=fp32_branch)
            proj = self.lin_mod(h, w_in)
            side = self._side_hidden(L)
            n_mix_out = self.attn_mods[li].out_width if L.kind == "attention" else self.ssm_mods[li].inner
            # [mixer output | activated hidden]; rows start 16 bytes apart at least (what the tensor-core attention's stores want) whatever the sizes
            mixed = torch.empty(h.shape[0], -(-(n_mix_out + side) // 8) * 8, dtype=h.dtype, device=h.device)[:, :n_mix_out + side]
            if L.kind == "attention":
                a = L.attn
                caches = [state_manager.get_cache(ci) for ci in self._cache_index[li]]
                k0 = a.heads * a.dim
                own = a.kv_from is None
                self.attn_mods[li](proj, (0, k0, k0 + a.kv_heads * a.dim), caches[0], caches[1] if len(caches) > 1 else None, batch, None, None,
                                   mixed[:, :n_mix_out], biases=(W["bias_q"], W["bias_k"] if own else None, W["bias_v"] if own else None))
            else:
                self.ssm_mods[li](proj, 0, W["conv_w"], W["conv_b"], W["dt_bias"], W["rate"], W["skip"], W["mix_norm"], batch, state_manager,
                                  f"l{li}.mix", mixed[:, :n_mix_out])
            if side:  # silu(gate) * up; the shared expert's hidden values also times its gate (one number per token)
                K.clamped_swish_gate_cols(proj, ff0, ff0 + side, side, mixed[:, n_mix_out:], 1.0, float("inf"), 0.0,
                                          row_gate_col=ff0 + 2 * side if L.mlp.kind == "moe" else None)
            y = self.lin_mod(mixed, w_out)  # mixer output projection + dense / shared down projection, summed inside the GEMM
            y32 = None
            if moe is not None:
                y32 = moe(h, W["router_w"], W["experts_gu"], W["experts_dn"], router_bias=W["router_b"], router_input=h32)
            pending = ((y, ), y32)
            if self._layer_hook is not None:
                self.norm_mod(x, pending[0], None, fp32_branch=pending[1])
                pending = None
                self._layer_hook(li, x)
        return self.unembed_mod(x, nt.lm_head, batch, gamma=nt.final_norm_w, beta=nt.final_norm_b, alpha=nt.final_norm_alpha, pending=pending)
