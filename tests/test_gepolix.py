"""Gepolix on the ragged engine against the plain float64 oracle of tests/gepolix_oracle.py: every mechanism alone (the state-space kernels of
csrc/ragged/ssd_ops.cu and ssd_chunk.cu, the tanh norm / biased router / gated shared expert of csrc/ragged/latent_ops.cu, the windowed, biased
and cache-sharing attention of csrc/ragged/sink_attention_ops.cu and csrc/attn/paged_flash.cu), then whole models of several small random
configurations through the engine factory, the paged cache, the state slots, the scheduler and the decode-step graphs."""
import copy
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import gepolix_oracle as O  # noqa: E402

F64 = torch.float64


# ------------------------------------------------------------------------------------------------------------------ CPU: plumbing
def test_spec_reads_every_size_from_the_config():
    from deepspeedsyclsupport_b200.inference.v2.model_implementations.gepolix import GepolixSpec
    cfg = O.make_config([O.attention_layer(6, 3, 10, 14, 9, scale=0.3, rot_dims=4, base=500.0, mlp=O.moe(5, 3, 12, shared_ff=7)),
                         O.mamba2_layer(6, 9, 5, groups=3, conv=3, norm_groups=2, mlp=O.dense(22)), O.attention_layer(3, 3, 10, 14, 0, kv_from=0),
                         O.mamba2_layer(2, 4, 4)], vocab=77, width=40, eps=3e-5)
    s = GepolixSpec.from_config(cfg)
    assert (s.vocab_size, s.hidden_size, s.norm_eps, s.num_layers) == (77, 40, 3e-5, 4)
    a, f = s.layers[0].attn, s.layers[0].mlp
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.rot_dims, a.rot_base, a.kv_from) == (6, 3, 10, 14, 0.3, 9, 4, 500.0, None)
    assert (f.kind, f.experts, f.top, f.ff, f.shared_ff) == ("moe", 5, 3, 12, 7)
    g, d = s.layers[1].ssm, s.layers[1].mlp
    assert (g.heads, g.vdim, g.state, g.groups, g.conv, g.norm_groups) == (6, 9, 5, 3, 3, 2) and (d.kind, d.ff) == ("dense", 22)
    assert s.layers[2].attn.kv_from == 0 and s.layers[2].attn.window == 0 and s.layers[2].mlp is None
    for i, change in ((0, dict(type="other")), (1, dict(mlp={"kind": "other"})), (2, dict(mixer=dict(cfg["layers"][2]["mixer"], kv_from=1))),
                      (2, dict(mixer=dict(cfg["layers"][2]["mixer"], kv_from=2))), (2, dict(mixer=dict(cfg["layers"][2]["mixer"], dim=12)))):
        layers = copy.deepcopy(cfg["layers"])
        layers[i].update(change)
        with pytest.raises(ValueError):
            GepolixSpec.from_config(dict(cfg, layers=layers))


def test_family_is_registered_and_chosen_by_the_config():
    from deepspeedsyclsupport_b200.inference.v2.engine_factory import model_type_of
    from deepspeedsyclsupport_b200.inference.v2.model_implementations import GepolixPolicy, policy_for
    assert model_type_of({"architecture": "Gepolix"}) == "gepolix" and policy_for("gepolix") is GepolixPolicy


def _cpu_model(cfg, w, dt):
    from deepspeedsyclsupport_b200.inference.v2.checkpoint import InMemoryModelEngine
    from deepspeedsyclsupport_b200.inference.v2.engine_factory import build_model_from_checkpoint
    return build_model_from_checkpoint("gepolix", cfg, InMemoryModelEngine(w), None, device=torch.device("cpu"), dtype=dt)


def test_cache_state_and_fused_weights_of_a_model():
    cfg = O.make_config([O.mamba2_layer(3, 6, 5, conv=3, mlp=O.dense(20)), O.attention_layer(4, 2, 6, 10, 7, rot_dims=4, mlp=O.moe(3, 2, 10, shared_ff=12)),
                         O.attention_layer(2, 1, 12, 12, 5), O.attention_layer(8, 2, 6, 10, 3, rot_dims=4, kv_from=1), O.mamba2_layer(2, 4, 4, conv=1, mlp=O.moe(2, 1, 6))],
                        width=24)
    w = O.random_weights(cfg)
    m = _cpu_model(cfg, w, torch.float32)
    kc = m.kv_cache_config(block_size=32)
    # unequal key / value head sizes: a key tensor and a value tensor; equal: one two-plane tensor; a layer that reads another's has none of its own
    assert kc.layer_shapes == [(1, 2, 6), (1, 2, 10), (2, 1, 12)] and kc.cache_dtype == "fp32" and m._cache_index == {1: (0, 1), 2: (2, ), 3: (0, 1)}
    specs = {s.name: (tuple(s.shape), s.dtype) for s in m.state_config()}
    assert specs == {"l0.mix.S": ((3, 5, 6), torch.float32), "l0.mix.conv": ((2, 18 + 2 * 5), torch.float32), "l4.mix.S": ((2, 4, 4), torch.float32)}
    w_in, ff0, w_out = m._fused[0]
    n_mix = 2 * 18 + 2 * 5 + 3
    assert ff0 == 56 and w_in.shape == (56 + 40, 24) and w_out.shape == (24, 18 + 20)  # (z | x | B | C | steps | fill | gate | up), (o | down)
    assert torch.equal(w_in[:n_mix], w["l0.mix.in"].float()) and float(w_in[n_mix:56].abs().max()) == 0
    w_in, ff0, w_out = m._fused[1]
    assert ff0 == 56 and w_in.shape == (56 + 32, 24) and w_out.shape == (24, 4 * 10 + 12)  # the shared expert and its gate row ride along
    assert torch.equal(w_in[ff0 + 24:ff0 + 25], w["l1.mlp.shared.sg"].float()) and float(w_in[ff0 + 25:].abs().max()) == 0
    assert m._fused[3][0].shape == (48, 24) and m._fused[3][2].shape == (24, 80)  # queries only
    assert torch.allclose(m.layers[0]["rate"].double(), w["l0.mix.A_log"].double().exp(), rtol=1e-6) and m.layers[0]["conv_w"].shape == (3, 28)
    assert m.layers[1]["experts_gu"].shape == (3, 20, 24) and m.layers[1]["router_b"].dtype == torch.float32 and m.layers[0].get("experts_gu") is None
    for missing in ("l1.mlp.router.b", "l1.mlp.shared.sg", "l0.mlp.down", "l0.mix.dt_bias", "l1.mix.k.b", "l3.mix.q.b", "l2.norm1.alpha", "final.norm.b"):
        with pytest.raises(Exception):  # a missing tensor is reported, not ignored
            w2 = dict(w)
            w2.pop(missing)
            _cpu_model(cfg, w2, torch.float32)


def test_bf16_heads_get_a_tensor_core_width_and_slots():
    """bf16: heads padded to 64 / 128, three query heads per key / value head in four slots; zero columns of the output weight meet both."""
    cfg = O.make_config([O.attention_layer(6, 2, 6, 10, 8, mlp=O.dense(8)), O.attention_layer(5, 1, 96, 40, 8), O.attention_layer(2, 2, 130, 20, 8)], width=24)
    w = O.random_weights(cfg)
    m = _cpu_model(cfg, w, torch.bfloat16)
    assert m.kv_cache_config(block_size=16).layer_shapes == [(2, 2, 64), (2, 1, 128), (1, 2, 130), (1, 2, 20)]
    assert [(a.head_slots, a.out_head_width, a.out_width) for a in m.attn_mods] == [(4, 64, 512), (8, 128, 1024), (1, 20, 40)]
    w_out = m._fused[0][2]
    slots = w_out[:, :512].view(24, 2, 4, 64)
    assert torch.equal(slots[:, :, :3, :10].reshape(24, 60), w["l0.mix.o"]) and float(slots[:, :, 3].abs().max()) == 0 and float(slots[..., 10:].abs().max()) == 0
    assert torch.equal(w_out[:, 512:], w["l0.mlp.down"])


def test_module_choice():
    from deepspeedsyclsupport_b200.inference.v2.inference_utils import ActivationType, DtypeEnum, NormTypeEnum
    from deepspeedsyclsupport_b200.inference.v2.modules import heuristics
    from deepspeedsyclsupport_b200.inference.v2.modules.configs import DSMoEConfig, DSNormConfig, DSStateSpaceConfig
    io = dict(input_dtype=DtypeEnum.bf16, output_dtype=DtypeEnum.bf16)
    moe = DSMoEConfig(max_tokens=8, model_dim=8, intermediate_features=4, n_experts=3, top_k=2, activation=ActivationType.SiGLU, normalize_scores=True, router_bias=True, **io)
    assert heuristics.instantiate_moe(moe, None).name() == "grouped_topk_moe"
    norm = DSNormConfig(max_tokens=8, type=NormTypeEnum.DynamicTanh, channels=8, residual_dtype=DtypeEnum.fp32, shared_input=True, **io)
    assert heuristics.instantiate_pre_norm(norm, None).name() == "cuda_dynamic_tanh"
    kw = dict(max_tokens=8, n_heads=4, value_size=6, state_size=5, max_sequences=2, **io)
    assert heuristics.instantiate_recurrent(DSStateSpaceConfig(**kw), None).name() == "state_space"
    for bad in (dict(n_groups=3), dict(norm_groups=5), dict(conv_taps=0)):
        with pytest.raises(ValueError):
            DSStateSpaceConfig(**dict(kw, **bad))


def test_step_metadata_knows_its_longest_and_shortest_portion():
    from deepspeedsyclsupport_b200.inference.v2.ragged.ragged_wrapper import RaggedBatchWrapper
    b = RaggedBatchWrapper.__new__(RaggedBatchWrapper)
    b._seq_ntok = []
    assert b.portion_range == (0, 0)
    b._seq_ntok = [3, 40, 1]
    assert b.portion_range == (40, 1)


# ------------------------------------------------------------------------------------------------------------- GPU: mechanisms
gpu = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _K():
    from deepspeedsyclsupport_b200.inference.v2 import kernels
    return kernels


class _Batch:
    """Ragged metadata of a step, built by hand: seqs = [(slot, seen, new tokens, block ids)]."""

    def __init__(self, seqs, block, max_blocks=16):
        tok_seq, tok_pos, desc, at = [], [], [], 0
        bt = torch.zeros(len(seqs), max_blocks, dtype=torch.int32)
        for i, (slot, seen, n, blocks) in enumerate(seqs):
            tok_seq += [i] * n
            tok_pos += list(range(seen, seen + n))
            desc.append([at, n, seen, slot])
            bt[i, :len(blocks)] = torch.tensor(blocks, dtype=torch.int32)
            at += n
        self.current_sequences, self.current_tokens = len(seqs), at
        self.portion_range = (max(s[2] for s in seqs), min(s[2] for s in seqs))
        self._ts, self._tp = torch.tensor(tok_seq, dtype=torch.int32).cuda(), torch.tensor(tok_pos, dtype=torch.int32).cuda()
        self._bt, self._desc = bt.cuda(), torch.tensor(desc, dtype=torch.int32).cuda()

    def tok_seq(self):
        return self._ts

    def tok_pos(self):
        return self._tp

    def block_table(self):
        return self._bt

    def seq_desc(self):
        return self._desc


class _State:
    """Stand-in for the state manager: named per-slot buffers (filled with garbage: a sequence at position 0 must not read them)."""

    def __init__(self, specs, slots):
        self.buf = {s.name: torch.full((slots, ) + tuple(s.shape), 7.5, dtype=s.dtype, device="cuda") for s in specs}

    def get_state(self, name):
        return self.buf[name]


def _rel(got, want):
    return float((got.cpu().double() - want).norm() / want.norm())


def _cuts(total, sizes):
    out, at = [], 0
    for n in sizes:
        out.append((at, min(n, total - at)))
        at += n
        if at >= total:
            break
    if at < total:
        out.append((at, total - at))
    return out


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("dim", [6, 42, 320, 1024])
def test_tanh_norm_sums_the_branches_into_the_stream(dim, dt):
    """Widths on and off the 16-byte path; zero to three branches; a row gather that adds the branches to the gathered rows only and leaves the
    stream alone; the unrounded copy.  One row is 50x larger: a norm with a statistic would shrink it, this one saturates."""
    K = _K()
    g = torch.Generator().manual_seed(dim)
    x0 = torch.randn(9, dim, generator=g)
    x0[4] *= 50
    x0 = x0.cuda()
    ya, yb = ((torch.randn(9, dim, generator=g) * 0.5).to(dt).cuda() for _ in range(2))
    yc = torch.randn(9, dim, generator=g).cuda()
    w, b, alpha = (1 + 0.3 * torch.randn(dim, generator=g)).cuda(), torch.randn(dim, generator=g).cuda(), torch.tensor([0.37]).cuda()
    tol = dict(rtol=1e-5, atol=1e-5) if dt == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    for branches, extra in (((), None), ((ya, ), None), ((ya, yb), yc), ((), yc)):
        total = x0.cpu().double() + sum(t.cpu().double() for t in branches) + (extra.cpu().double() if extra is not None else 0)
        want = O.tanh_norm(total, w.cpu(), 0.37, b.cpu())
        x = x0.clone()
        out, out32 = K.stream_tanh_norm(x, branches, extra, alpha, w, b, out_dtype=dt, fp32_copy=True)
        assert torch.allclose(x.cpu().double(), total, rtol=1e-6, atol=1e-5)
        assert out.dtype == dt and out32.dtype == torch.float32 and torch.allclose(out.cpu().double(), want, **tol)
        assert torch.allclose(out32.cpu().double(), want, rtol=1e-5, atol=1e-5) and torch.equal(out32.to(dt), out)
        x = x0.clone()
        assert K.stream_tanh_norm(x, branches, extra) is None and torch.allclose(x.cpu().double(), total, rtol=1e-6, atol=1e-5)
        rows = torch.tensor([7, 4, 7, 3], dtype=torch.int32).cuda()
        x = x0.clone()
        got = K.stream_tanh_norm(x, branches, extra, alpha, w, b, out_dtype=dt, rows=rows)
        assert torch.equal(x, x0) and torch.allclose(got.cpu().double(), want[[7, 4, 7, 3]], **tol)


# ---- attention
def _attention_module(m, dt):
    from deepspeedsyclsupport_b200.inference.v2.inference_utils import DtypeEnum
    from deepspeedsyclsupport_b200.inference.v2.modules import heuristics
    from deepspeedsyclsupport_b200.inference.v2.modules.configs import DSSinkAttentionConfig
    rot = m.get("rot") or {}
    return heuristics.instantiate_attention(DSSinkAttentionConfig(
        max_tokens=1024, n_heads_q=m["heads"], n_heads_kv=m["kv_heads"], head_size=m["dim"], value_size=m["vdim"], scale=m["scale"], sink=0.0, qk_norm=False,
        v_norm=False, rotate_dim=rot.get("dims", 0), theta_base=rot.get("base", 10000.0), window=(m.get("mask") or {}).get("size", 0),
        reads_cache=m.get("kv_from") is not None, max_sequences=8, input_dtype=DtypeEnum(dt), output_dtype=DtypeEnum(dt)), None)


def _caches(mod, blocks, block, dt):
    return [torch.full((blocks, ) + ((p, ) if p != 1 else ()) + (block, h, d), 3.0, dtype=dt, device="cuda") for p, h, d in mod.cache_shapes()]


def _run_attention(mod, w, h, dt, caches, batch, own=True):
    """Output heads without their padding [n, H, dv] of one step whose rows are h (float64)."""
    c = mod._config
    names = ("q", "k", "v") if own else ("q", )
    H, G, d, dv = c.n_heads_q, c.n_heads_kv, c.head_size, c.value_size
    proj = (h @ torch.cat([w[n] for n in names]).double().T).to(dt).cuda()
    biases = tuple(w[n + ".b"].float().cuda() if n in names else None for n in ("q", "k", "v"))
    out = torch.empty(h.shape[0], mod.out_width, dtype=dt, device="cuda")
    mod(proj, (0, H * d, (H + G) * d), caches[0], caches[1] if len(caches) > 1 else None, batch, None, None, out, biases=biases)
    return out.view(-1, G, mod.head_slots, mod.out_head_width)[:, :, :H // G, :dv].reshape(-1, H, dv)


ATTENTION_CASES = [
    dict(heads=6, kv_heads=2, dim=10, vdim=6, mask=dict(size=19), rot=dict(dims=6, base=300.0)),  # grouped heads (three per key / value head), unequal sizes
    dict(heads=2, kv_heads=2, dim=8, vdim=8, mask=dict(size=1), rot=dict(dims=8, base=50.0)),  # a window of one: the token itself
    dict(heads=5, kv_heads=1, dim=14, vdim=20, mask=dict(size=500)),  # five heads on one, no rotation, a window that covers everything
    dict(heads=4, kv_heads=4, dim=64, vdim=32, mask=dict(size=33), rot=dict(dims=32, base=1e5)),
    dict(heads=4, kv_heads=2, dim=128, vdim=128, mask=dict(size=48), rot=dict(dims=128, base=1e6)),
    dict(heads=3, kv_heads=3, dim=32, vdim=96, rot=dict(dims=16, base=1000.0)),  # no window; values wider than keys
    dict(heads=2, kv_heads=1, dim=136, vdim=40, mask=dict(size=16), rot=dict(dims=136, base=1e4)),  # heads above 128: the CUDA-core kernel in bf16 too
]


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", range(len(ATTENTION_CASES)))
@pytest.mark.parametrize("sizes", [[90], [50] + [1] * 40, [2, 5, 1, 25, 2, 9, 46]])
def test_attention_mixer_and_a_layer_that_reads_its_cache(case, sizes, dt):
    """Whole, a prompt followed by single tokens, and portions cut inside pages (block 16), on shuffled pages that held something else.  A second
    layer with queries and a window of its own -- and another number of query heads -- reads the first one's keys and values."""
    m = dict(ATTENTION_CASES[case])
    m["scale"] = 1.7 * m["dim"] ** -0.5
    D, T, H, G, dv = 24, 90, m["heads"], m["kv_heads"], m["vdim"]
    reader = dict(m, heads=2 * G, mask=dict(size=27), kv_from=0)
    cfg = O.make_config([dict(type="attention", mixer=m, mlp=None), dict(type="attention", mixer=reader, mlp=None)], width=D)
    ws = O.random_weights(cfg, seed=case)
    w, wr = O.sub(ws, "l0.mix."), O.sub(ws, "l1.mix.")
    assert "k" not in wr and "v" not in wr
    w["o"], wr["o"] = torch.eye(H * dv).bfloat16(), torch.eye(2 * G * dv).bfloat16()
    g = torch.Generator().manual_seed(5)
    h, hr = (torch.randn(T, D, generator=g).bfloat16().double() for _ in range(2))
    want, kv = O.attention_mixer(h, w, m)
    want_r, _ = O.attention_mixer(hr, wr, reader, foreign=kv)
    mod, mod_r = _attention_module(m, dt), _attention_module(reader, dt)
    assert mod_r.cache_shapes() == []
    caches, pages = _caches(mod, 9, 16, dt), [5, 2, 7, 0, 3, 8]
    got, got_r = [], []
    for at, n in _cuts(T, sizes):
        b = _Batch([(0, at, n, pages)], 16)
        got.append(_run_attention(mod, w, h[at:at + n], dt, caches, b))
        got_r.append(_run_attention(mod_r, wr, hr[at:at + n], dt, caches, b, own=False))
    tol = 2e-5 if dt == torch.float32 else 2.5e-2
    assert _rel(torch.cat(got).reshape(T, -1), want) < tol
    assert _rel(torch.cat(got_r).reshape(T, -1), want_r) < tol


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("d,G,group", [(64, 2, 2), (128, 1, 3), (24, 2, 1)])
@pytest.mark.parametrize("window", [15, 16, 17, 64, 130])
def test_a_strong_key_is_seen_until_the_last_position_of_the_window(window, d, G, group, dt):
    """ONE key that every query loves among hundreds it does not: it takes the output of the window - 1 queries behind it and is gone for the next
    one -- keys at a page's first / last row and at the kernels' chunk borders, in prompt portions and for decoded tokens."""
    H, T, block = G * group, 400, 16
    m = dict(heads=H, kv_heads=G, dim=d, vdim=d, scale=1.0, mask=dict(size=window))
    mod = _attention_module(m, dt)
    g = torch.Generator().manual_seed(window + d)
    for far in (0, 100, 127, 128, 255):
        q = torch.randn(T, H, d, generator=g, dtype=F64) * 0.05
        k = torch.randn(T, G, d, generator=g, dtype=F64) * 0.05
        v = torch.randn(T, G, d, generator=g, dtype=F64)
        q[..., 0] += 3.0
        k[far, :, 0] += 4.0
        v[far] += 20.0
        q, k, v = (t.bfloat16().double() for t in (q, k, v))
        want = O.window_attention(q, k, v, 1.0, window)
        last, gone = far + window - 1, far + window
        assert float(want[last].min()) > 14 and float(want[gone].max()) < 8  # the oracle shows the edge
        proj = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=1)
        pages = torch.randperm(30, generator=g)[:T // block].tolist()
        caches = _caches(mod, 30, block, dt)
        eye = dict(q=torch.eye(proj.shape[1])[:H * d], k=torch.eye(proj.shape[1])[H * d:(H + G) * d], v=torch.eye(proj.shape[1])[(H + G) * d:])
        eye.update({n + ".b": torch.zeros(eye[n].shape[0]) for n in ("q", "k", "v")})
        cut = min(last - 3, T - 2) if last > 4 else 2
        rows, at = [], 0
        for n in [cut] + [1] * min(8, T - cut) + [T]:  # decoded tokens across the edge, portions before and behind
            n = min(n, T - at)
            if n <= 0:
                break
            rows.append(_run_attention(mod, eye, proj[at:at + n], dt, caches, _Batch([(0, at, n, pages)], block, max_blocks=32)))
            at += n
        got = torch.cat(rows).cpu().double()
        assert float((got - want).abs().max()) < (1e-3 if dt == torch.float32 else 0.25), far


@gpu
@pytest.mark.parametrize("dt", DTYPES)
def test_unequal_sequences_in_one_attention_step(dt):
    """A portion, a single token far behind its window's start and a two-token portion in one batch, each against the sequence alone; in bf16 on the
    tensor cores with three query heads per key / value head."""
    m = dict(heads=6, kv_heads=2, dim=40, vdim=24, scale=0.4, mask=dict(size=21), rot=dict(dims=20, base=77.0))
    cfg = O.make_config([dict(type="attention", mixer=m, mlp=None)], width=24)
    w = O.sub(O.random_weights(cfg, seed=3), "l0.mix.")
    w["o"] = torch.eye(6 * 24).bfloat16()
    mod = _attention_module(m, dt)
    caches = _caches(mod, 24, 16, dt)
    g = torch.Generator().manual_seed(1)
    hs = {u: torch.randn(n, 24, generator=g).bfloat16().double() for u, n in ((0, 80), (1, 101), (2, 35))}
    pages = {0: [3, 9, 1, 7, 12], 1: [0, 2, 4, 6, 8, 10, 11], 2: [13, 5, 14]}
    want = {u: O.attention_mixer(h, w, m)[0] for u, h in hs.items()}
    at, got = {u: 0 for u in hs}, {u: [] for u in hs}
    for step in ([(1, 100)], [(0, 33), (1, 1), (2, 2)], [(2, 33), (0, 47)]):
        b = _Batch([(0, at[u], n, pages[u]) for u, n in step], 16)
        out = _run_attention(mod, w, torch.cat([hs[u][at[u]:at[u] + n] for u, n in step]), dt, caches, b)
        r = 0
        for u, n in step:
            got[u].append(out[r:r + n])
            r += n
            at[u] += n
    for u in hs:
        assert _rel(torch.cat(got[u]).reshape(at[u], -1), want[u]) < (2e-5 if dt == torch.float32 else 2.5e-2), u


# ---- state-space mixer
def _ssm_module(m, dt, eps=1e-5):
    from deepspeedsyclsupport_b200.inference.v2.inference_utils import DtypeEnum
    from deepspeedsyclsupport_b200.inference.v2.modules import heuristics
    from deepspeedsyclsupport_b200.inference.v2.modules.configs import DSStateSpaceConfig
    return heuristics.instantiate_recurrent(DSStateSpaceConfig(max_tokens=2048, n_heads=m["heads"], value_size=m["vdim"], state_size=m["state"], n_groups=m["groups"],
                                                               conv_taps=m["conv"], norm_groups=m["norm_groups"], eps=eps, max_sequences=8,
                                                               input_dtype=DtypeEnum(dt), output_dtype=DtypeEnum(dt)), None)


def _ssm_params(mod, w):
    f = lambda n: w[n].float().cuda()
    return (mod.transform_conv_param(w["conv"]).cuda(), f("conv.b"), f("dt_bias"), mod.transform_rate_param(w["A_log"]).cuda(), f("D"), f("norm"))


def _run_ssm(mod, w, params, h, dt, batch, st, lead=0):
    proj = (h @ w["in"].double().T).to(dt)
    if lead:  # the mixer's columns start behind others and its rows are longer than it needs
        proj = torch.cat([torch.full((h.shape[0], lead), 9.0, dtype=dt), proj, torch.full((h.shape[0], 3), 9.0, dtype=dt)], dim=1)
    out = torch.empty(h.shape[0], mod.inner + 5, dtype=dt, device="cuda")[:, :mod.inner]
    return mod(proj.cuda(), lead, *params, batch, st, "m", out)


def _ssm_setup(m, D, seed, dt, slots=3):
    cfg = O.make_config([dict(type="mamba2", mixer=m, mlp=None)], width=D)
    w = O.sub(O.random_weights(cfg, seed=seed), "l0.mix.")
    w["o"] = torch.eye(m["heads"] * m["vdim"]).bfloat16()
    mod = _ssm_module(m, dt)
    return w, mod, _ssm_params(mod, w), _State(mod.state_specs("m"), slots)


SSM_CASES = [
    dict(heads=3, vdim=6, state=5, groups=1, conv=4, norm_groups=1),  # odd sizes
    dict(heads=4, vdim=7, state=9, groups=2, conv=3, norm_groups=4),  # one value at a time, two groups of heads, parts that are not the groups
    dict(heads=2, vdim=20, state=12, groups=2, conv=2, norm_groups=2),
    dict(heads=1, vdim=80, state=130, groups=1, conv=1, norm_groups=5),  # no convolution memory, several column tiles
    dict(heads=6, vdim=32, state=48, groups=3, conv=4, norm_groups=2),  # sizes the chunked form takes
    dict(heads=2, vdim=64, state=128, groups=1, conv=6, norm_groups=1),  # its largest, more taps than the unrolled kernels
    dict(heads=4, vdim=16, state=16, groups=4, conv=4, norm_groups=4),  # its smallest
]


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", range(len(SSM_CASES)))
@pytest.mark.parametrize("sizes", [[160], [40] + [1] * 40, [2, 3, 1, 2, 35, 1, 64, 2, 50], [129, 31]])
def test_state_space_mixer(case, sizes, dt):
    """Whole, a prompt followed by single tokens, portions down to two tokens that switch between the two forms of the recurrence; a slot that held
    garbage before."""
    m = SSM_CASES[case]
    T = min(160, sum(sizes))
    w, mod, params, st = _ssm_setup(m, 24, case, dt)
    h = torch.randn(T, 24, generator=torch.Generator().manual_seed(6)).bfloat16().double()
    want, _ = O.mamba2_mixer(h, w, m, 1e-5)
    got = torch.cat([_run_ssm(mod, w, params, h[at:at + n], dt, _Batch([(2, at, n, [0])], 4096), st, lead=(case % 2) * 8) for at, n in _cuts(T, sizes)])
    assert _rel(got, want) < (2e-5 if dt == torch.float32 else 2e-2)
    assert int(_K().wait_error_word(got.device)) == 0


@gpu
@pytest.mark.parametrize("dt", DTYPES)
def test_state_space_sequences_side_by_side_and_a_slot_taken_over(dt):
    """A step that mixes a long portion, a short one and a single token (both forms of the recurrence and the convolution's rows of three sequences
    side by side), each against the sequence alone; then a new sequence in a used slot."""
    m = dict(heads=4, vdim=32, state=48, groups=2, conv=4, norm_groups=1)
    w, mod, params, st = _ssm_setup(m, 40, 11, dt)
    g = torch.Generator().manual_seed(9)
    hs = {u: torch.randn(n, 40, generator=g).bfloat16().double() for u, n in ((0, 250), (1, 45), (2, 9), (3, 70))}
    slot = {0: 1, 1: 0, 2: 2, 3: 0}
    want = {u: O.mamba2_mixer(h, w, m, 1e-5)[0] for u, h in hs.items()}
    at, got = {u: 0 for u in hs}, {u: [] for u in hs}
    for step in ([(1, 5), (2, 1)], [(0, 140), (1, 2), (2, 3)], [(2, 1), (0, 33), (1, 38)], [(0, 1), (2, 4)], [(0, 76), (3, 2)], [(3, 68)]):
        out = _run_ssm(mod, w, params, torch.cat([hs[u][at[u]:at[u] + n] for u, n in step]), dt, _Batch([(slot[u], at[u], n, [0]) for u, n in step], 4096), st)
        r = 0
        for u, n in step:
            got[u].append(out[r:r + n])
            r += n
            at[u] += n
    for u in hs:
        assert at[u] == hs[u].shape[0] and _rel(torch.cat(got[u]), want[u]) < (2e-5 if dt == torch.float32 else 2e-2), u


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("taps,C,H", [(4, 48, 6), (3, 21, 2), (1, 16, 3), (7, 40, 5)])
def test_convolution_and_steps_of_many_rows(taps, C, H, dt):
    """More than 512 rows (several rows per thread): sequences of 1, 2, 300, 3 and 290 rows side by side, some new, some with kept rows, so that a
    thread's run of rows enters new sequences in its middle."""
    K = _K()
    g = torch.Generator().manual_seed(taps)
    seqs = [(1, 0), (2, 9), (300, 1), (3, 0), (290, 2), (1, 50)]  # (new rows, rows seen before)
    total = sum(n for n, _ in seqs)
    proj = torch.randn(total, 5 + C + H + 2, generator=g).to(dt)
    w, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    bias, rate = torch.randn(H, generator=g) * 3, torch.rand(H, generator=g) * 4
    kept = torch.randn(len(seqs), max(taps - 1, 1), C, generator=g).to(dt)
    want, at, desc, tok_seq = [], 0, [], []
    for i, (n, seen) in enumerate(seqs):
        tail = kept[i, :taps - 1].double().clone()
        if seen < taps - 1:
            tail[:taps - 1 - seen] = 0  # positions before the sequence's start: whatever the slot holds does not count
        want.append(O.causal_conv_silu(proj[at:at + n, 5:5 + C].double(), w, b, tail)[0])
        desc.append([at, n, seen, i])
        tok_seq += [i] * n
        at += n
    desc, tok_seq = torch.tensor(desc, dtype=torch.int32).cuda(), torch.tensor(tok_seq, dtype=torch.int32).cuda()
    state = kept.cuda() if taps > 1 else None
    xbc, dt_, la = K.ssd_prepare(proj.cuda(), 5, 5 + C, w.t().contiguous().cuda(), b.cuda(), state, desc, tok_seq, bias.cuda(), rate.cuda(), C, H, taps)
    assert _rel(xbc, torch.cat(want)) < (1e-6 if dt == torch.float32 else 5e-3)
    step = torch.nn.functional.softplus(proj[:, 5 + C:5 + C + H].double() + bias.double(), threshold=1e9)
    assert _rel(dt_, step) < 1e-6 and _rel(la, -rate.double() * step) < 1e-6


def _recurrence_inputs(T, H, G, N, P, dt_range, rate, seed, dt):
    g = torch.Generator().manual_seed(seed)
    xbc = torch.randn(T, H * P + 2 * G * N, generator=g).to(dt)
    step = dt_range[0] + (dt_range[1] - dt_range[0]) * torch.rand(T, H, generator=g)
    return xbc, step, torch.tensor(rate).float(), torch.randn(H, generator=g)


def _recurrence_want(xbc, step, rate, D, H, G, N, P):
    T = xbc.shape[0]
    x, B, C = xbc[:, :H * P].double().reshape(T, H, P), xbc[:, H * P:H * P + G * N].double().reshape(T, G, N), xbc[:, H * P + G * N:].double().reshape(T, G, N)
    y, S = O.ssd_recurrence(x, B, C, step.double(), rate.double().log(), D, torch.zeros(H, N, P, dtype=F64))
    return y.reshape(T, H * P), S


@gpu
@pytest.mark.parametrize("form", ["scan", "scan bf16", "chunks"])
@pytest.mark.parametrize("far", [0, 127, 128, 200])
def test_a_token_far_back_shows_in_the_read_out(far, form):
    """ONE token hundreds of positions back, written 60x as strongly as the others: a head that hardly forgets carries it to the end, a head that
    forgets at once has lost it a few tokens later, and so has one whose decay underflows.  Every form of the recurrence, against float64; the step
    by step read-out of the slow head must be exact over 500 tokens."""
    K = _K()
    H, G, N, P, T = 4, 2, 32, 48, 500
    dt = torch.float32 if form == "scan" else torch.bfloat16
    xbc, step, rate, D = _recurrence_inputs(T, H, G, N, P, (0.2, 1.0), [1e-4, 0.02, 30.0, 1000.0], far, dt)
    xbc[far, :H * P] *= 60
    xbc[-1, H * P + G * N:] = xbc[far, H * P:H * P + G * N]  # the last token asks for exactly what that one wrote
    want, S_want = _recurrence_want(xbc, step, rate, D, H, G, N, P)
    quiet = xbc.clone()
    quiet[far, :H * P] /= 60
    calm, _ = _recurrence_want(quiet, step, rate, D, H, G, N, P)
    change = (want - calm).view(T, H, P).norm(dim=-1) / calm.view(T, H, P).norm(dim=-1)
    assert float(change[-1, 0]) > 1 and float(change[far + 3, 2]) < 1e-2 and float(change[-1, 3]) < 1e-6  # the oracle shows it
    step, la = step.cuda(), (-rate * step).cuda()
    state = torch.full((2, H, N, P), 5.0, device="cuda")
    desc = torch.tensor([[0, T, 0, 1]], dtype=torch.int32).cuda()
    out = torch.empty(T, H * P, device="cuda")
    args = (xbc.cuda(), step, la, D.cuda(), desc, 1, state)
    if form == "chunks":
        assert K.ssd_chunk_ok(args[0], H, G, N, P)
        K.ssd_chunk(*args, out, H, G, N, P)
    else:
        K.ssd_scan(*args, H, G, N, P, out=out)
    tol = 3e-6 if form != "chunks" else 3e-5  # the chunked form splits its operands into two bf16 numbers (16 bits)
    size = want.view(T, H, P).norm(dim=-1)  # a read-out that happens to be small among large states is measured by its head's usual size
    err = (out.cpu().double() - want).view(T, H, P).norm(dim=-1) / torch.maximum(size, size.pow(2).mean(0).sqrt())
    assert float(err.max()) < tol * 10 and float(err.median()) < tol, (float(err.max()), float(err.median()))
    assert _rel(state[1], S_want) < tol and float((state[0] - 5).abs().max()) == 0
    assert int(K.wait_error_word(out.device)) == 0


@gpu
def test_the_two_forms_hand_the_state_over_and_share_a_step():
    """Chunked portions, single tokens and portions with the state in front of them, several sequences per launch: the forms agree to far below a
    bf16 rounding, whatever the order."""
    K = _K()
    H, G, N, P = 4, 1, 128, 64
    lens = [300, 1, 128, 17, 129, 33]
    total = sum(lens)
    xbc, step, rate, D = _recurrence_inputs(2 * total, H, G, N, P, (0.001, 0.3), [0.01, 0.3, 2.0, 8.0], 1, torch.bfloat16)
    xbc, step, D = xbc.cuda(), step.cuda(), D.cuda()
    la = -rate.cuda() * step
    slots = [4, 0, 5, 1, 3, 2]
    res = []
    for chunked in (False, True):
        state = torch.full((6, H, N, P), 2.0, device="cuda")
        outs = []
        for turn in range(2):
            lo, seen = turn * total, 0 if turn == 0 else 1
            rows, at = [], 0
            for n, s in zip(lens, slots):
                rows.append([at, n, seen * n, s])
                at += n
            desc = torch.tensor(rows, dtype=torch.int32).cuda()
            part = slice(lo, lo + total)
            args = (xbc[part].contiguous(), step[part].contiguous(), la[part].contiguous(), D, desc, len(lens), state)
            out = torch.full((total, H * P), float("nan"), device="cuda")
            if chunked:
                K.ssd_chunk(*args, out, H, G, N, P, min_new=32)
                K.ssd_scan(*args, H, G, N, P, out=out, max_new=31)
            else:
                K.ssd_scan(*args, H, G, N, P, out=out)
            outs.append(out)
        res.append((torch.cat(outs), state))
    assert bool(torch.isfinite(res[1][0]).all()) and _rel(res[1][0], res[0][0].cpu().double()) < 2e-5 and _rel(res[1][1], res[0][1].cpu().double()) < 2e-5
    assert int(K.wait_error_word(xbc.device)) == 0


@gpu
@pytest.mark.parametrize("dt", DTYPES)
def test_long_decoding_of_the_state_space_mixer(dt):
    """400 single tokens behind a short prompt; slow heads still show the first tokens at the end."""
    m = dict(heads=3, vdim=16, state=16, groups=3, conv=4, norm_groups=1)
    w, mod, params, st = _ssm_setup(m, 16, 2, dt)
    w["A_log"] = torch.tensor([-6.0, -3.0, 1.0]).bfloat16()
    params = _ssm_params(mod, w)
    h = torch.randn(410, 16, generator=torch.Generator().manual_seed(8)).bfloat16().double()
    want, _ = O.mamba2_mixer(h, w, m, 1e-5)
    other, _ = O.mamba2_mixer(torch.cat([h[10:20], h[10:]]), w, m, 1e-5)
    assert float((want[-1] - other[-1]).norm() / want[-1].norm()) > 1e-2  # the first ten tokens are still in the last read-out
    got = torch.cat([_run_ssm(mod, w, params, h[at:at + n], dt, _Batch([(0, at, n, [0])], 4096), st) for at, n in _cuts(410, [10] + [1] * 400)])
    assert _rel(got, want) < (2e-5 if dt == torch.float32 else 2e-2)


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("inner,groups", [(6, 3), (35, 5), (96, 4), (512, 1), (12288, 2)])
def test_gate_comes_before_the_grouped_norm(inner, groups, dt):
    K = _K()
    g = torch.Generator().manual_seed(inner)
    y = torch.randn(7, inner, generator=g)
    y[:, :inner // groups] *= 30  # one part much larger: a norm over the whole row would flatten the others
    z = (torch.randn(7, inner + 8, generator=g) * 2).to(dt).cuda()[:, :inner]
    w = 1 + 0.3 * torch.randn(inner, generator=g)
    want = O.grouped_rms(y.double() * torch.nn.functional.silu(z.cpu().double()), w, groups, 1e-5)
    wide = torch.zeros(7, inner + 4, dtype=dt, device="cuda")
    K.gated_group_norm(y.cuda(), z, w.cuda(), wide[:, :inner], groups, 1e-5)
    assert _rel(wide[:, :inner], want) < (1e-6 if dt == torch.float32 else 5e-3) and float(wide[:, inner:].abs().max()) == 0
    after = O.grouped_rms(y, w, groups, 1e-5) * torch.nn.functional.silu(z.cpu().double())
    assert float((after - want).norm() / want.norm()) > 0.05  # the other order would show


# ---- feed-forward
def _moe_module(f, D, dt):
    from deepspeedsyclsupport_b200.inference.v2.inference_utils import ActivationType, DtypeEnum
    from deepspeedsyclsupport_b200.inference.v2.modules import heuristics
    from deepspeedsyclsupport_b200.inference.v2.modules.configs import DSMoEConfig
    return heuristics.instantiate_moe(DSMoEConfig(max_tokens=512, model_dim=D, intermediate_features=f["expert"]["ff"], n_experts=f["router"]["experts"],
                                                  top_k=f["router"]["top"], activation=ActivationType.SiGLU, normalize_scores=True, router_bias=True,
                                                  fp32_combine=True, input_dtype=DtypeEnum(dt), output_dtype=DtypeEnum(dt)), None)


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("experts,top,ff,D", [(5, 3, 12, 24), (4, 1, 8, 40), (3, 3, 16, 64), (8, 2, 32, 128)])
def test_router_bias_counts_for_selection_and_weights(experts, top, ff, D, dt):
    """A bias that lifts the otherwise weakest expert into every selection AND into the weights; the softmax runs over the chosen logits alone."""
    f = O.moe(experts, top, ff)
    cfg = O.make_config([O.mamba2_layer(1, 4, 4, mlp=f)], width=D)
    w = O.sub(O.random_weights(cfg, seed=experts, router_gain=2.0), "l0.mlp.")
    w["router.b"] = torch.tensor([9.0] + [0.25 * e for e in range(1, experts)]).bfloat16()
    h = torch.randn(50, D, generator=torch.Generator().manual_seed(2)).to(dt)
    idx, wt = O.route(h, w, top)
    assert bool((idx == 0).any(-1).all()) and float((wt.sum(-1) - 1).abs().max()) < 1e-12
    plain, _ = O.route(h, dict(w, **{"router.b": torch.zeros(experts)}), top)
    assert not torch.equal(plain.sort(-1).values, idx.sort(-1).values) or top == experts
    mod = _moe_module(f, D, dt)
    gu = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)]).to(dt).cuda()
    dn = torch.stack([w[f"e{e}.down"] for e in range(experts)]).to(dt).cuda()
    got = mod(h.cuda(), w["router"].float().cuda(), gu, dn, router_bias=w["router.b"].float().cuda(), router_input=h.float().cuda())
    assert got.dtype == torch.float32 and _rel(got, O.moe_ff(h, w, f)) < (2e-5 if dt == torch.float32 else 1.5e-2)


@gpu
@pytest.mark.parametrize("dt", DTYPES)
def test_a_number_per_token_gates_the_shared_expert(dt):
    """Gate, up and the row gate as columns of one projection, odd and aligned; without the gate column nothing changes."""
    K = _K()
    g = torch.Generator().manual_seed(4)
    for c0, F, lead in ((7, 18, 5), (8, 20, 4)):
        proj = (torch.randn(13, c0 + 2 * F + 4, generator=g) * 2).to(dt).cuda()
        wide = torch.zeros(13, lead + F, dtype=dt, device="cuda")
        p = proj.cpu().double()
        want = torch.nn.functional.silu(p[:, c0:c0 + F]) * p[:, c0 + F:c0 + 2 * F]
        for col in (None, c0 + 2 * F):
            K.clamped_swish_gate_cols(proj, c0, c0 + F, F, wide[:, lead:], 1.0, float("inf"), 0.0, row_gate_col=col)
            ref = want if col is None else want * torch.sigmoid(p[:, col:col + 1])
            assert torch.allclose(wide[:, lead:].cpu().double(), ref, rtol=1e-5 if dt == torch.float32 else 1e-2, atol=1e-5 if dt == torch.float32 else 1e-2)


# ------------------------------------------------------------------------------------------------------------ GPU: whole models
CONFIGS = {
    # odd sizes that differ per layer; grouped and single key / value heads; unequal and equal head sizes; rotation of some, all and no entries;
    # windows below, at and above a page; a layer that reads another's cache with another window; every kind of feed-forward including none, no
    # shared expert, top 1; one to six taps; norm parts that are not the groups
    "odd": O.make_config([
        O.mamba2_layer(3, 6, 5, groups=3, conv=3, norm_groups=2, mlp=O.dense(20)),
        O.attention_layer(6, 2, 10, 6, 13, scale=0.5, rot_dims=6, base=300.0, mlp=O.moe(5, 3, 18, shared_ff=10)),
        O.mamba2_layer(1, 12, 7, conv=6),
        O.attention_layer(2, 2, 8, 8, 16, scale=0.4, rot_dims=8, base=40.0, mlp=O.moe(3, 1, 9)),
        O.attention_layer(4, 2, 10, 6, 29, scale=0.3, rot_dims=6, base=300.0, kv_from=1, mlp=O.dense(30)),
        O.mamba2_layer(4, 4, 4, groups=2, conv=1, norm_groups=4, mlp=O.moe(4, 2, 6)),
        O.attention_layer(3, 1, 14, 20, 7, scale=0.3),
    ], vocab=61, width=42, eps=1e-5),
    # aligned sizes (tensor-core GEMMs in bf16, 16-byte paths, the chunked recurrence), head sizes 64 and 128, three query heads on one, no window
    "aligned": O.make_config([
        O.attention_layer(3, 1, 64, 64, 24, rot_dims=32, base=1e5, mlp=O.moe(8, 2, 32, shared_ff=64)),
        O.mamba2_layer(4, 48, 64, groups=1, norm_groups=4, mlp=O.moe(8, 3, 32)),
        O.attention_layer(2, 1, 128, 128, 0, rot_dims=128, mlp=O.dense(128)),
        O.mamba2_layer(2, 64, 16, groups=2, conv=2, mlp=O.dense(192)),
        O.attention_layer(4, 1, 128, 128, 37, rot_dims=128, kv_from=2, mlp=O.dense(128)),
    ], vocab=96, width=192, eps=1e-6),
    # no attention layer at all: nothing is cached per token, everything lives in the state slots
    "recurrent": O.make_config([O.mamba2_layer(2, 8, 8, mlp=O.dense(16)), O.mamba2_layer(2, 4, 12, groups=2, conv=2, mlp=O.moe(2, 1, 8, shared_ff=8))], vocab=40, width=24),
    # no recurrent layer at all: no state slots; two layers read the first one's cache
    "attention": O.make_config([O.attention_layer(2, 1, 8, 12, 18, rot_dims=4, mlp=O.dense(16)), O.attention_layer(4, 1, 8, 12, 5, rot_dims=4, kv_from=0, mlp=O.moe(3, 2, 8)),
                                O.attention_layer(3, 1, 8, 12, 40, rot_dims=4, kv_from=0)], vocab=40, width=24),
}
_MODELS = {}


def _model(name, tmp_path_factory, dt=torch.float32):
    """fp32 runs keep the configured top-k (every selection is compared tightly).  bf16 runs let every token use ALL experts of a layer, weighted by
    their scores: a top-k choice between two close scores flips under rounding and the flipped token then colours the rest of its sequence through
    the recurrent state, which says nothing about the engine (the selection itself is checked on equal inputs above)."""
    every = dt == torch.bfloat16
    if (name, every) not in _MODELS:
        cfg = copy.deepcopy(CONFIGS[name])
        if every:
            for L in cfg["layers"]:
                if L["mlp"] is not None and L["mlp"]["kind"] == "moe":
                    L["mlp"]["router"]["top"] = L["mlp"]["router"]["experts"]
        # seeds whose models are well conditioned: with unlucky ones a token's gated values nearly cancel in front of a grouped norm, and rounding the
        # oracle's own convolution results to bf16 moves its logits by a quarter of their spread
        w = O.random_weights(cfg, seed=9 if name == "aligned" else len(name), router_gain=1.0 if every else 4.0)
        _MODELS[(name, every)] = (cfg, w, O.write_model(str(tmp_path_factory.mktemp(name)), cfg, w))
    return _MODELS[(name, every)]


def _engine(path, dt, pool_tokens=256, block=16, max_seqs=4):
    from deepspeedsyclsupport_b200.inference.v2.config_v2 import RaggedInferenceEngineConfig
    from deepspeedsyclsupport_b200.inference.v2.engine_factory import build_hf_engine
    from deepspeedsyclsupport_b200.inference.v2.ragged.manager_configs import AllocationMode, DSStateManagerConfig, MemoryConfig
    mgr = DSStateManagerConfig(max_tracked_sequences=max_seqs, max_ragged_sequence_count=max_seqs, max_ragged_batch_size=pool_tokens, max_context=pool_tokens,
                               memory_config=MemoryConfig(mode=AllocationMode.ALLOCATE, size=pool_tokens // block), kv_block_size=block)
    return build_hf_engine(path, RaggedInferenceEngineConfig(state_manager=mgr), dtype=dt)


def _close(got, want, dt):
    """Every logit row agrees up to a per-row shift, relative to the spread of the logits.  fp32: tightly.  bf16: within a few times what
    rounding of the matrix products does to these small random models, far below what a wrong key, a lost state or a wrong expert causes
    (order 1)."""
    d = got.cpu().double() - want
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.std()
    if dt == torch.float32:
        return float(err.max()) < 5e-5, float(err.max())
    return float(err.max()) < 0.2 and float(err.median()) < 0.05, (float(err.median()), float(err.max()))


def _tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n, ), generator=torch.Generator().manual_seed(seed))


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_every_layer(name, dt, tmp_path_factory):
    cfg, w, path = _model(name, tmp_path_factory, dt)
    eng = _engine(path, dt)
    toks = _tokens(cfg, 75, 1)
    want, res = O.run(cfg, w, toks.tolist(), collect_layers=True)
    got_res = []
    eng.model()._layer_hook = lambda li, x: got_res.append(x.clone())
    got = eng.put([7], [toks], logit_positions=[list(range(75))])
    assert got.shape == (75, cfg["vocab"]) and len(got_res) == len(res)
    for r, (a, b) in enumerate(zip(got_res, res)):
        if dt == torch.float32:
            assert torch.allclose(a.cpu().double(), b, rtol=1e-4, atol=1e-4), f"layer {r}"
        else:
            row = (a.cpu().double() - b).norm(dim=-1) / b.norm(dim=-1)
            assert float(row.max()) < 0.2 and float(row.median()) < 0.04, f"layer {r}"
    ok, err = _close(got, want, dt)
    assert ok, err
    eng.model()._layer_hook = None  # the same without the per-layer sums: the last layer's outputs join the stream inside the final norm
    eng.flush(7)
    again = eng.put([8], [toks], logit_positions=[[3, 74]])
    assert _close(again, want[[3, 74]], dt)[0]


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name,cuts", [("odd", [1] * 60), ("odd", [2, 2, 15, 1, 17, 3, 2, 18]), ("aligned", [16, 16, 1, 1, 6, 2, 30]), ("aligned", [31, 2, 7, 32]),
                                       ("recurrent", [3, 33, 2, 2, 1, 1, 9]), ("attention", [2, 14, 1, 1, 17, 2, 20])])
def test_portions_and_token_by_token_equal_the_whole_prompt(name, cuts, dt, tmp_path_factory):
    """Prefill against decoding token by token, and portions cut inside pages (block 16), down to two tokens."""
    cfg, w, path = _model(name, tmp_path_factory, dt)
    eng = _engine(path, dt)
    toks = _tokens(cfg, sum(cuts), 2)
    want = O.run(cfg, w, toks.tolist())
    rows, at = [], 0
    for n in cuts:
        rows.append(eng.put([3], [toks[at:at + n]], logit_positions=[list(range(n))]))
        at += n
    ok, err = _close(torch.cat(rows), want, dt)
    assert ok, err


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", ["odd", "aligned"])
def test_unequal_requests_in_one_batch_and_reused_pages_and_slots(name, dt, tmp_path_factory):
    """Four requests of unequal length share steps (portions beside single tokens), one pauses for a step, they finish at different
    times, and two more take over their state slots and pages: every logit row equals the request run alone."""
    cfg, w, path = _model(name, tmp_path_factory, dt)
    eng = _engine(path, dt, pool_tokens=160, block=16)
    prompts = {u: _tokens(cfg, n, 10 + u) for u, n in ((0, 50), (1, 17), (2, 33), (3, 1), (4, 48), (5, 31))}
    want = {u: O.run(cfg, w, p.tolist()) for u, p in prompts.items()}
    schedule = [[(0, 20), (1, 16), (3, 1)], [(0, 1), (2, 30)], [(0, 1), (1, 1), (2, 1)], [(0, 28), (2, 1)], [(2, 1), (4, 15)], [(4, 33), (5, 2)], [(5, 29)]]
    at, got = {u: 0 for u in prompts}, {u: [] for u in prompts}
    free0 = eng.free_blocks
    for step in schedule:
        uids = [u for u, _ in step]
        out = eng.put(uids, [prompts[u][at[u]:at[u] + n] for u, n in step], logit_positions=[list(range(n)) for _, n in step])
        r = 0
        for u, n in step:
            got[u].append(out[r:r + n])
            r += n
            at[u] += n
            if at[u] == len(prompts[u]):
                eng.flush(u)
    assert eng.free_blocks == free0 and all(at[u] == len(p) for u, p in prompts.items())
    assert eng._state_manager.state_slots.free_slots == 4
    for u in prompts:
        ok, err = _close(torch.cat(got[u]), want[u], dt)
        assert ok, (u, err)


@gpu
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_long_decoding_through_the_step_graphs(name, tmp_path_factory):
    """A prompt, then 150 single-token steps (the steady-state ones replay a captured graph) across page borders; some steps ask for no
    logits."""
    cfg, w, path = _model(name, tmp_path_factory)
    eng = _engine(path, torch.float32, pool_tokens=256, block=16)
    toks = _tokens(cfg, 200, 5)
    want = O.run(cfg, w, toks.tolist())
    got = [eng.put([1], [toks[:50]], logit_positions=[[49]])]
    keep = [49]
    for i in range(50, 200):
        wanted = i % 7 != 0
        out = eng.put([1], [toks[i:i + 1]], logit_positions=[[0] if wanted else []])
        assert out.shape[0] == int(wanted)
        if wanted:
            got.append(out)
            keep.append(i)
    ok, err = _close(torch.cat(got), want[keep], torch.float32)
    assert ok, err
    graphs = eng.model()._graphs
    assert 1 in graphs and (1, 0) in graphs, list(graphs)


@gpu
def test_greedy_generation_through_the_scheduler(tmp_path_factory):
    """Prompts are split into portions and fused with running decodes; the tokens are those of the oracle."""
    from deepspeedsyclsupport_b200.inference.v2.scheduler import SplitFuseScheduler
    cfg, w, path = _model("odd", tmp_path_factory)
    eng = _engine(path, torch.float32, pool_tokens=192, block=16)
    sched = SplitFuseScheduler(eng, token_budget=24)  # prompts are split into portions and fused with running decodes
    prompts = {0: _tokens(cfg, 37, 20), 1: _tokens(cfg, 5, 21), 2: _tokens(cfg, 21, 22)}
    for u, p in prompts.items():
        sched.add_request(u, p, max_new_tokens=6)
    done = sched.run_to_completion()
    for u, p in prompts.items():
        assert done[u] == O.greedy(cfg, w, p.tolist(), 6), u


@gpu
def test_trace_runner_replays_steps(tmp_path_factory):
    """bin/trace_run as a process: portions of three requests beside single tokens, a request that pauses for a step, wanted positions
    anywhere in a portion, requests ending at different steps with their pages and slots reused by a later one (pool of 3 pages)."""
    import json
    import subprocess
    cfg, w, path = _model("odd", tmp_path_factory)
    out_dir = str(tmp_path_factory.mktemp("trace_out"))
    reqs = {"a": _tokens(cfg, 70, 31).tolist(), "b": _tokens(cfg, 9, 32).tolist(), "c": _tokens(cfg, 64, 33).tolist(), "d": _tokens(cfg, 100, 34).tolist()}
    want = {k: O.run(cfg, w, v) for k, v in reqs.items()}
    plan = [[("a", 30, [0, 29]), ("b", 8, [3])], [("a", 2, [1]), ("c", 64, [63])], [("a", 37, [36]), ("b", 1, [0])], [("a", 1, [0]), ("d", 64, [])],
            [("d", 2, [0, 1])], [("d", 1, [])], [("d", 33, [32])]]
    at = {k: 0 for k in reqs}
    lines, expect = [], []
    for n, step in enumerate(plan):
        entries, end, rows = [], [], []
        for k, cnt, wanted in step:
            entries.append({"id": k, "tokens": reqs[k][at[k]:at[k] + cnt], "want": wanted})
            rows += [want[k][at[k] + p] for p in wanted]
            at[k] += cnt
            if at[k] == len(reqs[k]):
                end.append(k)
        lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
        expect.append(torch.stack(rows) if rows else None)
    assert all(at[k] == len(v) for k, v in reqs.items())
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", out_dir, "--max-tokens", "192"],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {n}" for n in range(len(plan))]
    for n, e in enumerate(expect):
        f = os.path.join(out_dir, f"{n}.f32")
        if e is None:
            assert not os.path.exists(f)
            continue
        got = torch.frombuffer(bytearray(open(f, "rb").read()), dtype=torch.float32).view(len(e), cfg["vocab"])
        ok, err = _close(got, e, torch.float32)
        assert ok, (n, err)


@gpu
def test_bf16_portions_of_every_kind_give_the_same_logits(tmp_path_factory):
    """The same 330 tokens whole (chunked recurrence), in portions around the chunk length, and half of them one by one: bf16 logits agree with the
    oracle and with one another however they were cut."""
    cfg, w, path = _model("aligned", tmp_path_factory, torch.bfloat16)
    toks = _tokens(cfg, 330, 12)
    want = O.run(cfg, w, toks.tolist())
    runs = []
    for cuts in ([330], [127, 129, 31, 2, 41], [165] + [1] * 165):
        eng = _engine(path, torch.bfloat16, pool_tokens=384, block=64)
        rows, at = [], 0
        for n in cuts:
            rows.append(eng.put([1], [toks[at:at + n]], logit_positions=[list(range(n))]))
            at += n
        runs.append(torch.cat(rows))
        ok, err = _close(runs[-1], want, torch.bfloat16)
        assert ok, (cuts[:4], err)
    for r in runs[1:]:
        assert _close(r, runs[0].cpu().double(), torch.bfloat16)[0]
