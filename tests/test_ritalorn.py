"""Ritalorn on the ragged engine against the plain float64 oracle of tests/ritalorn_oracle.py: every mechanism alone (the stream mixing of
csrc/ragged/hyper_ops.cu, the gelu gate of csrc/ragged/latent_ops.cu, the convolved / distance-biased / gated / cache-sharing attention and the
low-rank attention with neighbouring rotated pairs of csrc/ragged/sink_attention_ops.cu and csrc/attn/paged_flash.cu), then whole models of several
small random configurations through the engine factory, the paged cache, the state slots, the scheduler and the decode-step graphs."""
import copy
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import ritalorn_oracle as O  # noqa: E402

F64 = torch.float64
EPS = 1e-5


# ------------------------------------------------------------------------------------------------------------------ CPU: plumbing
def test_spec_reads_every_size_from_the_config():
    from deepspeedsyclsupport_b200.inference.v2.model_implementations.ritalorn import RitalornSpec
    cfg = O.make_config([O.attention_layer(6, 3, 10, 14, 9, scale=0.3, conv=5, ff=22), O.latent_layer(3, 6, 4, 9, 11, 13, scale=0.7, base=500.0),
                         O.attention_layer(3, 3, 10, 14, 0, kv_from=0, conv=0)], vocab=77, width=40, eps=3e-5, streams=5, softcap=12.5)
    s = RitalornSpec.from_config(cfg)
    assert (s.vocab_size, s.hidden_size, s.norm_eps, s.num_layers, s.streams, s.logit_softcap) == (77, 40, 3e-5, 3, 5, 12.5)
    a, m = s.layers[0].attn, s.layers[1].latent
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.conv, a.scale, a.chunk, a.kv_from, s.layers[0].ff) == (6, 3, 10, 14, 5, 0.3, 9, None, 22)
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.rot_dims, m.rot_base, m.window) == (3, 6, 4, 9, 11, 0.7, 4, 500.0, 13)
    r = s.layers[2].attn
    assert (r.kv_from, r.chunk, r.conv, s.layers[2].ff) == (0, 0, 1, 0)
    reader = cfg["layers"][2]["mixer"]
    for i, change in ((0, dict(type="other")), (1, dict(mlp={"kind": "other"})), (2, dict(mixer=dict(reader, kv_from=1))), (2, dict(mixer=dict(reader, kv_from=2))),
                      (2, dict(mixer=dict(reader, dim=12)))):
        layers = copy.deepcopy(cfg["layers"])
        layers[i].update(change)
        with pytest.raises(ValueError):
            RitalornSpec.from_config(dict(cfg, layers=layers))


def test_family_is_registered_and_chosen_by_the_config():
    from deepspeedsyclsupport_b200.inference.v2.engine_factory import model_type_of
    from deepspeedsyclsupport_b200.inference.v2.model_implementations import FAMILIES, RitalornPolicy, policy_for
    assert model_type_of({"architecture": "Ritalorn"}) == "ritalorn" and policy_for("ritalorn") is RitalornPolicy and "ritalorn" in FAMILIES


def _cpu_model(cfg, w, dt):
    from deepspeedsyclsupport_b200.inference.v2.checkpoint import InMemoryModelEngine
    from deepspeedsyclsupport_b200.inference.v2.engine_factory import build_model_from_checkpoint
    return build_model_from_checkpoint("ritalorn", cfg, InMemoryModelEngine(w), None, device=torch.device("cpu"), dtype=dt)


def test_cache_state_and_fused_weights_of_a_model():
    cfg = O.make_config([O.attention_layer(4, 2, 6, 10, 7, ff=20), O.latent_layer(3, 6, 4, 9, 11, 13), O.attention_layer(2, 1, 12, 12, 5, conv=0),
                         O.attention_layer(8, 2, 6, 10, 3, conv=4, kv_from=0)], width=24)
    w = O.random_weights(cfg)
    m = _cpu_model(cfg, w, torch.float32)
    kc = m.kv_cache_config(block_size=32)
    # unequal key / value head sizes: a key and a value tensor; equal: one two-plane tensor; a latent row; a reading layer has none of its own
    assert kc.layer_shapes == [(1, 2, 6), (1, 2, 10), (1, 1, 15), (2, 1, 12)] and kc.cache_dtype == "fp32"
    assert m._cache_index == {0: (0, 1), 1: (2, ), 2: (3, ), 3: (0, 1)}
    assert {s.name: tuple(s.shape) for s in m.state_config()} == {"l0.mix.conv": (2, 24 + 12 + 20), "l3.mix.conv": (3, 48)}
    c = m.layers[0]
    assert c["in_w"].shape == (56 + 40, 24) and torch.equal(c["in_w"][56:], w["l0.mix.g"].float()) and c["conv_w"].shape == (3, 56)
    odd = m.layers[2]["in_w"]  # 24 + 12 + 12 channels, then the gate; no fill needed; the convolution is absent
    assert odd.shape == (48 + 24, 24) and "conv_w" not in m.layers[2]
    assert m.layers[3]["in_w"].shape == (48 + 80, 24) and m.layers[1]["in_w"].shape == (30 + 15, 24) and m.layers[0]["ff_in_w"].shape == (40, 24)
    assert m.layers[0]["mix1"].shape == (3, 3) and m.layers[0]["mix1"].dtype == torch.float32 and "norm2_w" not in m.layers[1]
    for missing in ("l0.mix.k.b", "l0.mlp.down", "l0.hc2.mix", "l0.ls2", "l1.hc1.out", "l1.mix.dkv.norm", "l3.mix.q.conv", "l3.mix.o.b", "l2.norm1", "head",
                    "final.norm"):
        with pytest.raises(Exception):  # a missing tensor is reported, not ignored
            w2 = dict(w)
            w2.pop(missing)
            _cpu_model(cfg, w2, torch.float32)


def test_gate_rows_start_at_an_aligned_column():
    cfg = O.make_config([O.attention_layer(3, 1, 5, 7, 4)], width=16)  # 15 + 5 + 7 = 27 channels
    w = O.random_weights(cfg)
    in_w = _cpu_model(cfg, w, torch.float32).layers[0]["in_w"]
    assert in_w.shape == (32 + 21, 16) and float(in_w[27:32].abs().max()) == 0 and torch.equal(in_w[32:], w["l0.mix.g"].float())


def test_bf16_heads_get_a_tensor_core_width_and_slots():
    """bf16: heads padded to 64 / 128, three query heads per key / value head in four slots; the output is compact all the same."""
    cfg = O.make_config([O.attention_layer(6, 2, 6, 10, 8), O.attention_layer(5, 1, 96, 40, 8), O.attention_layer(2, 2, 130, 20, 8), O.latent_layer(3, 8, 6, 5, 40, 9)],
                        width=24)
    m = _cpu_model(cfg, O.random_weights(cfg), torch.bfloat16)
    assert m.kv_cache_config(block_size=16).layer_shapes == [(2, 2, 64), (2, 1, 128), (1, 2, 130), (1, 2, 20), (1, 1, 64)]
    assert [(a.head_slots, a.out_width) for a in m.attn_mods[:3]] == [(4, 60), (8, 200), (1, 40)]


def test_module_choice():
    from deepspeedsyclsupport_b200.inference.v2.inference_utils import DtypeEnum, NormTypeEnum
    from deepspeedsyclsupport_b200.inference.v2.modules import heuristics
    from deepspeedsyclsupport_b200.inference.v2.modules.configs import DSConvSinkAttentionConfig, DSNormConfig, DSRotaryLatentAttentionConfig
    io = dict(input_dtype=DtypeEnum.bf16, output_dtype=DtypeEnum.bf16)
    norm = DSNormConfig(max_tokens=8, type=NormTypeEnum.RMSNorm, channels=8, residual_dtype=DtypeEnum.fp32, streams=2, **io)
    assert heuristics.instantiate_pre_norm(norm, None).name() == "cuda_stream_mix_rms"
    kw = dict(max_tokens=8, n_heads_q=4, n_heads_kv=2, head_size=6, value_size=5, conv_taps=2, scale=1.0, max_sequences=2, **io)
    mod = heuristics.instantiate_attention(DSConvSinkAttentionConfig(linear_bias=True, output_gate=True, **kw), None)
    assert mod.name() == "conv_sink_attention" and torch.allclose(mod._linear_slopes(torch.device("cpu"))[0].double(), O.linear_slopes(4))
    for bad in (dict(linear_bias=True, distance_bias=True), dict(reads_cache=True, value_mix="mix"), dict(part_size=-1)):
        with pytest.raises(ValueError):
            DSConvSinkAttentionConfig(**dict(kw, **bad))
    lat = dict(max_tokens=8, n_heads=2, qk_dim=4, rot_dim=4, v_dim=4, kv_rank=8, scale=1.0, rotate_dim=4, max_sequences=2, **io)
    assert heuristics.instantiate_attention(DSRotaryLatentAttentionConfig(interleaved=True, window=5, **lat), None).name() == "rotary_latent_attention"
    with pytest.raises(ValueError):
        DSRotaryLatentAttentionConfig(window=-1, **lat)


# ------------------------------------------------------------------------------------------------------------- GPU: mechanisms
gpu = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _K():
    from deepspeedsyclsupport_b200.inference.v2 import kernels
    return kernels


class _Batch:
    """Ragged metadata of a step, built by hand: seqs = [(slot, seen, new tokens, block ids)]."""

    def __init__(self, seqs, block, max_blocks=32):
        tok_seq, tok_pos, desc, at = [], [], [], 0
        bt = torch.zeros(len(seqs), max_blocks, dtype=torch.int32)
        for i, (slot, seen, n, blocks) in enumerate(seqs):
            assert -(-(seen + n) // block) <= len(blocks) <= max_blocks
            tok_seq += [i] * n
            tok_pos += list(range(seen, seen + n))
            desc.append([at, n, seen, slot])
            bt[i, :len(blocks)] = torch.tensor(blocks, dtype=torch.int32)
            at += n
        self.current_sequences, self.current_tokens = len(seqs), at
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

    def __init__(self, slots=4):
        self.buf, self.slots = {}, slots

    def add(self, specs):
        self.buf.update({s.name: torch.full((self.slots, ) + tuple(s.shape), 7.5, dtype=s.dtype, device="cuda") for s in specs})
        return self

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


def _stream_weights(S, D, seed):
    g = torch.Generator().manual_seed(seed)
    r = lambda *n: torch.randn(*n, generator=g)
    return dict(mix=r(S, S), w_out=r(S), w_in=r(S), gamma=1 + 0.3 * r(D), scale=r(D), bias=r(D)), g


# ---- streams
@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("S,D", [(1, 6), (2, 42), (3, 320), (4, 1024), (2, 2056), (4, 6144), (5, 64), (7, 33), (2, 9000)])
def test_streams_are_read_mixed_and_written_at_once(S, D, dt):
    """Widths on and off the 16-byte path, more streams than the unrolled kernel holds, streams of very different size; the join alone, the read
    alone, both in one pass; equal streams given as one row; a row gather that joins for the gathered rows only; branches whose rows are longer than
    the width.  The mixing matrix is not symmetric: from and to must not be exchanged."""
    K = _K()
    p, g = _stream_weights(S, D, 10 * S + D)
    T = 7
    X = torch.randn(T, S, D, generator=g) * torch.tensor([10.0 ** (s % 3) for s in range(S)])[None, :, None]
    y = torch.randn(T, D + 5, generator=g).to(dt)[:, :D]
    dev = {k: v.cuda() for k, v in p.items()}
    tol = 2e-6 if dt == torch.float32 else 4e-3
    Xs = X.double().transpose(0, 1)

    def normed(streams, w_in):
        return O.rms(O.read_streams(streams, w_in), EPS) * p["gamma"].double()

    for bias, scale in ((True, True), (False, True), (False, False)):
        v = y.double() + (p["bias"].double() if bias else 0)
        v = v * p["scale"].double() if scale else v
        joined = O.write_streams(Xs, p["mix"], p["w_out"], v)
        branch = (y.cuda() if D % 2 else y.contiguous().cuda(), dev["bias"] if bias else None, dev["scale"] if scale else None, dev["mix"], dev["w_out"])
        x = X.cuda()
        x2, out = K.stream_mix_norm(x, S, branch, dev["w_in"], dev["gamma"], EPS, out_dtype=dt)
        assert x2.data_ptr() == x.data_ptr() and _rel(x2, joined.transpose(0, 1)) < 1e-6 and out.dtype == dt and _rel(out, normed(joined, p["w_in"])) < tol
        x = X.cuda()
        x2, none = K.stream_mix_norm(x, S, branch)
        assert none is None and _rel(x2, joined.transpose(0, 1)) < 1e-6
        rows = torch.tensor([6, 2, 6], dtype=torch.int32).cuda()
        x = X.cuda()
        _, out = K.stream_mix_norm(x, S, branch, None, dev["gamma"], EPS, out_dtype=dt, rows=rows)  # the model's end: the plain sum of the streams
        assert torch.equal(x.cpu(), X) and out.shape == (3, D) and _rel(out, normed(joined, torch.ones(S))[[6, 2, 6]]) < tol
        first = O.write_streams(torch.stack([Xs[0]] * S), p["mix"], p["w_out"], v)  # all streams equal: one row in, separate rows out
        e = X[:, 0].contiguous().cuda()
        x2, out = K.stream_mix_norm(e, S, branch, dev["w_in"], dev["gamma"], EPS, out_dtype=dt)
        assert x2.shape == (T, S, D) and torch.equal(e.cpu(), X[:, 0]) and _rel(x2, first.transpose(0, 1)) < 1e-6 and _rel(out, normed(first, p["w_in"])) < tol
    x = X.cuda()
    x2, out = K.stream_mix_norm(x, S, None, dev["w_in"], dev["gamma"], EPS, out_dtype=dt)
    assert torch.equal(x2.cpu(), X) and _rel(out, normed(Xs, p["w_in"])) < tol
    e = X[:, 0].contiguous().cuda()
    x2, out = K.stream_mix_norm(e, S, None, dev["w_in"], dev["gamma"], EPS, out_dtype=dt)
    assert x2 is e and _rel(out, normed(torch.stack([Xs[0]] * S), p["w_in"])) < tol


@gpu
@pytest.mark.parametrize("dt", DTYPES)
def test_gelu_gate_of_column_ranges(dt):
    """Aligned and odd columns; values from the far tails of the activation, where a sloppy tanh would leave something, to its middle."""
    K = _K()
    g = torch.Generator().manual_seed(4)
    for c0, F, lead in ((7, 19, 5), (8, 64, 4), (0, 20, 0)):
        gu = torch.randn(13, c0 + 2 * F + 8, generator=g) * 3
        gu[0, c0:c0 + 6] = torch.tensor([-60.0, -9.0, -4.0, 4.0, 60.0, 3e4])
        gu = gu.to(dt).cuda()
        wide = torch.zeros(13, lead + F + 4, dtype=dt, device="cuda")
        K.gelu_gate_cols(gu, c0, c0 + F, F, wide[:, lead:lead + F])
        p = gu.cpu().double()
        want = O.gelu_tanh(p[:, c0:c0 + F]) * p[:, c0 + F:c0 + 2 * F]
        assert torch.allclose(wide[:, lead:lead + F].cpu().double(), want, rtol=3e-6 if dt == torch.float32 else 8e-3, atol=1e-6)
        assert float(wide[:, :lead].abs().sum()) == 0 and float(wide[:, lead + F:].abs().max()) == 0


# ---- convolved attention
def _attention_module(m, dt, eps=EPS):
    from deepspeedsyclsupport_b200.inference.v2.inference_utils import DtypeEnum
    from deepspeedsyclsupport_b200.inference.v2.modules import heuristics
    from deepspeedsyclsupport_b200.inference.v2.modules.configs import DSConvSinkAttentionConfig
    return heuristics.instantiate_attention(DSConvSinkAttentionConfig(
        max_tokens=1024, n_heads_q=m["heads"], n_heads_kv=m["kv_heads"], head_size=m["dim"], value_size=m["vdim"], conv_taps=m.get("conv", 1), scale=m["scale"],
        part_size=(m.get("mask") or {}).get("size", 0), qk_norm_weight=False, linear_bias=True, output_gate=True, reads_cache=m.get("kv_from") is not None,
        eps=eps, max_sequences=8, input_dtype=DtypeEnum(dt), output_dtype=DtypeEnum(dt)), None)


def _caches(mod, blocks, block, dt):
    return [torch.full((blocks, ) + ((p, ) if p != 1 else ()) + (block, h, d), 3.0, dtype=dt, device="cuda") for p, h, d in mod.cache_shapes()]


def _run_attention(mod, w, h, dt, caches, batch, st, prefix="m"):
    """Gated heads [n, H dv] of one step whose rows are h (float64): the projections of a model, the module, no output projection."""
    c = mod._config
    names = ("q", ) if c.reads_cache else ("q", "k", "v")
    proj = torch.cat([h @ torch.cat([w[n] for n in names]).double().T, torch.full((h.shape[0], 3), 9.0, dtype=F64), h @ w["g"].double().T], 1).to(dt).cuda()
    C = mod.conv_channels
    taps = torch.cat([w[n + ".conv"] for n in names]).float().t().contiguous().cuda() if c.conv_taps > 1 else torch.ones(1, C).cuda()
    bias = torch.cat([w[n + ".b"] for n in names]).float().cuda()
    out = torch.full((h.shape[0], mod.out_width + 5), 4.0, dtype=dt, device="cuda")
    mod(proj, 0, bias, taps, None, None, None, None, None, caches[0], caches[1] if len(caches) > 1 else None, batch, st, prefix, out[:, :mod.out_width],
        gate=proj[:, C + 3:])
    assert float((out[:, mod.out_width:] - 4).abs().max()) == 0  # nothing behind the heads is touched
    return out[:, :mod.out_width]


def _bare(w, m):
    """The mixer without its output projection."""
    n = m["heads"] * m["vdim"]
    return dict(w, **{"o": torch.eye(n).bfloat16(), "o.b": torch.zeros(n)})


ATTENTION_CASES = [
    dict(heads=6, kv_heads=2, dim=10, vdim=6, conv=3, mask=dict(size=19)),  # three query heads per key / value head, unequal sizes
    dict(heads=2, kv_heads=2, dim=8, vdim=8, conv=1, mask=dict(size=1)),  # chunks of one: the token itself; no convolution
    dict(heads=5, kv_heads=1, dim=14, vdim=20, conv=6, mask=dict(size=500)),  # five heads on one, values wider than keys, one chunk
    dict(heads=4, kv_heads=4, dim=64, vdim=40, conv=4, mask=dict(size=33)),
    dict(heads=4, kv_heads=2, dim=128, vdim=128, conv=2, mask=dict(size=48)),
    dict(heads=12, kv_heads=2, dim=72, vdim=30, conv=3),  # no mask; six heads per key / value head padded to 128
    dict(heads=1, kv_heads=1, dim=32, vdim=96, conv=2, mask=dict(size=64)),  # one head: a slope of 2^-8
    dict(heads=2, kv_heads=1, dim=136, vdim=40, conv=3, mask=dict(size=16)),  # heads above 128: the CUDA-core kernel in bf16 too
]


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", range(len(ATTENTION_CASES)))
@pytest.mark.parametrize("sizes", [[90], [50] + [1] * 40, [2, 5, 1, 25, 2, 9, 46]])
def test_attention_mixer_and_a_layer_that_reads_its_cache(case, sizes, dt):
    """Whole, a prompt followed by single tokens, and portions cut inside pages (block 16), chunks and convolutions, on shuffled pages and in a slot
    that held something else.  A second layer with queries, a chunk length and taps of its own -- and another number of query heads -- reads the first
    one's keys and values."""
    m = dict(ATTENTION_CASES[case])
    m["scale"] = 1.7 * m["dim"] ** -0.5
    D, T, G = 24, 90, m["kv_heads"]
    reader = dict(m, heads=2 * G, mask=dict(size=27), kv_from=0, conv=1 + case % 4)
    strip = lambda x: {k: v for k, v in x.items() if k != "conv" or v > 1}
    cfg = O.make_config([dict(type="attention", mixer=strip(m), mlp=None), dict(type="attention", mixer=strip(reader), mlp=None)], width=D)
    ws = O.random_weights(cfg, seed=case)
    w, wr = _bare(O.sub(ws, "l0.mix."), m), _bare(O.sub(ws, "l1.mix."), reader)
    assert "k" not in wr and "v" not in wr
    g = torch.Generator().manual_seed(5)
    h, hr = (torch.randn(T, D, generator=g).bfloat16().double() for _ in range(2))
    want, st_own = O.attention_mixer(h, w, m, EPS)
    want_r, _ = O.attention_mixer(hr, wr, reader, EPS, foreign=st_own[1:])
    mod, mod_r = _attention_module(m, dt), _attention_module(reader, dt)
    assert mod_r.cache_shapes() == []
    st = _State().add(mod.state_specs("m")).add(mod_r.state_specs("r"))
    caches, pages = _caches(mod, 9, 16, dt), [5, 2, 7, 0, 3, 8]
    got, got_r = [], []
    for at, n in _cuts(T, sizes):
        b = _Batch([(2, at, n, pages)], 16)
        got.append(_run_attention(mod, w, h[at:at + n], dt, caches, b, st))
        got_r.append(_run_attention(mod_r, wr, hr[at:at + n], dt, caches, b, st, "r"))
    tol = 3e-5 if dt == torch.float32 else 2.5e-2
    assert _rel(torch.cat(got), want) < tol
    assert _rel(torch.cat(got_r), want_r) < tol


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("d,G,group", [(64, 2, 2), (128, 1, 3), (128, 2, 4), (24, 2, 1)])
@pytest.mark.parametrize("chunk", [15, 16, 80, 128, 130])
def test_a_strong_key_fills_its_chunk_and_no_other(chunk, d, G, group, dt):
    """ONE key that every query loves: it takes the output of every later query of its chunk and shows in none of the next chunk -- keys at a
    chunk's, a page's and a kernel tile's first / last row, in prompt portions and for decoded tokens."""
    K = _K()
    H, T, block = G * group, 330, 16
    P = 64 if d <= 64 else 128
    g = torch.Generator().manual_seed(chunk + d)
    pad = dt == torch.bfloat16
    slots = 1 << (group - 1).bit_length() if pad else group
    for far in (0, chunk - 1, chunk, 127, 128, 200):
        if far >= T - 2:
            continue
        q = torch.randn(T, H, d, generator=g, dtype=F64) * 0.05
        k = torch.randn(T, G, d, generator=g, dtype=F64) * 0.05
        v = torch.randn(T, G, d, generator=g, dtype=F64)
        q[..., 0] += 3.0
        k[far, :, 0] += 60.0  # stands out whatever the distance takes off
        v[far] += 20.0
        q, k, v = (t.bfloat16().double() for t in (q, k, v))
        want = O.attend(q, k, v, 1.0, lambda i, j: O.sees_part(i, j, chunk), slopes=O.linear_slopes(H))
        end = (far // chunk + 1) * chunk  # first position of the next chunk
        assert float(want[far:min(end, T)].min()) > 14 and (far == 0 or float(want[far - 1].max()) < 8) and (end >= T or float(want[end:].max()) < 8)
        pages = torch.randperm(30, generator=g)[:-(-T // block)].tolist()
        W = P if pad else d
        cache = torch.full((30, 2, block, G, W), 3.0, dtype=dt)
        blk, slot = torch.tensor(pages)[torch.arange(T) // block], torch.arange(T) % block
        for plane, rows in ((0, k), (1, v)):
            cache[blk, plane, slot] = torch.nn.functional.pad(rows, (0, W - d)).to(dt)
        cache = cache.cuda()
        qp = torch.zeros(T, G, slots, W, dtype=dt)
        qp[:, :, :group, :d] = q.view(T, G, group, d).to(dt)
        qp = qp.reshape(T, -1).cuda()
        sl = torch.zeros(G, slots)
        sl[:, :group] = O.linear_slopes(H).view(G, group).float()
        cut = max(2, min(end - 3, T - 9))
        rows, at = [], 0
        for n in [cut] + [1] * 8 + [T]:  # decoded tokens across the edge, portions before and behind
            n = min(n, T - at)
            if n <= 0:
                break
            b = _Batch([(0, at, n, pages)], block)
            out = torch.empty(n, H * d, dtype=dt, device="cuda")
            if pad:
                assert K.paged_flash_sink_ok(qp[at:at + n], cache, out, G * slots, G, W, W, compact=True)
                K.paged_flash_sink(qp[at:at + n], cache, b.tok_seq(), b.tok_pos(), b.block_table(), out, G * slots, G, W, 1.0, 0.0, 0.0, r1=sl.reshape(-1).cuda(),
                                   part=chunk, decode=n == 1, compact=(group, d))
            else:
                kp, vp = K.cache_planes(cache)
                K.sink_attention_ex(qp[at:at + n], d, kp, d, vp, d, b.tok_seq(), b.tok_pos(), b.block_table(), block, out, d, H, G, d, d, 1.0,
                                    r1=O.linear_slopes(H).float().cuda(), part=chunk)
            rows.append(out)
            at += n
        got = torch.cat(rows).cpu().double().view(T, H, d)
        assert float((got - want).abs().max()) < (1e-3 if dt == torch.float32 else 0.25), far


@gpu
@pytest.mark.parametrize("dt", DTYPES)
def test_the_distance_term_counts_positions_and_heads(dt):
    """Equal keys: the weights are those of the distance term alone, head by head (a steep first and an almost flat last head), far from the sequence's
    start, through the linear slopes of the module."""
    m = dict(heads=6, kv_heads=2, dim=16, vdim=12, scale=1.0, mask=dict(size=300))
    w = {n: torch.zeros(r, 4) for n, r in (("q", 96), ("k", 32), ("v", 24), ("g", 72))}
    w.update({"q.b": torch.ones(96), "k.b": torch.ones(32), "v.b": torch.zeros(24)})
    w["v"][:, 0] = 1.0
    w["g"][:, 1] = torch.linspace(-3, 3, 72)
    w = _bare(w, m)
    h = torch.zeros(280, 4, dtype=F64)
    h[:, 0] = (torch.arange(280) % 37).double() - 18
    h[:, 1] = torch.linspace(-1, 1, 280).bfloat16().double()
    want, _ = O.attention_mixer(h, w, m, EPS)
    flat = O.attend(torch.ones(280, 6, 16, dtype=F64), torch.ones(280, 2, 16, dtype=F64), h[:, :1, None].expand(280, 2, 12), 1.0, lambda i, j: j <= i)
    assert float((want.view(280, 6, 12)[-1, 0] - flat[-1, 0]).abs().max()) > 0.4  # the term shows
    mod = _attention_module(m, dt)
    caches, st = _caches(mod, 20, 16, dt), _State().add(mod.state_specs("m"))
    got = torch.cat([_run_attention(mod, w, h[at:at + n], dt, caches, _Batch([(0, at, n, list(range(18)))], 16), st) for at, n in _cuts(280, [250] + [1] * 30)])
    assert _rel(got, want) < (1e-5 if dt == torch.float32 else 1e-2)


@gpu
@pytest.mark.parametrize("d", [64, 128])
def test_split_keys_and_long_distances_on_the_tensor_cores(d):
    """The tcgen05 kernels against the CUDA-core one with and without key splits, chunks and a gate, on contexts of thousands of keys: distances far
    beyond what fp32 sums of (slope x position) would hold to the last bit."""
    K = _K()
    g = torch.Generator().manual_seed(d)
    G, group, block, H = 2, 3, 64, 6
    slots = 4
    lens = [(0, 5000, 1), (1, 37, 40), (2, 2100, 130), (3, 0, 2)]
    n_blocks = sum(-(-(s + n) // block) for _, s, n in lens)
    order = torch.randperm(n_blocks, generator=g).tolist()
    seqs = []
    for slot, seen, n in lens:
        k = -(-(seen + n) // block)
        seqs.append((slot, seen, n, order[:k]))
        order = order[k:]
    b = _Batch(seqs, block, max_blocks=80)
    T = b.current_tokens
    cache = (torch.randn(n_blocks, 2, block, G, d, generator=g) * 1.5).bfloat16().cuda()
    q = torch.zeros(T, G, slots, d)
    q[:, :, :group] = torch.randn(T, G, group, d, generator=g) * 1.5
    q = q.reshape(T, -1).bfloat16().cuda()
    dv = d - 24
    gate = (torch.randn(T, H * dv + 8, generator=g) * 2).bfloat16().cuda()[:, :H * dv]
    slopes = torch.tensor([2.0 ** (-2 * h) for h in range(H)])
    sl = torch.zeros(G, slots)
    sl[:, :group] = slopes.view(G, group)
    kp, vp = K.cache_planes(cache)
    for part in (0, 700):
        want = torch.empty(T, H * dv, dtype=torch.bfloat16, device="cuda")
        K.sink_attention_ex(q, d, kp, d, vp, d, b.tok_seq(), b.tok_pos(), b.block_table(), block, want, dv, H, G, d, dv, d ** -0.5, r1=slopes.cuda(), part=part,
                            q_group=slots, gate=gate)
        for splits in (1, 3, None):
            for dec in (False, True):
                got = torch.empty(T, H * dv, dtype=torch.bfloat16, device="cuda")
                K.paged_flash_sink(q, cache, b.tok_seq(), b.tok_pos(), b.block_table(), got, G * slots, G, d, d ** -0.5, 0.0, 0.0, r1=sl.reshape(-1).cuda(), part=part,
                                   decode=dec, n_splits=splits, compact=(group, dv), gate=gate)
                assert _rel(got, want.cpu().double()) < 1e-2, (part, splits, dec)


@gpu
@pytest.mark.parametrize("dt", DTYPES)
def test_unequal_sequences_in_one_attention_step_and_a_slot_taken_over(dt):
    """A portion, a single token and a two-token portion in one batch, each against the sequence alone; then a new sequence in a used slot and on
    used pages, whose convolution must not see the old one."""
    m = dict(heads=6, kv_heads=2, dim=40, vdim=24, conv=4, scale=0.4, mask=dict(size=21))
    cfg = O.make_config([dict(type="attention", mixer=m, mlp=None)], width=24)
    w = _bare(O.sub(O.random_weights(cfg, seed=3), "l0.mix."), m)
    mod = _attention_module(m, dt)
    caches, st = _caches(mod, 24, 16, dt), _State().add(mod.state_specs("m"))
    g = torch.Generator().manual_seed(1)
    hs = {u: torch.randn(n, 24, generator=g).bfloat16().double() for u, n in ((0, 80), (1, 101), (2, 35), (3, 40))}
    pages = {0: [3, 9, 1, 7, 12], 1: [0, 2, 4, 6, 8, 10, 11], 2: [13, 5, 14], 3: [14, 13, 9]}
    slot = {0: 1, 1: 0, 2: 3, 3: 3}
    want = {u: O.attention_mixer(h, w, m, EPS)[0] for u, h in hs.items()}
    at, got = {u: 0 for u in hs}, {u: [] for u in hs}
    for step in ([(1, 100)], [(0, 33), (1, 1), (2, 2)], [(2, 33), (0, 47)], [(3, 1)], [(3, 2)], [(3, 37)]):
        b = _Batch([(slot[u], at[u], n, pages[u]) for u, n in step], 16)
        out = _run_attention(mod, w, torch.cat([hs[u][at[u]:at[u] + n] for u, n in step]), dt, caches, b, st)
        r = 0
        for u, n in step:
            got[u].append(out[r:r + n])
            r += n
            at[u] += n
    for u in hs:
        assert at[u] == len(hs[u]) and _rel(torch.cat(got[u]), want[u]) < (3e-5 if dt == torch.float32 else 2.5e-2), u


# ---- low-rank attention
def _latent_module(m, dt):
    from deepspeedsyclsupport_b200.inference.v2.inference_utils import DtypeEnum
    from deepspeedsyclsupport_b200.inference.v2.modules import heuristics
    from deepspeedsyclsupport_b200.inference.v2.modules.configs import DSRotaryLatentAttentionConfig
    rot = m["rot"]
    return heuristics.instantiate_attention(DSRotaryLatentAttentionConfig(
        max_tokens=1024, n_heads=m["heads"], qk_dim=m["dim"], rot_dim=m["rot_dim"], v_dim=m["vdim"], kv_rank=m["kv_rank"], scale=m["scale"], rotate_dim=rot["dims"],
        interleaved=True, theta_base=rot["base"], window=(m.get("mask") or {}).get("size", 0), eps=EPS, max_sequences=8, input_dtype=DtypeEnum(dt),
        output_dtype=DtypeEnum(dt)), None)


def _run_latent(mod, w, h, dt, cache, batch):
    c = mod._config
    proj = (h @ torch.cat([w["q"], w["dkv"]]).double().T).to(dt).cuda()
    return mod(proj, (0, c.n_heads * (c.qk_dim + c.rot_dim)), cache, batch, w["dkv.norm"].float().cuda(), mod.transform_key_up_param(w["uk"]).cuda(),
               mod.transform_value_up_param(w["uv"]).cuda(), None)


LATENT_CASES = [
    O.latent_layer(3, 6, 4, 9, 10, 19, base=300.0)["mixer"],  # odd sizes; rows padded to 64 on the tensor cores
    dict(O.latent_layer(2, 8, 10, 8, 33, 1)["mixer"], rot=dict(dims=6, base=50.0)),  # a window of one; part of the rotated entries turns
    O.latent_layer(5, 24, 32, 40, 64, 33, base=1e5)["mixer"],  # rows padded to 128, five heads in eight
    O.latent_layer(16, 16, 16, 16, 112, 0)["mixer"],  # exactly 128 values per row, no window
    O.latent_layer(4, 12, 24, 20, 130, 40, base=1e6)["mixer"],  # rows too wide for the tensor-core kernels
    O.latent_layer(1, 5, 2, 3, 4, 500)["mixer"],  # one head, a window that covers everything
]


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case", range(len(LATENT_CASES)))
@pytest.mark.parametrize("sizes", [[90], [50] + [1] * 40, [2, 5, 1, 25, 2, 9, 46]])
def test_latent_mixer(case, sizes, dt):
    m = LATENT_CASES[case]
    cfg = O.make_config([dict(type="latent_attention", mixer=m, mlp=None)], width=24)
    w = O.sub(O.random_weights(cfg, seed=case), "l0.mix.")
    w["o"] = torch.eye(m["heads"] * m["vdim"]).bfloat16()
    h = torch.randn(90, 24, generator=torch.Generator().manual_seed(5)).bfloat16().double()
    want, _ = O.latent_mixer(h, w, m, EPS)
    mod = _latent_module(m, dt)
    (p, hh, row), = mod.cache_shapes()
    cache, pages = torch.full((9, 16, hh, row), 3.0, dtype=dt, device="cuda"), [5, 2, 7, 0, 3, 8]
    got = torch.cat([_run_latent(mod, w, h[at:at + n], dt, cache, _Batch([(0, at, n, pages)], 16)) for at, n in _cuts(90, sizes)])
    assert _rel(got, want) < (3e-5 if dt == torch.float32 else 2.5e-2)


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("R,dr,H", [(24, 8, 3), (96, 32, 4)])
@pytest.mark.parametrize("window", [15, 16, 17, 64, 130])
def test_a_strong_row_is_seen_until_the_last_position_of_the_window(window, R, dr, H, dt):
    """ONE token whose latent every query loves: it takes the output of the window - 1 queries behind it and is gone for the next one; rows at pages'
    and kernel tiles' borders, prompt portions and decoded tokens, after the rotation of thousands of positions would have mattered."""
    D, T, block = R + dr, 300, 16
    m = dict(heads=H, dim=R, rot_dim=dr, vdim=R, kv_rank=R, scale=1.0, mask=dict(size=window), rot=dict(dims=dr, base=100.0))
    eye = torch.eye(R)
    w = {"q": torch.zeros(H * D, D), "dkv": torch.eye(D), "dkv.norm": torch.ones(R), "uk": eye.repeat(H, 1), "uv": eye.repeat(H, 1), "o": torch.eye(H * R)}
    w["q"].view(H, D, D)[:, 0, R] = 1.0  # every query asks for the first latent entry, by an amount it reads from the rotated part's first entry
    mod = _latent_module(m, dt)
    (_, hh, row), = mod.cache_shapes()
    g = torch.Generator().manual_seed(window + R)
    for far in (0, 100, 127, 128, 200):
        h = torch.randn(T, D, generator=g, dtype=F64)
        h[:, 0] *= 0.05
        h[:, R] = 8.0
        h[far, :R] = 0.0
        h[far, 0] = 30.0  # its normed latent is sqrt(R) times the first unit vector
        h = h.bfloat16().double()
        want, _ = O.latent_mixer(h, w, m, EPS)
        first = want.view(T, H, R)[..., 0]
        last, gone = far + window - 1, far + window
        assert float(first[far:last + 1].min()) > 0.8 * R ** 0.5 and (gone >= T or float(first[gone:].abs().max()) < 0.3 * R ** 0.5)  # the oracle shows the edge
        pages = torch.randperm(30, generator=g)[:-(-T // block)].tolist()
        cache = torch.full((30, block, hh, row), 3.0, dtype=dt, device="cuda")
        cut = max(2, min(last - 3, T - 9))
        rows, at = [], 0
        for n in [cut] + [1] * 8 + [T]:
            n = min(n, T - at)
            if n <= 0:
                break
            rows.append(_run_latent(mod, w, h[at:at + n], dt, cache, _Batch([(0, at, n, pages)], block)))
            at += n
        assert float((torch.cat(rows).cpu().double() - want).abs().max()) < (1e-3 if dt == torch.float32 else 0.15), far


@gpu
@pytest.mark.parametrize("dt", DTYPES)
def test_rotation_pairs_neighbours_far_from_the_start(dt):
    """One rotated key part that matches a query only at ONE distance: positions in the thousands, angles far above 2 pi; halves instead of neighbours
    would miss it."""
    m = dict(heads=2, dim=4, rot_dim=12, vdim=4, kv_rank=8, scale=1.0, rot=dict(dims=12, base=7.0), mask=dict(size=40))
    cfg = O.make_config([dict(type="latent_attention", mixer=m, mlp=None)], width=24)
    w = O.sub(O.random_weights(cfg, seed=2), "l0.mix.")
    w["o"] = torch.eye(8).bfloat16()
    for n in ("q", "dkv"):
        w[n] = (w[n].float() * 2).bfloat16()
    h = torch.randn(60, 24, generator=torch.Generator().manual_seed(5)).bfloat16().double()
    pos0 = 3000
    # the oracle at positions pos0 ..: nothing in front is visible through the window of the last 20 rows
    past = (torch.zeros(pos0, 8, dtype=F64), torch.zeros(pos0, 12, dtype=F64))
    want, _ = O.latent_mixer(h, w, m, EPS, pos0, past)
    mod = _latent_module(m, dt)
    (_, hh, row), = mod.cache_shapes()
    blocks = -(-(pos0 + 60) // 64)
    cache = torch.zeros(blocks, 64, hh, row, dtype=dt, device="cuda")
    got = torch.cat([_run_latent(mod, w, h[at:at + n], dt, cache, _Batch([(0, pos0 + at, n, list(range(blocks)))], 64, max_blocks=64)) for at, n in _cuts(60, [41] + [1] * 19)])
    assert _rel(got[40:], want[40:]) < (5e-5 if dt == torch.float32 else 2.5e-2)
    turned = O.rotate_pairs(h[:, :12], torch.arange(60) + pos0, 12, 7.0)
    assert float((turned - h[:, :12]).norm() / h[:, :12].norm()) > 0.5


# ------------------------------------------------------------------------------------------------------------ GPU: whole models
CONFIGS = {
    # odd sizes that differ per layer; grouped and single key / value heads; unequal and equal head sizes; chunks and windows below, at and above a
    # page, absent ones; layers that read another's cache with another chunk; one to six taps; layers without a feed-forward; three streams
    "odd": O.make_config([
        O.attention_layer(6, 2, 10, 6, 13, scale=0.5, conv=3, ff=20),
        O.latent_layer(3, 6, 4, 9, 10, 11, scale=0.4, base=300.0, ff=18),
        O.attention_layer(2, 2, 8, 8, 16, scale=0.4, conv=6),
        O.attention_layer(4, 2, 10, 6, 29, scale=0.3, conv=2, kv_from=0, ff=30),
        O.latent_layer(5, 7, 6, 4, 13, 0, base=40.0),
        O.attention_layer(3, 1, 14, 20, 7, scale=0.3, conv=0, ff=9),
        O.attention_layer(6, 1, 14, 20, 0, scale=0.3, conv=4, kv_from=5),
    ], vocab=61, width=42, eps=1e-5, streams=3, softcap=7.0),
    # aligned sizes (tensor-core GEMMs in bf16, 16-byte paths), head sizes 64 and 128, three query heads on one, latent rows of 64 and 128; no cap
    "aligned": O.make_config([
        O.attention_layer(3, 1, 64, 64, 24, conv=4, ff=128),
        O.latent_layer(4, 32, 16, 48, 48, 24, base=1e5, ff=192),
        O.attention_layer(4, 2, 128, 128, 37, conv=2, ff=128),
        O.attention_layer(4, 2, 128, 128, 64, conv=4, kv_from=2, ff=64),
        O.latent_layer(8, 64, 32, 32, 96, 40, base=1e6, ff=128),
    ], vocab=96, width=192, eps=1e-6, streams=4, softcap=0.0),
    # one stream, no convolution anywhere (no state slots), one feed-forward
    "stateless": O.make_config([O.latent_layer(2, 8, 4, 6, 12, 9), O.attention_layer(2, 1, 8, 12, 18, conv=0, ff=16), O.attention_layer(4, 1, 8, 12, 5, conv=0, kv_from=1)],
                               vocab=40, width=24, streams=1),
    # more streams than the unrolled kernel holds
    "many": O.make_config([O.attention_layer(2, 2, 12, 4, 10, conv=5, ff=24), O.latent_layer(1, 8, 8, 10, 16, 30, ff=8)], vocab=40, width=32, streams=6, softcap=3.0),
}
_MODELS = {}


def _model(name, tmp_path_factory):
    if name not in _MODELS:
        cfg = CONFIGS[name]
        w = O.random_weights(cfg, seed=len(name))
        _MODELS[name] = (cfg, w, O.write_model(str(tmp_path_factory.mktemp(name)), cfg, w))
    return _MODELS[name]


def _engine(path, dt, pool_tokens=256, block=16, max_seqs=4):
    from deepspeedsyclsupport_b200.inference.v2.config_v2 import RaggedInferenceEngineConfig
    from deepspeedsyclsupport_b200.inference.v2.engine_factory import build_hf_engine
    from deepspeedsyclsupport_b200.inference.v2.ragged.manager_configs import AllocationMode, DSStateManagerConfig, MemoryConfig
    mgr = DSStateManagerConfig(max_tracked_sequences=max_seqs, max_ragged_sequence_count=max_seqs, max_ragged_batch_size=pool_tokens, max_context=pool_tokens,
                               memory_config=MemoryConfig(mode=AllocationMode.ALLOCATE, size=pool_tokens // block), kv_block_size=block)
    return build_hf_engine(path, RaggedInferenceEngineConfig(state_manager=mgr), dtype=dt)


def _close(got, want, dt):
    """Every logit row agrees up to a per-row shift, relative to the spread of the logits.  fp32: tightly.  bf16: within a few times what
    rounding of the matrix products does to these small random models, far below what a wrong key or a lost state causes (order 1)."""
    d = got.cpu().double() - want
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.std()
    if dt == torch.float32:
        return float(err.max()) < 5e-5, float(err.max())
    return float(err.max()) < 0.15 and (len(err) < 8 or float(err.median()) < 0.04), (float(err.median()), float(err.max()))


def _tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n, ), generator=torch.Generator().manual_seed(seed))


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_every_layer(name, dt, tmp_path_factory):
    cfg, w, path = _model(name, tmp_path_factory)
    eng = _engine(path, dt)
    toks = _tokens(cfg, 75, 1)
    want, res = O.run(cfg, w, toks.tolist(), collect_layers=True)
    got_res = []
    eng.model()._layer_hook = lambda li, x: got_res.append(x.clone())
    got = eng.put([7], [toks], logit_positions=[list(range(75))])
    assert got.shape == (75, cfg["vocab"]) and len(got_res) == len(res)
    for r, (a, b) in enumerate(zip(got_res, res)):
        row = (a.cpu().double() - b).norm(dim=-1) / b.norm(dim=-1)
        assert float(row.max()) < (5e-5 if dt == torch.float32 else 0.15) and float(row.median()) < (1e-5 if dt == torch.float32 else 0.03), f"layer {r}"
    ok, err = _close(got, want, dt)
    assert ok, err
    if cfg["logit_softcap"]:
        assert float(got.abs().max()) < cfg["logit_softcap"] < float(O.run(dict(cfg, logit_softcap=0.0), w, toks.tolist()).abs().max())  # the cap is at work
    eng.model()._layer_hook = None  # the same without the per-layer sums: every join happens inside the next norm, the last one inside the final norm
    eng.flush(7)
    again = eng.put([8], [toks], logit_positions=[[3, 74]])
    assert _close(again, want[[3, 74]], dt)[0]


@gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name,cuts", [("odd", [1] * 60), ("odd", [2, 2, 15, 1, 17, 3, 2, 18]), ("aligned", [16, 16, 1, 1, 6, 2, 30]), ("aligned", [31, 2, 7, 32]),
                                       ("stateless", [3, 33, 2, 2, 1, 1, 9]), ("many", [2, 14, 1, 1, 17, 2, 20])])
def test_portions_and_token_by_token_equal_the_whole_prompt(name, cuts, dt, tmp_path_factory):
    """Prefill against decoding token by token, and portions cut inside pages (block 16), chunks and windows, down to two tokens."""
    cfg, w, path = _model(name, tmp_path_factory)
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
    cfg, w, path = _model(name, tmp_path_factory)
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
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_long_decoding_through_the_step_graphs(name, dt, tmp_path_factory):
    """A prompt, then 150 single-token steps (the steady-state ones replay a captured graph) across pages, chunks and windows; some steps ask for no
    logits."""
    cfg, w, path = _model(name, tmp_path_factory)
    eng = _engine(path, dt, pool_tokens=256, block=16)
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
    ok, err = _close(torch.cat(got), want[keep], dt)
    assert ok, err
    graphs = eng.model()._graphs
    assert 1 in graphs and (1, 0) in graphs, list(graphs)


@gpu
def test_greedy_generation_through_the_scheduler(tmp_path_factory):
    """Prompts are split into portions and fused with running decodes; the tokens are those of the oracle."""
    from deepspeedsyclsupport_b200.inference.v2.scheduler import SplitFuseScheduler
    cfg, w, path = _model("odd", tmp_path_factory)
    eng = _engine(path, torch.float32, pool_tokens=192, block=16)
    sched = SplitFuseScheduler(eng, token_budget=24)
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
    """The same 330 tokens whole, in portions around the kernels' tile, and half of them one by one: bf16 logits agree with the oracle and with one
    another however they were cut."""
    cfg, w, path = _model("aligned", tmp_path_factory)
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
